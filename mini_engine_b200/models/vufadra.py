"""Vufadra laid out as parts.

The embedding adds a row of a table of token pairs.  A layer runs its mixer and its gated feed-forward side by side, each behind
a dynamic-tanh norm of the same stream, ``x <- x + (mixer(shift(norm1(x))) + ff(norm2(x)))``; the mixer's input is shifted by one
token, element by element.  A layer's mixer is one of

* ``general_delta``: the generalized delta rule, a matrix state per head with a decay and a removal rate per key channel;
* ``parallel``: attention inside chunks of positions with sigmoid weights, per-head q/k norms and stretched rotary positions,
  beside time mixing (a matrix state per head with a bonus for the current token); half the sum of the two normed outputs;
* ``rglru``: the real-gated linear recurrence behind a short convolution.

A span of layers may run several times in a row with the same weights, each pass with caches and states of its own; in front of
a pass the stream and the embedding's output go through a product and a vector of the pass is added.  Every size and every
constant that models of this design may differ in comes from the typed configuration, layer by layer; the constants below are
fixed by the design.
"""

from __future__ import annotations

import math

from mini_engine_b200.config.model_spec import LayerSpec, ModelSpec, OrderEntry, PartSpec
from mini_engine_b200.config.registry import Architecture, register_architecture
from mini_engine_b200.config.vufadra import ChunkedAttentionBranch, ParallelMixer, RecurrentMixer, StateHeads, VufadraConfig

UNIT_EPS = 1e-6  # under the root of the unit norm of the delta rule's keys
DECAY_SCALE = math.exp(-0.5)  # the delta rule's largest decay rate
DECAY_SHARPNESS = 8.0  # of the gated linear recurrence
BRANCH_SHARE = 0.5  # of each branch of a parallel mixer


def _general_delta(mixer: StateHeads, eps: float) -> PartSpec:
    names = {key: f"mix.{key}" for key in ("r", "k", "v", "g", "a", "w1", "w2", "w0", "norm", "o")}
    return PartSpec(
        "generalized_delta_rule",
        {
            "num_heads": mixer.heads, "head_dim": mixer.dim, "decay_rank": mixer.decay_rank, "norm_eps": eps,
            "decay_scale": DECAY_SCALE, "unit_eps": UNIT_EPS, "names": {**names, "a_bias": "mix.a.b"},
        },
    )  # fmt: skip


def _attention(branch: ChunkedAttentionBranch, eps: float) -> PartSpec:
    # double angles: the norms' exactness in float32 would otherwise be lost to the angles of far positions
    rope = {"head_dim": branch.dim, "theta": branch.rot.base, "rotary_dim": branch.rot.dims, "double_angles": True}
    if branch.rot.scaling is not None:
        rope["yarn"] = dict(zip(("factor", "original", "fast", "slow"), branch.rot.scaling))
    return PartSpec(
        "gqa_attention",
        {
            "num_heads": branch.heads, "kv_heads": branch.kv_heads, "head_dim": branch.dim, "value_dim": branch.vdim,
            "qk_norm_eps": eps, "position_encoding": PartSpec("rope", rope), "scale": branch.scale, "chunk": branch.chunk,
            "weights": "sigmoid",
            "names": {"q": "q", "k": "k", "v": "v", "o": "o", "q_norm": "q.norm", "k_norm": "k.norm", "weight_bias": "pb"},
        },
    )  # fmt: skip


def _time_mixing(branch: StateHeads, eps: float) -> PartSpec:
    names = {key: key for key in ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")}
    return PartSpec(
        "time_mixing",
        {
            "num_heads": branch.heads, "head_dim": branch.dim, "decay_rank": branch.decay_rank, "norm_eps": eps,
            "names": {**names, **{f"mu_{s}": f"mu.{s}" for s in "rkvgw"}},
        },
    )  # fmt: skip


def _parallel(mixer: ParallelMixer, eps: float) -> PartSpec:
    branches = [
        {"mixer": part, "factor": BRANCH_SHARE, "prefix": f"mix.{side}.", "norm": f"mix.{side}.out", "norm_eps": eps}
        for side, part in (("left", _attention(mixer.left, eps)), ("right", _time_mixing(mixer.right, eps)))
    ]
    return PartSpec("parallel_mixers", {"branches": branches})


def _rglru(mixer: RecurrentMixer, eps: float) -> PartSpec:
    return PartSpec(
        "gated_linear_recurrence",
        {
            "channels": mixer.width, "blocks": mixer.blocks, "taps": mixer.conv, "sharpness": DECAY_SHARPNESS,
            "names": {"y": "mix.y", "y_bias": "mix.y.b", "x": "mix.x", "x_bias": "mix.x.b", "conv": "mix.conv",
                      "conv_bias": "mix.conv.b", "ra": "mix.ra", "ra_bias": "mix.ra.b", "ri": "mix.ri", "ri_bias": "mix.ri.b",
                      "lam": "mix.lam", "o": "mix.o"},
        },
    )  # fmt: skip


_MIXERS = {"general_delta": _general_delta, "parallel": _parallel, "rglru": _rglru}


def vufadra_spec(cfg: VufadraConfig) -> ModelSpec:
    layers = []
    for index, layer in enumerate(cfg.layers):
        norms = {"mixer": "norm1"}
        unused: tuple[str, ...] = ("norm2", "norm2.b", "norm2.alpha")  # what a checkpoint may carry for a layer without feed-forward
        if layer.ff is not None:
            norms["feed_forward"], unused = "norm2", ()
        layers.append(
            LayerSpec(
                prefix=f"l{index}.", block="parallel_two_norms" + ("_mixer_only" if layer.ff is None else ""),
                mixer=_MIXERS[layer.type](layer.mixer, cfg.norm_eps),
                feed_forward=None if layer.ff is None else PartSpec(
                    "gated_mlp", {"intermediate_size": layer.ff, "names": {"gate": "mlp.gate", "up": "mlp.up", "down": "mlp.down"}}
                ),
                norms={key: PartSpec("dynamic_tanh", {"name": name}) for key, name in norms.items()},
                block_params={"shift": "shift", "unused_names": unused},
            )
        )  # fmt: skip
    embedding = PartSpec("token_embedding", {"weight": "embed"})
    if cfg.bigram is not None:
        embedding = PartSpec(
            "pair_hash_embedding",
            {"weight": "embed", "pair_weight": "bigram", "buckets": cfg.bigram.buckets, "mul_prev": cfg.bigram.mul_prev, "mul_cur": cfg.bigram.mul_cur},
        )
    junctions: tuple[PartSpec, ...] = ()
    if cfg.loop is not None:
        junctions = (PartSpec("reinjection", {"weight": "loop.in", "step": "loop.step", "turns": cfg.loop.times}),)
    return ModelSpec(
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        embedding=embedding,
        layers=tuple(layers),
        order=tuple(OrderEntry(index, junction=None if turn is None else 0, turn=turn or 0) for index, turn in cfg.execution()),
        final_norm=PartSpec("dynamic_tanh", {"name": "final.norm"}),
        head=PartSpec("linear_head", {"weight": "head"}),
        junctions=junctions,
    )


register_architecture(
    Architecture(
        name=VufadraConfig.architecture,
        read_config=VufadraConfig.from_folder,
        build_spec=vufadra_spec,
        config_type=VufadraConfig,
    )
)
