"""Tobadra laid out as parts.

The embedding's rows are RMS-normed.  Every sublayer stands between two norms and behind a gate: ``x <- x +
norm_b(sigmoid(W_r h + b_r) * sublayer(h))`` with ``h = norm_a(x)``; a mixer reads ``h`` plus a short causal convolution
of ``h`` over time.  A layer's mixer is one of

* ``attention``: grouped-query attention in a sliding window with biases on all four projections and a rotation that
  also turns the values: a value is cached turned by its own position, a head's output is turned back by the query's;
* ``lightning``: linear attention with a fixed decay per head, silu on q, k and v, one norm over all heads and a sigmoid
  gate;
* ``channel_delta``: the gated delta rule with a decay per head and key channel behind short convolutions, unit q and k,
  a norm per head and a low-rank sigmoid gate.

The feed-forward is a tanh-GELU unit without a gate, or routed GELU units (softmax over all units, a correction that
enters the choice but not the weights, groups valued by their best unit, units that return their input) beside a
shared unit with a sigmoid gate per token.  A layer may use another layer's tensors with a cache and states of its own.
The head is the embedding table, its logits scaled.  Every size and every constant that models of this design may
differ in comes from the typed configuration, layer by layer; the constants below are fixed by the design.
"""

from __future__ import annotations

from mini_engine_b200.config.model_spec import LayerSpec, ModelSpec, OrderEntry, PartSpec
from mini_engine_b200.config.registry import Architecture, register_architecture
from mini_engine_b200.config.tobadra import (
    ChannelDeltaMixer,
    FeedForward,
    LightningMixer,
    RotatedValueAttentionMixer,
    TobadraConfig,
)

UNIT_EPS = 1e-6  # under the root of the unit norm of the delta rule's q and k


def _rope(base: float, dims: int, head_dim: int, divisor: float = 1.0) -> PartSpec:
    return PartSpec("rope", {"head_dim": head_dim, "theta": base, "rotary_dim": dims, "frequency_divisor": divisor, "double_angles": True})


def _attention(mixer: RotatedValueAttentionMixer, eps: float) -> PartSpec:
    return PartSpec(
        "gqa_attention",
        {
            "num_heads": mixer.heads, "kv_heads": mixer.kv_heads, "head_dim": mixer.dim, "value_dim": mixer.vdim,
            "qk_norm_eps": None, "position_encoding": _rope(mixer.rot.base, mixer.rot.dims, mixer.dim, mixer.rot.factor),
            "value_encoding": _rope(mixer.rot.base, mixer.vdim, mixer.vdim), "scale": mixer.scale, "window": mixer.window,
            "qkv_bias": True, "o_bias": True,
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "o": "mix.o", "q_bias": "mix.q.b", "k_bias": "mix.k.b",
                      "v_bias": "mix.v.b", "o_bias": "mix.o.b"},
        },
    )  # fmt: skip


def _lightning(mixer: LightningMixer, eps: float) -> PartSpec:
    return PartSpec(
        "retention",
        {
            "num_heads": mixer.heads, "head_dim": mixer.dim, "value_dim": mixer.vdim, "decay": mixer.decay, "norm_eps": eps,
            "key_scale": 1.0, "qkv_activation": "silu", "norm_scope": "projection", "norm_weight": True, "gate_activation": "sigmoid",
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "g": "mix.g", "o": "mix.o", "norm": "mix.norm"},
        },
    )  # fmt: skip


def _channel_delta(mixer: ChannelDeltaMixer, eps: float) -> PartSpec:
    return PartSpec(
        "gated_delta_rule",
        {
            "num_heads": mixer.heads, "qk_heads": mixer.kv_heads, "head_dim": mixer.dim, "value_dim": mixer.vdim, "taps": mixer.conv,
            "decay_rank": mixer.decay_rank, "gate_rank": mixer.gate_rank, "norm_eps": eps, "unit_eps": UNIT_EPS,
            "names": {"q": "mix.q", "k": "mix.k", "v": "mix.v", "q_conv": "mix.q.conv", "k_conv": "mix.k.conv", "v_conv": "mix.v.conv",
                      "beta": "mix.b", "a_log": "mix.A_log", "a1": "mix.a1", "a2": "mix.a2", "dt_bias": "mix.dt_bias",
                      "norm": "mix.norm", "g1": "mix.g1", "g2": "mix.g2", "o": "mix.o"},
        },
    )  # fmt: skip


def _feed_forward(mlp: FeedForward) -> PartSpec:
    if mlp.kind == "dense":
        return PartSpec("mlp", {"intermediate_size": mlp.ff, "activation": "gelu_tanh", "names": {"up": "mlp.up", "down": "mlp.down"}})
    return PartSpec(
        "routed_experts",
        {
            "units": mlp.experts, "identity_units": mlp.identity, "top": mlp.top, "intermediate_size": mlp.ff, "gated": False,
            "activation": "gelu_erf", "scoring": "softmax_all", "choice_correction": True, "group_count": mlp.group_count,
            "group_keep": mlp.group_keep, "weight_scale": mlp.scale, "shared_intermediate_size": mlp.shared_ff or None,
            "shared_gate": bool(mlp.shared_ff),
            "names": {"router": "mlp.router", "correction": "mlp.correction", "unit": "mlp.e{index}.", "shared": "mlp.shared.",
                      "shared_gate": "mlp.shared.sg", "up": "up", "down": "down"},
        },
    )  # fmt: skip


_MIXERS = {"attention": _attention, "lightning": _lightning, "channel_delta": _channel_delta}


def tobadra_spec(cfg: TobadraConfig) -> ModelSpec:
    eps = cfg.norm_eps
    owners = [index for index in range(len(cfg.layers)) if cfg.layers[index].weights_of is None]
    layers = []
    for index in owners:
        layer = cfg.layers[index]
        norms = {"mixer": "norm1", "mixer_out": "norm1b"}
        gates = {"mixer": ("rg1", "rg1.b")}
        unused: tuple[str, ...] = ("norm2", "norm2b", "rg2", "rg2.b")  # what a checkpoint may carry for a layer without feed-forward
        if layer.mlp is not None:
            norms.update({"feed_forward": "norm2", "feed_forward_out": "norm2b"})
            gates["feed_forward"] = ("rg2", "rg2.b")
            unused = ()
        layers.append(
            LayerSpec(
                prefix=f"l{index}.", block="gated_sandwich" + ("_mixer_only" if layer.mlp is None else ""),
                mixer=_MIXERS[layer.type](layer.mixer, eps),
                feed_forward=None if layer.mlp is None else _feed_forward(layer.mlp),
                norms={key: PartSpec("rmsnorm", {"name": name, "eps": eps}) for key, name in norms.items()},
                block_params={"gates": gates, "conv": "canon1", "taps": cfg.canon_taps, "unused_names": unused},
            )
        )  # fmt: skip
    return ModelSpec(
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        embedding=PartSpec("token_embedding", {"weight": "embed", "norm": "embed.norm", "norm_eps": eps}),
        layers=tuple(layers),
        order=tuple(OrderEntry(owners.index(cfg.owner_of(index))) for index in range(len(cfg.layers))),
        final_norm=PartSpec("rmsnorm", {"name": "final.norm", "eps": eps}),
        head=PartSpec("linear_head", {"weight": "head", "tied_to": "embed", "logit_scale": cfg.logit_scale}),
    )


register_architecture(
    Architecture(
        name=TobadraConfig.architecture,
        read_config=TobadraConfig.from_folder,
        build_spec=tobadra_spec,
        config_type=TobadraConfig,
    )
)
