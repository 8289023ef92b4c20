"""Typed configuration of the Vufadra decoder, read from its own ``config.json`` keys.

``config.json`` gives ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``embedding.bigram`` (``buckets``, ``mul_prev``,
``mul_cur``: the table of token pairs; absent: there is none), ``loop`` (``start``, ``stop``, ``times``: layers ``start .. stop - 1``
run ``times`` times in a row with the same weights, each pass with caches and states of its own; absent: no layer repeats) and
``layers``: one entry per layer with its ``type`` (``general_delta``, ``parallel`` or ``rglru``), the mixer's sizes and constants
under ``mixer`` (a ``parallel`` mixer has those of its two branches under ``left`` and ``right``) and its feed-forward under
``mlp`` (``null``: the layer has none).  Layers may differ from one another in every size and come in any order.  The ranks of
the decays' low-rank projections are no keys of the configuration but the shapes of their tensors, so they are read from the
checkpoint's header (a configuration made in memory names them in ``mixer``).
"""

from __future__ import annotations

import json
import math
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from mini_engine_b200.config.bizurax import LayerLoop
from mini_engine_b200.config.pimezen import _need
from mini_engine_b200.config.qwen3 import ConfigError

NUMBER = (int, float)


@dataclass(frozen=True)
class StretchedRotation:
    """Rotary positions on the first ``dims`` elements of a head, with YaRN's four constants where the model has them."""

    base: float
    dims: int
    scaling: tuple[float, float, float, float] | None = None  # factor, original, fast, slow

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str, most: int) -> "StretchedRotation":
        scaling = raw.get("scaling")
        if scaling is not None:
            scaling = tuple(float(_need(scaling, key, NUMBER, where + "scaling.")) for key in ("factor", "original", "fast", "slow"))
            if not all(value > 0 for value in scaling):
                raise ConfigError(f"{where}scaling: constants must be positive")
        out = cls(float(_need(raw, "base", NUMBER, where)), _need(raw, "dims", int, where), scaling)
        if out.dims % 2 or not 2 <= out.dims <= most:
            raise ConfigError(f"{where}dims must be even and between 2 and {most}, got {out.dims}")
        if not out.base > 0 or (scaling is not None and not out.base > 1):
            raise ConfigError(f"{where}base must be positive (with scaling: above 1)")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return out


@dataclass(frozen=True)
class ChunkedAttentionBranch:
    """Grouped-query attention inside chunks of positions, whose weights are sigmoids and no softmax."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None
    rot: StretchedRotation

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "ChunkedAttentionBranch":
        dim, mask = _need(raw, "dim", int, where), raw.get("mask")
        out = cls(
            heads=_need(raw, "heads", int, where),
            kv_heads=_need(raw, "kv_heads", int, where),
            dim=dim,
            vdim=_need(raw, "vdim", int, where),
            scale=float(_need(raw, "scale", NUMBER, where)),
            chunk=None if mask is None else _need(mask, "size", int, where + "mask."),
            rot=StretchedRotation.from_dict(_need(raw, "rot", Mapping, where), where + "rot.", max(dim, 2)),
        )
        if min(out.heads, out.kv_heads, out.dim, out.vdim) < 1 or (out.chunk is not None and out.chunk < 1):
            raise ConfigError(f"{where}: sizes must be positive")
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}heads ({out.heads}) must be a multiple of kv_heads ({out.kv_heads})")
        if not math.isfinite(out.scale):
            raise ConfigError(f"{where}scale must be finite")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale, "rot": self.rot.to_dict()}  # fmt: skip
        if self.chunk is not None:
            out["mask"] = {"size": self.chunk}
        return out


@dataclass(frozen=True)
class StateHeads:
    """A mixer with a matrix state per head (the generalized delta rule, or time mixing) and a low-rank decay."""

    heads: int
    dim: int
    decay_rank: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str, rank: int | None = None) -> "StateHeads":
        rank = raw.get("decay_rank", rank)
        if rank is None:
            raise ConfigError(f"{where}: the rank of the decay's projection is neither given nor found in the checkpoint")
        out = cls(_need(raw, "heads", int, where), _need(raw, "dim", int, where), int(rank))
        if min(out.heads, out.dim, out.decay_rank) < 1:
            raise ConfigError(f"{where}: sizes must be positive")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "decay_rank": self.decay_rank}


@dataclass(frozen=True)
class ParallelMixer:
    left: ChunkedAttentionBranch
    right: StateHeads

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str, rank: int | None = None) -> "ParallelMixer":
        return cls(
            ChunkedAttentionBranch.from_dict(_need(raw, "left", Mapping, where), where + "left."),
            StateHeads.from_dict(_need(raw, "right", Mapping, where), where + "right.", rank),
        )

    def to_dict(self) -> dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class RecurrentMixer:
    """The real-gated linear recurrence of ``width`` channels whose gates are ``blocks`` square blocks."""

    width: int
    blocks: int
    conv: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "RecurrentMixer":
        out = cls(*(_need(raw, key, int, where) for key in ("width", "blocks", "conv")))
        if min(out.width, out.blocks, out.conv) < 1 or out.width % out.blocks:
            raise ConfigError(f"{where}: sizes must be positive and blocks must divide width")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


# type -> (mixer, the tensor behind "l<i>.mix." whose first extent is the rank of its decay's projection)
MIXERS = {"general_delta": (StateHeads, "w1"), "parallel": (ParallelMixer, "right.w1"), "rglru": (RecurrentMixer, None)}


@dataclass(frozen=True)
class VufadraLayer:
    type: str  # a key of MIXERS
    mixer: StateHeads | ParallelMixer | RecurrentMixer
    ff: int | None  # features of the gated feed-forward; None: the layer has none

    def to_dict(self) -> dict[str, Any]:
        mlp = None if self.ff is None else {"kind": "dense", "ff": self.ff}
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": mlp}


@dataclass(frozen=True)
class PairTable:
    """A second embedding table whose row is chosen by a token and the one in front of it."""

    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class VufadraConfig:
    vocab: int
    width: int
    norm_eps: float
    bigram: PairTable | None
    loop: LayerLoop | None
    layers: tuple[VufadraLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    architecture = "Vufadra"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def execution(self) -> list[tuple[int, int | None]]:
        """The layers' numbers in the order they run; with the first layer of a pass comes the pass's number."""
        count = len(self.layers)
        if self.loop is None:
            return [(index, None) for index in range(count)]
        start, stop = self.loop.start, self.loop.stop
        span = [(index, turn if index == start else None) for turn in range(self.loop.times) for index in range(start, stop)]
        return [(index, None) for index in range(start)] + span + [(index, None) for index in range(stop, count)]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], ranks: Mapping[int, int] | None = None) -> "VufadraConfig":
        """``ranks``: per layer the rank of its decay's projection (from the checkpoint's tensor shapes); ``decay_rank`` in the
        mixer's sizes is used where present."""
        if raw.get("architecture") != cls.architecture:
            raise ConfigError(f"architecture must be {cls.architecture!r}, got {raw.get('architecture')!r}")
        entries = _need(raw, "layers", list, "")
        if not entries:
            raise ConfigError("config.json lists no layers")
        layers: list[VufadraLayer] = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]."
            kind = _need(entry, "type", str, where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design (known: {', '.join(map(repr, MIXERS))})")
            mixer_class, ranked = MIXERS[kind]
            given = ((ranks or {}).get(index),) if ranked else ()
            mixer = mixer_class.from_dict(_need(entry, "mixer", Mapping, where), where + "mixer.", *given)
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                if _need(mlp, "kind", str, where + "mlp.") != "dense":
                    raise ConfigError(f"{where}mlp.kind {mlp['kind']!r} is not a feed-forward of this design (known: 'dense')")
                ff = _need(mlp, "ff", int, where + "mlp.")
                if ff < 1:
                    raise ConfigError(f"{where}mlp.ff must be positive")
            layers.append(VufadraLayer(kind, mixer, ff))
        pairs = (raw.get("embedding") or {}).get("bigram")
        bigram = None if pairs is None else PairTable(*(_need(pairs, key, int, "embedding.bigram.") for key in ("buckets", "mul_prev", "mul_cur")))
        if bigram is not None and (bigram.buckets < 1 or min(bigram.mul_prev, bigram.mul_cur) < 0):
            raise ConfigError("embedding.bigram.buckets must be positive and its multipliers not negative")
        loop_raw, loop = raw.get("loop"), None
        if loop_raw is not None:
            loop = LayerLoop(*(_need(loop_raw, key, int, "loop.") for key in ("start", "stop", "times")))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ConfigError(f"loop must name layers start < stop <= {len(layers)} and times >= 1, got {loop}")
        eos = raw.get("eos_token_id")
        out = cls(
            vocab=_need(raw, "vocab", int, ""),
            width=_need(raw, "width", int, ""),
            norm_eps=float(_need(_need(raw, "norm", Mapping, ""), "eps", NUMBER, "norm.")),
            bigram=bigram,
            loop=loop,
            layers=tuple(layers),
            eos_token_ids=() if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos)),
        )
        if min(out.vocab, out.width) < 1 or not out.norm_eps > 0:
            raise ConfigError("vocab, width and norm.eps must be positive")
        return out

    @classmethod
    def from_folder(cls, folder: str | Path) -> "VufadraConfig":
        from mini_engine_b200.weights.safetensors_io import read_folder_index

        folder = Path(folder)
        raw = json.loads((folder / "config.json").read_text())
        index = read_folder_index(folder) if any(folder.glob("*.safetensors")) else {}
        ranks: dict[int, int] = {}
        for layer, entry in enumerate(raw.get("layers") or []):
            _mixer, tensor = MIXERS.get(entry.get("type"), (None, None))
            name = f"l{layer}.mix.{tensor}"
            if tensor is not None and name in index:
                ranks[layer] = int(index[name].entries[name][1][0])
        return cls.from_dict(raw, ranks)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}}
        if self.bigram is not None:
            out["embedding"] = {"bigram": {"buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur}}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        out["layers"] = [layer.to_dict() for layer in self.layers]
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
