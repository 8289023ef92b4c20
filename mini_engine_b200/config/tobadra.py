"""Typed configuration of the Tobadra decoder, read from its own ``config.json`` keys.

``config.json`` gives ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``canon.taps`` (taps of the convolution in
front of every mixer), ``logit_scale`` (absent: 1) and ``layers``: one entry per layer with its ``type`` (``attention``,
``lightning`` or ``channel_delta``), the mixer's sizes and constants under ``mixer`` and its feed-forward under ``mlp``
(``null``: the layer has none; ``kind`` ``dense`` or ``moe``).  ``weights_of: j`` says that a layer uses layer ``j``'s
tensors with a cache and states of its own.  Layers may differ from one another in every size and come in any order.
The ranks of the two low-rank projections of a ``channel_delta`` mixer are no keys of the configuration but the shapes of
their tensors, so they are read from the checkpoint's header (a configuration made in memory names them in ``mixer``).
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from mini_engine_b200.config.bizurax import Rotation
from mini_engine_b200.config.pimezen import _need
from mini_engine_b200.config.qwen3 import ConfigError

NUMBER = (int, float)


@dataclass(frozen=True)
class RotatedValueAttentionMixer:
    """Windowed grouped-query attention with biases whose values are rotated like the keys."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None
    rot: Rotation

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "RotatedValueAttentionMixer":
        dim = _need(raw, "dim", int, where)
        mask = raw.get("mask")
        out = cls(
            heads=_need(raw, "heads", int, where),
            kv_heads=_need(raw, "kv_heads", int, where),
            dim=dim,
            vdim=_need(raw, "vdim", int, where),
            scale=float(_need(raw, "scale", NUMBER, where)),
            window=None if mask is None else _need(mask, "size", int, where + "mask."),
            rot=Rotation.from_dict(_need(raw, "rot", Mapping, where), where + "rot.", max(dim, 2)),
        )
        if min(out.heads, out.kv_heads, out.dim, out.vdim) < 1 or (out.window is not None and out.window < 1):
            raise ConfigError(f"{where}: sizes must be positive")
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}heads ({out.heads}) must be a multiple of kv_heads ({out.kv_heads})")
        if out.vdim % 2:
            raise ConfigError(f"{where}vdim must be even (its elements are rotated in pairs), got {out.vdim}")
        return out

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale, "rot": self.rot.to_dict()}  # fmt: skip
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class LightningMixer:
    """Linear attention with a fixed decay per head behind silu activations."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "LightningMixer":
        decay = _need(raw, "decay", list, where)
        if not all(isinstance(a, NUMBER) and not isinstance(a, bool) for a in decay):
            raise ConfigError(f"{where}decay must be a list of numbers")
        out = cls(
            heads=_need(raw, "heads", int, where),
            dim=_need(raw, "dim", int, where),
            vdim=_need(raw, "vdim", int, where),
            decay=tuple(float(a) for a in decay),
        )
        if min(out.heads, out.dim, out.vdim) < 1:
            raise ConfigError(f"{where}: sizes must be positive")
        if len(out.decay) != out.heads or not all(0.0 < a <= 1.0 for a in out.decay):
            raise ConfigError(f"{where}decay must hold one number in (0, 1] per head ({out.heads}), got {list(out.decay)}")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ChannelDeltaMixer:
    """The gated delta rule with one decay per head and key channel, behind short convolutions."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str, ranks: tuple[int, int] | None = None) -> "ChannelDeltaMixer":
        decay_rank, gate_rank = ranks or (None, None)
        decay_rank, gate_rank = raw.get("decay_rank", decay_rank), raw.get("gate_rank", gate_rank)
        if decay_rank is None or gate_rank is None:
            raise ConfigError(f"{where}: the ranks of the decay's and the gate's projections are neither given nor found in the checkpoint")
        out = cls(
            heads=_need(raw, "heads", int, where),
            kv_heads=_need(raw, "kv_heads", int, where),
            dim=_need(raw, "dim", int, where),
            vdim=_need(raw, "vdim", int, where),
            conv=_need(raw, "conv", int, where),
            decay_rank=int(decay_rank),
            gate_rank=int(gate_rank),
        )
        if min(out.heads, out.kv_heads, out.dim, out.vdim, out.conv, out.decay_rank, out.gate_rank) < 1:
            raise ConfigError(f"{where}: sizes must be positive")
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}heads ({out.heads}) must be a multiple of kv_heads ({out.kv_heads})")
        return out

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv,
                "decay_rank": self.decay_rank, "gate_rank": self.gate_rank}  # fmt: skip


@dataclass(frozen=True)
class FeedForward:
    """``dense``: ``ff`` features behind a tanh-GELU.  ``moe``: ``experts`` small units of ``ff`` features and
    ``identity`` units that return their input, of which a token uses ``top``, chosen within the ``group_keep`` best
    of ``group_count`` groups; and a unit of ``shared_ff`` features (0: none) that every token uses."""

    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    identity: int = 0
    scale: float = 1.0
    group_count: int = 1
    group_keep: int = 1
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], where: str) -> "FeedForward":
        kind = _need(raw, "kind", str, where)
        if kind == "dense":
            out = cls("dense", _need(raw, "ff", int, where))
        elif kind == "moe":
            router, shared = _need(raw, "router", Mapping, where), raw.get("shared")
            groups, scale = router.get("groups"), router.get("scale")
            identity = router.get("identity")
            count, keep = (1, 1) if groups is None else (_need(groups, k, int, where + "router.groups.") for k in ("count", "keep"))
            out = cls(
                "moe",
                _need(_need(raw, "expert", Mapping, where), "ff", int, where + "expert."),
                experts=_need(router, "experts", int, where + "router."),
                top=_need(router, "top", int, where + "router."),
                identity=0 if identity is None else _need(router, "identity", int, where + "router."),
                scale=1.0 if scale is None else float(_need(router, "scale", NUMBER, where + "router.")),
                group_count=count,
                group_keep=keep,
                shared_ff=0 if shared is None else _need(shared, "ff", int, where + "shared."),
            )
            units = out.experts + out.identity
            if out.experts < 1 or out.identity < 0 or out.shared_ff < 0:
                raise ConfigError(f"{where}: router.experts must be positive, router.identity and shared.ff not negative")
            if count < 1 or units % count or not 1 <= keep <= count or not 1 <= out.top <= keep * (units // count):
                raise ConfigError(f"{where}router: {units} units do not form {count} equal groups of which {keep} hold {out.top} choices")
        else:
            raise ConfigError(f"{where}kind {kind!r} is not a feed-forward of this design (known: 'dense', 'moe')")
        if out.ff < 1:
            raise ConfigError(f"{where}ff must be positive")
        return out

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        router: dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if self.identity:
            router["identity"] = self.identity
        if (self.group_count, self.group_keep) != (1, 1):
            router["groups"] = {"count": self.group_count, "keep": self.group_keep}
        out: dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff:
            out["shared"] = {"ff": self.shared_ff}
        return out


MIXERS = {"attention": RotatedValueAttentionMixer, "lightning": LightningMixer, "channel_delta": ChannelDeltaMixer}


@dataclass(frozen=True)
class TobadraLayer:
    type: str  # a key of MIXERS
    mixer: RotatedValueAttentionMixer | LightningMixer | ChannelDeltaMixer
    mlp: FeedForward | None
    weights_of: int | None = None  # the layer whose tensors this one uses

    def to_dict(self) -> dict[str, Any]:
        out = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


def _owner(layers: list, index: int) -> int:
    """The layer whose tensors layer ``index`` uses: itself, or the end of its chain of ``weights_of``."""
    seen = [index]
    while layers[seen[-1]].get("weights_of") is not None:
        target = _need(layers[seen[-1]], "weights_of", int, f"layers[{seen[-1]}].")
        if not 0 <= target < len(layers) or target in seen:
            raise ConfigError(f"layers[{index}].weights_of must lead to a layer with tensors of its own, got {target}")
        seen.append(target)
    return seen[-1]


@dataclass(frozen=True)
class TobadraConfig:
    vocab: int
    width: int
    norm_eps: float
    canon_taps: int
    logit_scale: float
    layers: tuple[TobadraLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    architecture = "Tobadra"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def owner_of(self, index: int) -> int:
        """The layer whose tensors layer ``index`` uses."""
        while self.layers[index].weights_of is not None:
            index = self.layers[index].weights_of
        return index

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any], ranks: Mapping[int, tuple[int, int]] | None = None) -> "TobadraConfig":
        """``ranks``: per layer with tensors of its own the ranks of a ``channel_delta`` mixer's decay and gate
        projections (from the checkpoint's tensor shapes); ``mixer.decay_rank`` and ``mixer.gate_rank`` are used where
        present."""
        if raw.get("architecture") != cls.architecture:
            raise ConfigError(f"architecture must be {cls.architecture!r}, got {raw.get('architecture')!r}")
        norm, canon = _need(raw, "norm", Mapping, ""), _need(raw, "canon", Mapping, "")
        entries = _need(raw, "layers", list, "")
        if not entries:
            raise ConfigError("config.json lists no layers")
        layers: list[TobadraLayer] = []
        for index, entry in enumerate(entries):
            where = f"layers[{index}]."
            kind = _need(entry, "type", str, where)
            if kind not in MIXERS:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design (known: {', '.join(map(repr, MIXERS))})")
            owner = _owner(entries, index)
            mixer_raw = _need(entry, "mixer", Mapping, where)
            if kind == "channel_delta":
                own = entries[owner].get("mixer") or {}
                given = (own["decay_rank"], own["gate_rank"]) if "decay_rank" in own and "gate_rank" in own else (ranks or {}).get(owner)
                mixer = ChannelDeltaMixer.from_dict(mixer_raw, where + "mixer.", given)
            else:
                mixer = MIXERS[kind].from_dict(mixer_raw, where + "mixer.")
            mlp_raw = entry.get("mlp")
            mlp = None if mlp_raw is None else FeedForward.from_dict(mlp_raw, where + "mlp.")
            layers.append(TobadraLayer(kind, mixer, mlp, entry.get("weights_of")))
        for index, layer in enumerate(layers):
            held = layers[_owner(entries, index)]
            if (layer.type, layer.mixer, layer.mlp) != (held.type, held.mixer, held.mlp):
                raise ConfigError(f"layers[{index}] uses the tensors of layer {_owner(entries, index)} but differs from it")
        scale, eos = raw.get("logit_scale"), raw.get("eos_token_id")
        out = cls(
            vocab=_need(raw, "vocab", int, ""),
            width=_need(raw, "width", int, ""),
            norm_eps=float(_need(norm, "eps", NUMBER, "norm.")),
            canon_taps=_need(canon, "taps", int, "canon."),
            logit_scale=1.0 if scale is None else float(_need(raw, "logit_scale", NUMBER, "")),
            layers=tuple(layers),
            eos_token_ids=() if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos)),
        )
        if min(out.vocab, out.width, out.canon_taps) < 1 or not out.norm_eps > 0:
            raise ConfigError("vocab, width, canon.taps and norm.eps must be positive")
        return out

    @classmethod
    def from_folder(cls, folder: str | Path) -> "TobadraConfig":
        from mini_engine_b200.weights.safetensors_io import read_folder_index

        folder = Path(folder)
        raw = json.loads((folder / "config.json").read_text())
        index = read_folder_index(folder) if any(folder.glob("*.safetensors")) else {}
        ranks: dict[int, tuple[int, int]] = {}
        for layer in range(len(raw.get("layers") or [])):
            names = [f"l{layer}.mix.{which}" for which in ("a1", "g1")]
            if all(name in index for name in names):
                ranks[layer] = tuple(int(index[name].entries[name][1][0]) for name in names)  # type: ignore[assignment]
        return cls.from_dict(raw, ranks)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
            "canon": {"taps": self.canon_taps}, "logit_scale": self.logit_scale, "layers": [layer.to_dict() for layer in self.layers],
        }  # fmt: skip
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out
