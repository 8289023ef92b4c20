"""Host-side pieces of the Tobadra design: its configuration and registry entry, ranks read from the checkpoint, the
tensors it declares, layers that use another layer's tensors, what its layers ask of the cache manager (pages, matrix
states, the convolutions' pasts), and identities of the plain implementation: lightning attention against its sum over
earlier tokens, the delta rule's correction, and rotated values against values turned by the distance."""

from __future__ import annotations

import copy
import json

import pytest
import torch

import plain_tobadra as plain
from mini_engine_b200.cache.storage import allocate_cache, plan_groups
from mini_engine_b200.config import TobadraConfig, load_model_config
from mini_engine_b200.config.qwen3 import ConfigError
from mini_engine_b200.config.registry import architecture_for
from mini_engine_b200.parts.base import PagedCacheSpec, StateSpec
from mini_engine_b200.parts.model import DecoderModel, declared_weights
from mini_engine_b200.weights import write_random_model


def raw_config():
    attention = {"heads": 6, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.4, "mask": {"size": 11}, "rot": {"base": 500.0, "dims": 12}}
    delta = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 12, "conv": 4, "decay_rank": 5, "gate_rank": 7}
    routed = {"kind": "moe", "expert": {"ff": 16}, "shared": {"ff": 24},
              "router": {"experts": 6, "top": 3, "identity": 2, "scale": 1.7, "groups": {"count": 4, "keep": 2}}}  # fmt: skip
    return copy.deepcopy({
        "architecture": "Tobadra", "vocab": 90, "width": 48, "norm": {"eps": 2e-5}, "canon": {"taps": 3}, "logit_scale": 0.7,
        "layers": [
            {"type": "channel_delta", "mixer": delta, "mlp": routed},
            {"type": "lightning", "mixer": {"heads": 3, "dim": 16, "vdim": 24, "decay": [0.9, 0.99, 1.0]}, "mlp": None},
            {"type": "attention", "mixer": attention, "mlp": {"kind": "dense", "ff": 40}},
            {"type": "channel_delta", "mixer": delta, "mlp": routed, "weights_of": 0},
            {"type": "attention", "mixer": attention, "mlp": {"kind": "dense", "ff": 40}, "weights_of": 2},
            {"type": "lightning", "mixer": {"heads": 1, "dim": 8, "vdim": 8, "decay": [0.5]},
             "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 4, "top": 2, "scale": 1.0}}},
        ],
    })  # fmt: skip


def test_config_round_trip_and_registry(tmp_path):
    cfg = TobadraConfig.from_dict(raw_config())
    assert TobadraConfig.from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == raw_config()
    assert cfg.layers[2].mixer.window == 11 and cfg.layers[0].mlp.identity == 2 and cfg.layers[5].mlp.group_count == 1
    assert [cfg.owner_of(i) for i in range(6)] == [0, 1, 2, 0, 2, 5] and cfg.canon_taps == 3 and cfg.logit_scale == 0.7
    write_random_model(tmp_path, cfg, seed=1)
    arch, loaded = load_model_config(tmp_path)
    assert arch.name == "Tobadra" and loaded == cfg


def test_the_low_ranks_come_from_the_checkpoint_when_the_config_is_silent(tmp_path):
    cfg = TobadraConfig.from_dict(raw_config())
    write_random_model(tmp_path, cfg, seed=1)
    raw = raw_config()
    for entry in raw["layers"]:
        entry["mixer"].pop("decay_rank", None), entry["mixer"].pop("gate_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    _, loaded = load_model_config(tmp_path)
    assert loaded == cfg  # the layer that uses layer 0's tensors included
    with pytest.raises(ConfigError, match="ranks"):
        TobadraConfig.from_dict(raw)


@pytest.mark.parametrize(
    "path,value,message",
    [
        (("layers", 0, "type"), "conv", "not a mixer"),
        (("layers", 5, "mixer", "decay"), [0.5, 0.5], "one number"),
        (("layers", 1, "mixer", "decay"), [0.9, 0.99, 1.5], "one number"),
        (("layers", 1, "mixer", "dim"), 0, "positive"),
        (("layers", 3, "weights_of"), 6, "weights_of"),
        (("layers", 3, "weights_of"), 3, "weights_of"),
        (("layers", 3, "weights_of"), 1, "differs"),
        (("layers", 5, "mlp", "kind"), "gated", "not a feed-forward"),
        (("layers", 5, "mlp", "router", "top"), 5, "groups"),
        (("layers", 5, "mlp", "router", "groups"), {"count": 3, "keep": 1}, "groups"),
        (("layers", 5, "mlp", "router", "identity"), -1, "negative"),
        (("canon", "taps"), 0, "positive"),
        (("canon",), None, "lacks the key"),
        (("norm",), None, "lacks the key"),
    ],
)
def test_config_errors_name_the_key(path, value, message):
    raw = raw_config()
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=message):
        TobadraConfig.from_dict(raw)


@pytest.mark.parametrize("key,value,message", [("heads", 5, "multiple of kv_heads"), ("vdim", 7, "even"), ("mask", {"size": 0}, "positive"),
                                               ("rot", {"base": 10.0, "dims": 18}, "dims"), ("rot", {"base": 10.0, "dims": 3}, "dims")])  # fmt: skip
def test_attention_config_errors(key, value, message):
    raw = raw_config()
    raw["layers"] = [raw["layers"][2]]
    raw["layers"][0]["mixer"][key] = value
    with pytest.raises(ConfigError, match=message):
        TobadraConfig.from_dict(raw)


def test_declared_tensors_and_the_order_of_layers():
    spec = architecture_for("Tobadra").build_spec(TobadraConfig.from_dict(raw_config()))
    declared = {s.name: s for s in declared_weights(spec)}
    assert [(entry.layer, entry.cache_of) for entry in spec.order] == [(0, None), (1, None), (2, None), (0, None), (2, None), (3, None)]
    assert [layer.prefix for layer in spec.layers] == ["l0.", "l1.", "l2.", "l5."] and not any(n.startswith(("l3.", "l4.")) for n in declared)
    assert [layer.block for layer in spec.layers] == ["gated_sandwich", "gated_sandwich_mixer_only", "gated_sandwich", "gated_sandwich"]
    assert declared["embed"].shape == (90, 48) and declared["embed.norm"].shape == (48,) and declared["head"].alias_of == "embed"
    for name in ("norm1", "norm1b", "norm2", "norm2b", "rg1.b", "rg2.b"):
        assert declared["l0." + name].shape == (48,) and declared["l0." + name].role == "vector"
    assert declared["l0.rg1"].shape == (48, 48) and declared["l0.canon1"].shape == (48, 3)
    # a layer without feed-forward: a checkpoint may carry what belongs to one
    assert all(declared["l1." + n].optional for n in ("norm2", "norm2b", "rg2", "rg2.b")) and not declared["l1.rg1"].optional
    assert declared["l0.mix.q"].shape == (32, 48) and declared["l0.mix.v"].shape == (48, 48) and declared["l0.mix.v.conv"].shape == (48, 4)
    assert declared["l0.mix.b"].shape == (4, 48) and declared["l0.mix.A_log"].shape == (4,) and declared["l0.mix.dt_bias"].shape == (64,)
    assert declared["l0.mix.a1"].shape == (5, 48) and declared["l0.mix.a2"].shape == (64, 5) and declared["l0.mix.g2"].shape == (48, 7)
    assert declared["l0.mix.norm"].shape == (12,) and declared["l1.mix.norm"].shape == (72,) and declared["l1.mix.g"].shape == (72, 48)
    assert declared["l2.mix.q.b"].shape == (96,) and declared["l2.mix.v.b"].shape == (48,) and declared["l2.mix.o.b"].shape == (48,)
    assert declared["l2.mlp.up"].shape == (40, 48) and "l2.mlp.gate" not in declared
    assert declared["l0.mlp.router"].shape == (8, 48) and declared["l0.mlp.correction"].shape == (8,) and "l0.mlp.e6.up" not in declared
    assert declared["l0.mlp.e5.up"].shape == (16, 48) and "l0.mlp.e5.gate" not in declared and declared["l0.mlp.shared.sg"].shape == (1, 48)
    assert "l5.mlp.shared.up" not in declared and declared["l5.mlp.correction"].shape == (4,)


def test_caches_and_states_of_every_layer():
    model = DecoderModel(architecture_for("Tobadra").build_spec(TobadraConfig.from_dict(raw_config())))
    needs, blocks = model.cache_needs(), model.block_states()
    matrix, past = 4 * 16 * 12, 3 * (2 * 2 * 16 + 4 * 12)
    assert needs[0] == needs[3] == (None, StateSpec((matrix + past,), torch.float32), None)
    assert needs[1] == (None, StateSpec((3, 16, 24), torch.float32), None)
    assert needs[2] == needs[4] == (PagedCacheSpec(2, 16, 11, 24, 0), None, None)
    assert blocks == [StateSpec((2, 48), torch.float32)] * 6 and model.capturable and not model.programmatic_launch
    specs, group_of = plan_groups(needs)
    assert len(specs) == 1 and group_of == [None, None, 0, None, 0, None]
    layout = allocate_cache(needs, 8, 4, 2, torch.float32, "cpu", max_step_tokens=16, block_states=blocks)
    assert layout.has_state and len(layout.slot_groups) == 4 + 6
    views = layout.views
    assert views[0].state.shape == (3, matrix + past) and views[0].block_state.shape == (3, 2, 48)
    # a layer that uses another one's tensors has pages, states and a past of its own
    for a, b in ((0, 3), (2, 4)):
        for name in ("state", "block_state", "k", "v"):
            x, y = getattr(views[a], name), getattr(views[b], name)
            assert (x is None) == (y is None) and (x is None or x.data_ptr() != y.data_ptr())


def test_a_model_with_one_tap_has_no_past():
    raw = raw_config()
    raw["canon"]["taps"] = 1
    model = DecoderModel(architecture_for("Tobadra").build_spec(TobadraConfig.from_dict(raw)))
    assert model.block_states() == [None] * 6


def test_plain_lightning_equals_the_sum_over_earlier_tokens():
    torch.manual_seed(0)
    q, k, v = (torch.randn(9, 2, n, dtype=torch.float64) for n in (6, 6, 5))
    decay = [0.9, 0.5]
    got, _ = plain.lightning_recurrence(q, k, v, decay)
    for t in range(9):
        for h in range(2):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(got[t, h], want)


def test_plain_delta_rule_replaces_what_a_key_held():
    """With beta 1 and no decay, writing to a unit key a second time leaves the second value alone; a key orthogonal to
    it keeps its own; a decay of zero on a key's channel forgets it."""
    k = torch.eye(3, dtype=torch.float64)[[0, 1, 0, 2]].unsqueeze(1)
    v = torch.randn(4, 1, 5, dtype=torch.float64)
    one = torch.ones(4, 1, dtype=torch.float64)
    g = torch.ones(4, 1, 3, dtype=torch.float64)
    out, state = plain.delta_recurrence(k, k, v, one, g)
    assert torch.allclose(out, v) and torch.allclose(state[0], v[[2, 1, 3], 0])
    g[3, 0, 1] = 0.0
    assert torch.allclose(plain.delta_recurrence(k, k, v, one, g)[1][0, 1], torch.zeros(5, dtype=torch.float64))


def test_plain_rotated_values_depend_on_the_distance_alone():
    torch.manual_seed(1)
    q, k, v = torch.randn(7, 2, 4).double(), torch.randn(7, 1, 4).double(), torch.randn(7, 1, 6).double()
    here = plain.attention_heads(q, k, v, 0.5, 30.0, 4)
    later = plain.attention_heads(q, k, v, 0.5, 30.0, 4, positions=torch.arange(7) + 1000)
    assert torch.allclose(here, later, atol=1e-9)
    unturned = torch.softmax((q[6, 0] @ k[3:, 0].T) * 0.5, -1) @ v[3:, 0]
    assert not torch.allclose(here[6, 0], unturned, atol=1e-2)
