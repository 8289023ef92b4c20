"""Host-side pieces of the Vufadra design: its configuration and registry entry, ranks read from the checkpoint, the tensors it
declares, the order of looped layers and the junction in front of their passes, what its layers ask of the cache manager (pages
of chunks, matrix states, last inputs), pages given back behind a chunk, and identities of the plain implementation."""

from __future__ import annotations

import copy
import json
import math

import pytest
import torch

import plain_vufadra as plain
from mini_engine_b200.cache.manager import NULL_PAGE, CacheManager, GroupSpec
from mini_engine_b200.cache.storage import allocate_cache, plan_groups
from mini_engine_b200.config import VufadraConfig, load_model_config
from mini_engine_b200.config.model_spec import OrderEntry
from mini_engine_b200.config.qwen3 import ConfigError
from mini_engine_b200.config.registry import architecture_for
from mini_engine_b200.parts.attention import GroupedQueryAttention
from mini_engine_b200.parts.base import PagedCacheSpec, StateSpec
from mini_engine_b200.parts.model import DecoderModel, declared_weights
from mini_engine_b200.parts.rotary import RotaryEncoding
from mini_engine_b200.weights import write_random_model


def raw_config():
    scaling = {"factor": 4.0, "original": 64.0, "fast": 8.0, "slow": 1.0}
    left = {"heads": 6, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.4, "mask": {"size": 11}, "rot": {"base": 500.0, "dims": 12, "scaling": scaling}}
    return copy.deepcopy({
        "architecture": "Vufadra", "vocab": 90, "width": 48, "norm": {"eps": 2e-5},
        "embedding": {"bigram": {"buckets": 53, "mul_prev": 31, "mul_cur": 17}}, "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [
            {"type": "general_delta", "mixer": {"heads": 4, "dim": 12, "decay_rank": 5}, "mlp": {"kind": "dense", "ff": 40}},
            {"type": "parallel", "mixer": {"left": left, "right": {"heads": 3, "dim": 16, "decay_rank": 7}}, "mlp": {"kind": "dense", "ff": 56}},
            {"type": "rglru", "mixer": {"width": 36, "blocks": 3, "conv": 4}, "mlp": None},
            {"type": "parallel", "mixer": {"left": {**left, "rot": {"base": 500.0, "dims": 16}}, "right": {"heads": 1, "dim": 8, "decay_rank": 2}}, "mlp": None},
        ],
    })  # fmt: skip


def built(raw=None):
    return DecoderModel(architecture_for("Vufadra").build_spec(VufadraConfig.from_dict(raw or raw_config())))


def test_config_round_trip_and_registry(tmp_path):
    cfg = VufadraConfig.from_dict(raw_config())
    assert VufadraConfig.from_dict(cfg.to_dict()) == cfg and cfg.to_dict() == raw_config()
    assert cfg.layers[1].mixer.left.chunk == 11 and cfg.layers[1].mixer.left.rot.scaling == (4.0, 64.0, 8.0, 1.0)
    assert cfg.layers[3].mixer.left.rot.scaling is None and cfg.layers[2].ff is None and cfg.bigram.mul_cur == 17
    write_random_model(tmp_path, cfg, seed=1)
    arch, loaded = load_model_config(tmp_path)
    assert arch.name == "Vufadra" and loaded == cfg


def test_the_low_ranks_come_from_the_checkpoint_when_the_config_is_silent(tmp_path):
    cfg = VufadraConfig.from_dict(raw_config())
    write_random_model(tmp_path, cfg, seed=1)
    raw = raw_config()
    for entry in raw["layers"]:
        for sizes in (entry["mixer"], entry["mixer"].get("right", {})):
            sizes.pop("decay_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    _, loaded = load_model_config(tmp_path)
    assert loaded == cfg
    with pytest.raises(ConfigError, match="rank"):
        VufadraConfig.from_dict(raw)


@pytest.mark.parametrize(
    "path,value,message",
    [
        (("layers", 0, "type"), "conv", "not a mixer"),
        (("layers", 0, "mixer", "heads"), 0, "positive"),
        (("layers", 1, "mixer", "left", "heads"), 5, "multiple of kv_heads"),
        (("layers", 1, "mixer", "left", "mask", "size"), 0, "positive"),
        (("layers", 1, "mixer", "left", "rot", "dims"), 18, "dims"),
        (("layers", 1, "mixer", "left", "rot", "dims"), 3, "dims"),
        (("layers", 1, "mixer", "left", "rot", "base"), 1.0, "base"),
        (("layers", 1, "mixer", "left", "rot", "scaling", "fast"), 0, "positive"),
        (("layers", 1, "mixer", "left", "rot", "scaling"), {"factor": 2.0}, "lacks the key"),
        (("layers", 1, "mixer", "right"), None, "lacks the key"),
        (("layers", 2, "mixer", "blocks"), 5, "divide"),
        (("layers", 1, "mlp", "kind"), "moe", "not a feed-forward"),
        (("loop", "stop"), 5, "loop"),
        (("loop", "times"), 0, "loop"),
        (("embedding", "bigram", "buckets"), 0, "positive"),
        (("norm",), None, "lacks the key"),
        (("vocab",), None, "lacks the key"),
    ],
)
def test_config_errors_name_the_key(path, value, message):
    raw = raw_config()
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=message):
        VufadraConfig.from_dict(raw)


def test_declared_tensors():
    spec = architecture_for("Vufadra").build_spec(VufadraConfig.from_dict(raw_config()))
    declared = {s.name: s for s in declared_weights(spec)}
    assert [layer.block for layer in spec.layers] == ["parallel_two_norms", "parallel_two_norms", *["parallel_two_norms_mixer_only"] * 2]
    assert declared["embed"].shape == (90, 48) and declared["bigram"].shape == (54, 48) and declared["head"].alias_of is None
    assert declared["loop.in"].shape == (48, 96) and declared["loop.step"].shape == (3, 48) and declared["loop.step"].role == "vector"
    for name in ("final.norm", "l0.norm1", "l0.norm2", "l3.norm1"):
        assert declared[name].shape == declared[name + ".b"].shape == (48,) and declared[name + ".alpha"].shape == ()
    assert declared["l0.shift"].shape == (48,) and declared["l2.shift"].shape == (48,)
    # a layer without feed-forward: a checkpoint may carry what belongs to one
    assert all(declared["l2." + n].optional for n in ("norm2", "norm2.b", "norm2.alpha")) and "l2.mlp.up" not in declared
    for name in ("r", "k", "v", "g", "a"):
        assert declared[f"l0.mix.{name}"].shape == (48, 48)
    assert declared["l0.mix.a.b"].shape == declared["l0.mix.w0"].shape == declared["l0.mix.norm"].shape == (48,)
    assert declared["l0.mix.w1"].shape == (5, 48) and declared["l0.mix.w2"].shape == (48, 5) and declared["l0.mix.o"].shape == (48, 48)
    left, right = "l1.mix.left.", "l1.mix.right."
    assert declared[left + "q"].shape == (96, 48) and declared[left + "v"].shape == (48, 48) and declared[left + "o"].shape == (48, 144)
    assert declared[left + "q.norm"].shape == declared[left + "k.norm"].shape == (16,) and declared[left + "pb"].shape == (6,)
    assert declared[left + "out"].shape == declared[right + "out"].shape == declared[right + "mu.w"].shape == (48,)
    assert declared[right + "u"].shape == (3, 16) and declared[right + "w1"].shape == (7, 48) and declared[right + "o"].shape == (48, 48)
    assert declared["l2.mix.ra"].shape == (3, 12, 12) and declared["l2.mix.conv"].shape == (36, 4)
    without = {s.name for s in declared_weights(architecture_for("Vufadra").build_spec(VufadraConfig.from_dict({**raw_config(), "loop": None, "embedding": None})))}
    assert not {"bigram", "loop.in", "loop.step"} & without


def test_looped_layers_run_in_place_with_a_junction_in_front_of_every_pass():
    model = built()
    want = [(0, None, 0), (1, 0, 0), (2, None, 0), (1, 0, 1), (2, None, 0), (1, 0, 2), (2, None, 0), (3, None, 0)]
    assert [(e.layer, e.junction, e.turn) for e in model.spec.order] == want
    assert [index for index, _ in plain.passes(raw_config())] == [e.layer for e in model.spec.order]
    assert len(model.junctions) == 1 and model.junctions[0].turns == 3
    assert model.capturable and not model.programmatic_launch
    with pytest.raises(ValueError, match="junction"):
        type(model.spec)(**{**model.spec.__dict__, "order": (OrderEntry(0, junction=1),)})


def test_caches_and_states_of_every_layer_run():
    model = built()
    needs, blocks = model.cache_needs(), model.block_states()
    page = PagedCacheSpec(2, 16, 11, 24, 0, 11)
    one = (page, StateSpec((3 * 16 * 16 + 48,), torch.float32), None)
    assert needs[0] == (None, StateSpec((4 * 12 * 12,), torch.float32), None)
    assert needs[1] == needs[3] == needs[5] == one and needs[7] == (page, StateSpec((8 * 8 + 48,), torch.float32), None)
    assert needs[2] == (None, StateSpec((4, 36), torch.float32), None)
    assert blocks == [StateSpec((48,), torch.float32)] * 8 and model.embedding_state() == StateSpec((1,), torch.int32)
    specs, group_of = plan_groups(needs)
    assert specs == [page] and group_of == [None, 0, None, 0, None, 0, None, 0]
    layout = allocate_cache(needs, 8, 4, 2, torch.float32, "cpu", max_step_tokens=16, block_states=blocks, embedding_state=model.embedding_state())
    assert layout.groups[0].chunk == 11 and len(layout.slot_groups) == 8 + 8 + 1
    for a, b in ((1, 3), (3, 5), (2, 4)):  # every pass has pages and states of its own
        for name in ("state", "block_state", "k", "v"):
            x, y = getattr(layout.views[a], name), getattr(layout.views[b], name)
            assert (x is None) == (y is None) and (x is None or x.data_ptr() != y.data_ptr())


@pytest.mark.parametrize("chunk,page", [(11, 4), (8, 4), (3, 4), (1, 4), (16, 16), (20, 16)])
def test_pages_behind_a_chunk_are_given_back(chunk, page):
    """After every number of computed tokens the pages that the next query's chunk begins in or behind are held, all others are
    free again."""
    manager = CacheManager([GroupSpec("c", window=chunk, num_blocks=32, chunk=chunk)], 32, page, max_num_seqs=1, enable_prefix_caching=False)
    request = manager.new_request()
    for computed in range(1, 70):
        assert manager.try_allocate(request, computed)
        manager.release_behind_window(request, computed)
        table = request.block_tables[0]
        first = computed // chunk * chunk // page
        assert all((entry == NULL_PAGE) == (i < first) for i, entry in enumerate(table))
        manager.check_invariants([request])
    manager.free(request)
    assert manager.pools[0].num_free == 32


def test_attention_options_that_do_not_combine():
    def make(**options):
        return GroupedQueryAttention("", 32, num_heads=4, kv_heads=2, head_dim=16, position_encoding=None, **options)

    assert make(chunk=7).paged_cache() == PagedCacheSpec(2, 16, 7, None, 0, 7)
    assert "weight_bias" in [s.name for s in make(weights="sigmoid").weight_specs()]
    for options in (dict(weights="tanh"), dict(chunk=0), dict(chunk=4, window=4), dict(weights="sigmoid", softmax_sink=True),
                    dict(weights="sigmoid", element_gate=True), dict(weights="sigmoid", qkv_bias=True), dict(chunk=4, talking_heads=True)):  # fmt: skip
        with pytest.raises(ValueError):
            make(**options)


def test_stretched_frequencies():
    """Fast frequencies stay, slow ones are divided, those in between lie between; no stretch at factor 1; the ramp's two ends
    may fall together."""
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 1.0}}
    freq, amplitude = plain.frequencies(rot)
    plain_freq, _ = plain.frequencies({"base": 10000.0, "dims": 64})
    ratio = [a / b for a, b in zip(plain_freq, freq)]
    assert abs(ratio[0] - 1.0) < 1e-12 and abs(ratio[-1] - 8.0) < 1e-9 and sorted(ratio) == ratio and any(1.1 < r < 7.9 for r in ratio)
    assert abs(amplitude - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    for scaling in (rot["scaling"], {"factor": 3.0, "original": 40, "fast": 2.0, "slow": 2.0}, {"factor": 1.0, "original": 64, "fast": 3.0, "slow": 1.0}):
        rope = RotaryEncoding("", 0, head_dim=64, theta=10000.0, yarn=scaling, double_angles=True)
        want, factor = plain.frequencies({**rot, "scaling": scaling})
        assert torch.equal(rope.inv_freq(), torch.tensor(want, dtype=torch.float64)) and rope.amplitude == factor
    with pytest.raises(ValueError, match="one scaling"):
        RotaryEncoding("", 0, head_dim=8, theta=10.0, yarn=rot["scaling"], wavelength_scaling={"factor": 2, "low": 1, "high": 2, "original": 8})


def test_plain_removal_takes_out_what_the_key_reads():
    """With rates of one and no decay a unit key's old value is replaced; with rates of zero values add up under their keys."""
    k = torch.eye(3, dtype=torch.float64)[[0, 1, 0]].unsqueeze(1)
    v = torch.randn(3, 1, 5, dtype=torch.float64)
    one = torch.ones(3, 1, 3, dtype=torch.float64)
    out, state = plain.removal_recurrence(k, k, v, one, one)
    assert torch.allclose(out, v, atol=1e-5) and torch.allclose(state[0, :2], v[[2, 1], 0], atol=1e-5)
    _, added = plain.removal_recurrence(k, k, v, one, 0 * one)
    assert torch.allclose(added[0, 0], v[0, 0] + v[2, 0])


def test_plain_bonus_recurrence_equals_the_sum_over_earlier_tokens():
    torch.manual_seed(0)
    r, k, v = (torch.randn(6, 2, n, dtype=torch.float64) for n in (4, 4, 3))
    decay, bonus = torch.rand(6, 2, 4, dtype=torch.float64), torch.randn(2, 4, dtype=torch.float64)
    got, _ = plain.bonus_recurrence(r, k, v, decay, bonus)
    for t in range(6):
        for h in range(2):
            want = (r[t, h] * bonus[h] * k[t, h]).sum() * v[t, h]
            for j in range(t):
                want = want + (r[t, h] * decay[j + 1 : t, h].prod(0) * k[j, h]).sum() * v[j, h]
            assert torch.allclose(got[t, h], want)


def test_plain_mix_and_chunks():
    h = torch.arange(6, dtype=torch.float64).view(3, 2) + 1.0
    assert torch.equal(plain.mix_previous(h, torch.tensor([0.0, 1.0])), torch.tensor([[1.0, 0.0], [3.0, 2.0], [5.0, 4.0]], dtype=torch.float64))
    seen = plain.chunk_mask(7, 3)
    assert seen[2].tolist() == [True] * 3 + [False] * 4 and seen[3].tolist() == [False] * 3 + [True] + [False] * 3 and bool(seen[5, 3]) and not bool(seen[5, 2])
