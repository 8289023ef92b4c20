"""The Vufadra design through the framework against the plain implementation of ``plain_vufadra.py``: whole prompts against
portions and token-by-token decoding, mixed batches with pages and state slots that are used again, long decoding, several
sizes, looped layers, and greedy generation through the engine's entry point."""

from __future__ import annotations

import dataclasses
import json
import random
from pathlib import Path

import pytest
import torch

import plain_vufadra as plain
import schedules
from conftest import note_error

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# Largest |engine - plain| relative to the request's largest |logit|.
TOLERANCE = {"float32": 3e-5, "bfloat16": 6e-2}


def attention(heads, kv_heads, dim, vdim, chunk, scale, base, dims, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}, "rot": rot}


def states(heads, dim, rank):
    return {"heads": heads, "dim": dim, "decay_rank": rank}


def delta(heads, dim, rank, ff):
    return layer("general_delta", states(heads, dim, rank), ff)


def both(left, right, ff):
    return layer("parallel", {"left": left, "right": right}, ff)


def recurrence(width, blocks, conv, ff):
    return layer("rglru", {"width": width, "blocks": blocks, "conv": conv}, ff)


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, eps, layers, bigram=None, loop=None):
    out = {"architecture": "Vufadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if bigram:
        out["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# A head's first outputs are one key's product with the query times its value, and dividing by their root mean square leaves hardly
# more than that product's sign: an eps that is not small keeps such a model's logits from turning with rounding.
#
# All three mixers; heads rotated in part; value heads wider and narrower than key heads; chunks that are no multiple of a page;
# layers without feed-forward; a loop of three passes that ends in front of the last layer.
CONFIG_S = model(90, 48, 0.6, [
    both(attention(6, 2, 16, 24, 21, 0.3, 500.0, 12, (4.0, 64, 8.0, 1.0)), states(3, 16, 5), 40),
    delta(4, 12, 7, 56),
    recurrence(36, 3, 4, None),
    both(attention(2, 2, 24, 8, 34, 0.2, 10000.0, 24), states(1, 40, 3), None),
    delta(2, 40, 3, None),
], bigram=(53, 31, 17), loop=(1, 4, 3))  # fmt: skip
# Widths that the tensor-core products take, heads of 64 and 128; a loop over all layers.
CONFIG_T = model(64, 128, 0.2, [
    both(attention(4, 2, 64, 64, 33, 0.15, 20000.0, 32, (8.0, 128, 32.0, 1.0)), states(2, 64, 16), 96),
    recurrence(128, 2, 3, 64),
    both(attention(2, 1, 128, 128, 70, 0.1, 500.0, 128, (2.0, 32, 4.0, 0.5)), states(4, 32, 8), 64),
    delta(2, 64, 24, 160),
], bigram=(211, 5, 3), loop=(0, 4, 2))  # fmt: skip
# Sizes that no fast path takes: a width that is no multiple of 8, odd head widths, one head, a rotation of two elements, ranks
# of one, one tap, one block and blocks of one channel, chunks of one token; no table of pairs, no loop.
CONFIG_U = model(51, 36, 1e-3, [
    both(attention(1, 1, 11, 6, 1, 0.6, 30.0, 2), states(1, 9, 1), 9),
    recurrence(21, 1, 1, 17),
    delta(3, 5, 1, None),
    both(attention(3, 1, 14, 20, 50, 0.3, 1000.0, 6, (3.0, 20, 2.0, 2.0)), states(3, 7, 2), 12),
    recurrence(10, 10, 6, None),
])  # fmt: skip
CONFIGS = {"S": CONFIG_S, "T": CONFIG_T, "U": CONFIG_U}
LENGTHS = {"S": [70, 45, 133, 9, 97, 33, 1, 2], "T": [150, 64, 17, 81, 49, 130], "U": [40, 3, 77, 18, 1, 60]}


def random_ids(seed, count, vocab):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(count)]


def make_tensors(specs, seed, scale):
    """Random weights with slow and fast decays, token shifts and mixes of every size, sigmoid weights that are small, and
    convolutions that mostly pass the current token."""
    from mini_engine_b200.weights.random_init import random_tensors

    tensors = random_tensors(specs, seed, torch.bfloat16, scale=scale)
    for name, t in tensors.items():
        last = name.rsplit(".", 1)[-1]
        if last == "w0":
            tensors[name] = (torch.linspace(-6.0, 1.0, t.numel()) + t.float()).to(torch.bfloat16)
        elif last == "pb":
            tensors[name] = (t.float() - 2.0).to(torch.bfloat16)
        elif last == "shift" or ".mu." in name:
            tensors[name] = (5.0 * t.float()).to(torch.bfloat16)
        elif name.endswith(".conv"):
            tensors[name][:, -1] += 0.75
            tensors[name][:, :-1] *= 3.0
        elif last == "lam":
            tensors[name] = (torch.linspace(-5.0, 0.5, t.numel()) + t.float()).to(torch.bfloat16)
        elif last == "step":
            tensors[name] = (10.0 * t.float()).to(torch.bfloat16)
        elif last in ("embed", "bigram"):
            tensors[name] = (4.0 * t.float()).to(torch.bfloat16)
    return tensors


def write_model(folder, raw, seed=31):
    """Matrices whose products keep their input's size whatever the width; the ranks are left to the tensors' shapes."""
    from mini_engine_b200.config import VufadraConfig
    from mini_engine_b200.config.registry import architecture_for
    from mini_engine_b200.parts.model import declared_weights
    from mini_engine_b200.weights.safetensors_io import write_safetensors

    specs = declared_weights(architecture_for("Vufadra").build_spec(VufadraConfig.from_dict(raw)))
    silent = json.loads(json.dumps(raw))
    for entry in silent["layers"]:
        for sizes in (entry["mixer"], entry["mixer"].get("right", {})):
            sizes.pop("decay_rank", None)
    (folder / "config.json").write_text(json.dumps(silent))
    write_safetensors(folder / "model.safetensors", make_tensors(specs, seed, 55.0 / raw["width"] ** 0.5))
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(tmp_path_factory.mktemp(f"vufadra_{name}"), raw) for name, raw in CONFIGS.items()}


_loaded: dict = {}


def load_plain(folder):
    from safetensors.torch import load_file

    if folder not in _loaded:
        weights = {k: v.to(torch.float64) for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}
        _loaded[folder] = weights, json.loads((Path(folder) / "config.json").read_text())
    return _loaded[folder]


_expected: dict = {}


def expected_logits(folder, requests):
    weights, config = load_plain(folder)
    out = {}
    for name, toks in requests.items():
        key = (folder, tuple(toks))
        if key not in _expected:
            _expected[key] = plain.forward(config, weights, toks).float()
        out[name] = _expected[key]
    return out


def replay(folder, dtype_name, steps, block_size=16, max_tokens=None, max_live=4, max_step_tokens=512):
    from mini_engine_b200.engine.replay import Replayer

    replayer = Replayer(folder, DTYPES[dtype_name], max_tokens or schedules.peak_live_tokens(steps), block_size,
                        max_step_tokens=max_step_tokens, max_live=max_live)  # fmt: skip
    outputs = {}
    for record in steps:
        logits = replayer.step(record)
        if logits is not None:
            outputs[record["step"]] = logits.clone()
    replayer.manager.check_invariants([])
    assert all(pool.num_free == pool.num_pages for pool in replayer.manager.pools), "pages were lost"
    return schedules.collect(steps, outputs)


def compare(got, expected, requests, dtype_name):
    worst = 0.0
    for name, toks in requests.items():
        assert sorted(got[name]) == list(range(len(toks))), f"{name}: positions missing"
        scale = float(expected[name].abs().max())
        for position, row in got[name].items():
            error = float((row - expected[name][position]).abs().max()) / scale
            worst = max(worst, error)
            assert error <= TOLERANCE[dtype_name], f"{name} position {position}: relative error {error:.3g}"
    note_error("vufadra " + dtype_name, worst)


def replay_and_compare(folder, dtype_name, steps, requests, **options):
    compare(replay(folder, dtype_name, steps, **options), expected_logits(folder, requests), requests, dtype_name)


def requests_for(name):
    return {f"r{i}": random_ids(500 + i, n, CONFIGS[name]["vocab"]) for i, n in enumerate(LENGTHS[name])}


# --------------------------------------------------------------- whole models, every way of cutting


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["S", "T", "U"])
@pytest.mark.parametrize("schedule", ["whole", "tail_one_by_one", "changing_portions", "mixed"])
def test_schedules_match_plain(name, dtype_name, schedule, folders):
    """Whole prompts (requests of one and two tokens among them); the last 32 tokens one by one; portions down to two
    tokens; up to four live requests whose pages and state slots are handed out again."""
    requests = requests_for(name)
    replay_and_compare(folders[name], dtype_name, getattr(schedules, schedule)(requests), requests)


@pytest.mark.parametrize("what", ["shift", "loop.step", "bigram", "pb", "decay", "order", "pass", "chunk"])
def test_the_test_weights_show_every_mechanism(folders, what):
    """The plain implementation with one mechanism changed is far from itself: what the comparisons above would not see is
    not there."""
    weights, config = load_plain(folders["S"])
    toks = requests_for("S")["r2"]
    want = plain.forward(config, weights, toks)
    changed, other = dict(weights), json.loads(json.dumps(config))
    if what == "shift":
        changed["l1.shift"] = torch.zeros_like(weights["l1.shift"])
    elif what == "loop.step":
        changed["loop.step"] = weights["loop.step"].flip(0)
    elif what == "bigram":
        other["embedding"]["bigram"]["mul_prev"] += 1
    elif what == "pb":
        changed["l0.mix.left.pb"] = weights["l0.mix.left.pb"].roll(1)
    elif what == "decay":
        changed["l1.mix.w0"] = weights["l1.mix.w0"] + 0.5
    elif what == "order":
        changed["loop.in"] = weights["loop.in"].roll(48, dims=1)
    elif what == "pass":
        other["loop"]["times"] = 2
    elif what == "chunk":
        other["layers"][0]["mixer"]["left"]["mask"]["size"] += 1
    assert float((plain.forward(other, changed, toks) - want).abs().max()) > 2 * TOLERANCE["bfloat16"] * float(want.abs().max()) * (0.1 if what in ("chunk", "pb") else 1)


@pytest.mark.parametrize("block_size", [4, 16, 32])
def test_float32_hardly_depends_on_the_cut_or_the_batch(folders, block_size):
    """In float32 every kernel's sums for a token depend on that token's position alone, except that the matrix states run long
    portions in chunks, whose sums are ordered by a token's place in its portion: portions, single tokens, mixed batches and
    other page sizes give the whole prompt's logits up to rounding."""
    requests = {name: toks for name, toks in list(requests_for("S").items())[:5]}
    whole = replay(folders["S"], "float32", schedules.whole(requests), block_size)
    for maker in (schedules.changing_portions, schedules.mixed, lambda r: schedules.tail_one_by_one(r, 40)):
        cut = replay(folders["S"], "float32", maker(requests), block_size)
        for name, toks in requests.items():
            for position in range(len(toks)):
                a, b = whole[name][position], cut[name][position]
                assert float((a - b).abs().max()) <= 5e-6 * float(a.abs().max()), f"{name} position {position}"


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_long_steps_of_many_tokens(folders, dtype_name):
    """A prompt long enough for runs of tokens per thread and unsplit products, then a batch that brings two long portions side
    by side and decoded tokens."""
    toks = {name: random_ids(60 + i, n, CONFIG_T["vocab"]) for i, (name, n) in enumerate((("a", 1150), ("b", 300), ("c", 290), ("d", 40)))}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:1140], "want": list(range(1140))}], "end": []}]
    steps.append({"step": 1, "entries": [{"id": "a", "tokens": toks["a"][1140:1141], "want": [0]}, {"id": "d", "tokens": toks["d"][:30], "want": list(range(30))}], "end": []})
    entries = [{"id": "b", "tokens": toks["b"], "want": list(range(300))}, {"id": "d", "tokens": toks["d"][30:31], "want": [0]},
               {"id": "c", "tokens": toks["c"], "want": list(range(290))}, {"id": "a", "tokens": toks["a"][1141:1142], "want": [0]}]  # fmt: skip
    steps.append({"step": 2, "entries": entries, "end": ["b", "c"]})
    rest = [{"id": "a", "tokens": toks["a"][1142:], "want": list(range(8))}, {"id": "d", "tokens": toks["d"][31:], "want": list(range(9))}]
    steps.append({"step": 3, "entries": rest, "end": ["a", "d"]})
    replay_and_compare(folders["T"], dtype_name, steps, toks, max_step_tokens=1200)


def test_long_decoding(folders):
    """Three prompt tokens, then 200 tokens one by one: states and last inputs are carried through 200 steps, chunks end under
    decoded tokens and give their pages back."""
    for name in ("S", "T"):
        requests = {"long": random_ids(77, 203, CONFIGS[name]["vocab"])}
        steps = schedules.tail_one_by_one(requests, tail=200)
        for dtype_name in ("float32", "bfloat16"):
            replay_and_compare(folders[name], dtype_name, steps, requests)


def test_pages_and_slots_that_are_used_again_hold_nothing_of_their_past(folders):
    """A pool of four pages and one state slot: the second request gets the first one's pages and its slot, and must see
    neither the keys nor the states nor the last inputs and tokens that they held."""
    from mini_engine_b200.engine.replay import Replayer

    a, b = random_ids(5, 60, CONFIG_S["vocab"]), random_ids(6, 37, CONFIG_S["vocab"])
    replayer = Replayer(folders["S"], torch.float32, 64, 16, max_live=1)
    first = replayer.step({"step": 0, "entries": [{"id": "a", "tokens": a, "want": [59]}], "end": ["a"]})
    assert replayer.step({"step": 1, "entries": [{"id": "b", "tokens": b[:1], "want": []}], "end": []}) is None
    second = replayer.step({"step": 2, "entries": [{"id": "b", "tokens": b[1:], "want": [35]}], "end": ["b"]})
    alone = Replayer(folders["S"], torch.float32, 64, 16).step({"step": 0, "entries": [{"id": "b", "tokens": b, "want": [36]}], "end": ["b"]})
    assert torch.allclose(second, alone, atol=1e-5 * float(alone.abs().max())) and not torch.allclose(first, alone, atol=1e-2)


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_the_replay_program_itself(folders, dtype_name, tmp_path):
    """`bin/trace_run` as a process on a model folder of this design: mixed steps in, `done` lines and logit files out."""
    import subprocess
    import sys

    import numpy as np
    from conftest import ROOT

    requests = requests_for("U")
    steps = schedules.mixed(requests)
    out = tmp_path / "out"
    feed = "".join(json.dumps(record) + "\n" for record in steps)
    proc = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folders["U"]), "--dtype", dtype_name,
         "--out", str(out), "--max-tokens", str(schedules.peak_live_tokens(steps))],
        input=feed, capture_output=True, text=True, timeout=900,
    )  # fmt: skip
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [line for line in proc.stdout.splitlines() if line.startswith("done ")] == [f"done {s['step']}" for s in steps]
    outputs = {}
    for record in steps:
        wanted = sum(len(e.get("want", [])) for e in record["entries"])
        if wanted:
            data = np.fromfile(out / f"{record['step']}.f32", dtype="<f4")
            outputs[record["step"]] = torch.from_numpy(data.reshape(wanted, CONFIG_U["vocab"]).copy())
    compare(schedules.collect(steps, outputs), expected_logits(folders["U"], requests), requests, dtype_name)


@pytest.mark.parametrize("name", ["S", "U"])
def test_the_stream_after_every_layer(folders, name):
    """The residual stream behind each layer run, with what is still pending, against the plain layers, in float32."""
    from mini_engine_b200.engine.replay import Replayer
    from mini_engine_b200.parts import block as block_module

    weights, config = load_plain(folders[name])
    toks = random_ids(9, 50, config["vocab"])
    _, want = plain.forward(config, weights, toks, return_layers=True)
    seen = []
    original = block_module.TwoNormParallelBlock.forward

    def recording(self, state, ctx, cache):
        original(self, state, ctx, cache)
        pending = [p.sum(0) for p in (state.pending, state.pending_more) if p is not None]
        seen.append(sum(pending, state.x.clone()))

    block_module.TwoNormParallelBlock.forward = recording
    try:
        Replayer(folders[name], torch.float32, 64).step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    finally:
        block_module.TwoNormParallelBlock.forward = original
    assert len(seen) == len(plain.passes(config))
    for index, got in enumerate(seen):
        assert torch.allclose(got.cpu(), want[index].float(), atol=2e-5 * float(want[index].abs().max())), f"layer run {index}"


@pytest.mark.parametrize("kind", ["general_delta", "parallel", "rglru"])
def test_a_model_of_one_mixer(kind, tmp_path):
    """Each mixer as the only one of a model (caches without page groups among them), long enough for its chunks or its
    memory, the second layer in a loop."""
    one = {"general_delta": delta(2, 32, 8, 32), "parallel": both(attention(4, 2, 64, 64, 40, 0.2, 3000.0, 64), states(2, 32, 8), 32),
           "rglru": recurrence(64, 4, 4, 32)}[kind]  # fmt: skip
    folder = write_model(tmp_path, model(100, 64, 0.02, [one, one], loop=(1, 2, 2)), seed=5)
    requests = {"a": random_ids(1, 300, 100), "b": random_ids(2, 2, 100)}
    for dtype_name in ("float32", "bfloat16"):
        for maker in (schedules.whole, schedules.changing_portions, lambda r: schedules.tail_one_by_one(r, 32)):
            replay_and_compare(folder, dtype_name, maker(requests), requests)


def test_states_in_slots_of_an_odd_length(tmp_path):
    """Time mixing keeps its last input behind its matrix states: with a width of 54 the slots of heads that the chunks would
    take start on no 16 bytes, and long portions walk token by token."""
    raw = model(80, 54, 0.1, [both(attention(2, 1, 32, 32, 50, 0.2, 3000.0, 16), states(2, 32, 6), 40), delta(2, 32, 6, None)], bigram=(40, 9, 4))
    folder = write_model(tmp_path, raw, seed=8)
    requests = {"a": random_ids(3, 160, 80), "b": random_ids(4, 47, 80), "c": random_ids(5, 1, 80)}
    for dtype_name in ("float32", "bfloat16"):
        for maker in (schedules.whole, schedules.changing_portions, schedules.mixed):
            replay_and_compare(folder, dtype_name, maker(requests), requests)


def test_the_block_with_another_norm(monkeypatch):
    """The arrangement with layer norms in the place of dynamic tanh: three kernels in the place of one, the same layer."""
    from mini_engine_b200.cache.manager import CacheManager
    from mini_engine_b200.config import VufadraConfig
    from mini_engine_b200.config.model_spec import PartSpec
    from mini_engine_b200.engine.batch import StepEntry
    from mini_engine_b200.engine.runner import ModelRunner
    from mini_engine_b200.models.vufadra import vufadra_spec
    from mini_engine_b200.parts.model import DecoderModel
    from mini_engine_b200.weights.loader import place_tensors

    raw = {**CONFIG_S, "loop": None}
    spec = vufadra_spec(VufadraConfig.from_dict(raw))
    to_layernorm = lambda norm: PartSpec("layernorm", {**norm.params, "eps": 1e-3})  # noqa: E731
    spec = dataclasses.replace(
        spec, final_norm=to_layernorm(spec.final_norm),
        layers=tuple(dataclasses.replace(l, norms={k: to_layernorm(n) for k, n in l.norms.items()}) for l in spec.layers),
    )  # fmt: skip
    built = DecoderModel(spec)
    specs = built.weight_specs()
    tensors = make_tensors(specs, 3, 8.0)
    built.load(place_tensors(tensors, specs, torch.float32, "cuda"))
    runner = ModelRunner(built, dtype=torch.float32, num_blocks=16, block_size=16, max_num_seqs=2, max_num_batched_tokens=64, max_model_len=128)
    manager = CacheManager(runner.layout.groups, 16, 16, max_num_seqs=2, enable_prefix_caching=False, slot_groups=runner.layout.slot_groups)
    toks, cache, got, done = random_ids(4, 60, raw["vocab"]), manager.new_request(), [], 0
    for count in (37, 2, 1, 20):
        assert manager.try_allocate(cache, done + count)
        got.append(runner.execute([StepEntry(cache, done, toks[done : done + count], tuple(range(count)))]).cpu().clone())
        done += count

    def layer_norm(x, w, name):
        centred = x - x.mean(-1, keepdim=True)
        return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + 1e-3) * w[name] + w[name + ".b"]

    monkeypatch.setattr(plain, "dynamic_tanh", layer_norm)
    want = plain.forward(raw, {k: v.double() for k, v in tensors.items()}, toks).float()
    assert float((torch.cat(got) - want).abs().max()) <= TOLERANCE["float32"] * float(want.abs().max())


# ------------------------------------------------------------- the engine's entry point, scheduler and command line


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["S", "T"])
def test_greedy_generation_through_the_engine(folders, dtype_name, name):
    """`LLMEngine.generate`: the scheduler, portions under a 48-token budget, captured decode steps.  Every generated
    token is checked teacher-forced: its plain logit lies within the tolerance of the largest one at its position."""
    from mini_engine_b200 import EngineConfig, LLMEngine, SamplingParams

    folder = folders[name]
    weights, config = load_plain(folder)
    prompts = [random_ids(40 + i, n, config["vocab"]) for i, n in enumerate((19, 70, 3, 41, 100))]
    engine = LLMEngine.from_pretrained(
        folder, EngineConfig(block_size=16, num_blocks=64, max_model_len=256, max_num_seqs=3, max_num_batched_tokens=48,
                             dtype=DTYPES[dtype_name])  # fmt: skip
    )
    got = engine.generate(prompts, SamplingParams(max_tokens=24, ignore_eos=True))
    assert engine.stats.graph_steps > 0
    for prompt, tokens in zip(prompts, got):
        assert len(tokens) == 24
        logits = plain.forward(config, weights, (prompt + tokens)[:-1]).float()
        slack = 2 * TOLERANCE[dtype_name] * float(logits.abs().max())
        for i, token in enumerate(tokens):
            row = logits[len(prompt) - 1 + i]
            assert float(row.max() - row[token]) <= slack, f"token {i} of a {len(prompt)}-token prompt"
    again = engine.generate(prompts[:2], SamplingParams(max_tokens=24, ignore_eos=True))
    assert len(again) == 2 and all(len(tokens) == 24 for tokens in again)
    if dtype_name == "float32":  # slots and pages of finished requests serve new ones: the same tokens bit for bit
        assert again == got[:2]


def test_the_command_line(folders, capsys):
    """`python -m mini_engine_b200.cli.generate` on a folder of this design: greedy output equals the engine's, and a
    run with temperature draws tokens of the vocabulary through the device sampler."""
    from mini_engine_b200 import EngineConfig, LLMEngine, SamplingParams
    from mini_engine_b200.cli import generate

    folder = str(folders["S"])
    prompts = [random_ids(70 + i, n, CONFIG_S["vocab"]) for i, n in enumerate((12, 30))]
    ids = ";".join(",".join(map(str, p)) for p in prompts)
    common = ["--model", folder, "--dtype", "fp32", "--max-tokens", "6", "--ignore-eos", "--num-blocks", "32", "--max-model-len", "128",
              "--max-num-seqs", "2", "--prompt-ids", ids]  # fmt: skip
    assert generate.main(common) == 0
    greedy = capsys.readouterr().out
    engine = LLMEngine.from_pretrained(folder, EngineConfig(block_size=16, num_blocks=32, max_model_len=128, max_num_seqs=2, dtype=torch.float32))
    want = engine.generate(prompts, SamplingParams(max_tokens=6, ignore_eos=True))
    for prompt, tokens in zip(prompts, want):
        assert f"prompt ({len(prompt)} tokens) -> {tokens}" in greedy
    assert generate.main(common + ["--temperature", "0.8", "--seed", "3"]) == 0
    drawn = capsys.readouterr().out.splitlines()[:2]
    for line, prompt in zip(drawn, prompts):
        tokens = json.loads(line.split("-> ")[1])
        assert line.startswith(f"prompt ({len(prompt)} tokens)") and len(tokens) == 6 and all(0 <= t < CONFIG_S["vocab"] for t in tokens)


def test_preempted_requests_are_computed_again(tmp_path):
    """A pool so small that running requests are preempted: their pages and states go back, they are computed again, and
    the tokens are those of a run with room for everyone."""
    from mini_engine_b200 import EngineConfig, LLMEngine, SamplingParams

    raw = {**CONFIG_T, "layers": [both(attention(4, 2, 64, 64, 200, 0.1, 20000.0, 32), states(2, 32, 4), 64), *CONFIG_T["layers"][1:3]], "loop": None}
    folder = write_model(tmp_path, raw)
    prompts = [random_ids(90 + i, n, CONFIG_T["vocab"]) for i, n in enumerate((40, 33, 25, 47))]
    params = SamplingParams(max_tokens=30, ignore_eos=True)
    roomy = LLMEngine.from_pretrained(folder, EngineConfig(block_size=16, num_blocks=64, max_model_len=128, max_num_seqs=4, dtype=torch.float32))
    want = roomy.generate(prompts, params)
    tight = LLMEngine.from_pretrained(folder, EngineConfig(block_size=16, num_blocks=11, max_model_len=128, max_num_seqs=4, dtype=torch.float32))
    got = tight.generate(prompts, params)
    assert tight.scheduler.num_preemptions > 0
    assert got == want
