"""The Tobadra design through the framework against the plain implementation of ``plain_tobadra.py``: whole prompts against
portions and token-by-token decoding, mixed batches with pages and state slots that are used again, long decoding, several
sizes, layers that use another layer's tensors, and greedy generation through the engine's entry point."""

from __future__ import annotations

import json
import random
from pathlib import Path

import pytest
import torch

import plain_tobadra as plain
import schedules
from conftest import note_error

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# Largest |engine - plain| relative to the request's largest |logit|.
TOLERANCE = {"float32": 3e-5, "bfloat16": 6e-2}
# A router's choice that was won by less than this (in choice score) may fall the other way when activations are rounded
# to bfloat16, and everything behind it follows the other choice.  In bfloat16 the plain implementation is therefore told
# what the engine chose and takes that where its own decision was this close (a differing choice on a clear decision fails
# the comparison); float32 is compared without any of this.
CLOSE_CALL = 0.05


def attention(heads, kv_heads, dim, vdim, window, scale, base, dims):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": window}, "rot": {"base": base, "dims": dims}}}  # fmt: skip


def lightning(heads, dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": decay_rank, "gate_rank": gate_rank}}  # fmt: skip


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, identity=None, groups=None, shared=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if identity:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp, weights_of=None):
    out = {**mixer, "mlp": mlp}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


# All three mixers and every kind of feed-forward; heads rotated in part; value heads wider and narrower than key heads;
# a window that is no multiple of a page and one of two tokens; a decay of one; four taps here, three in the layers;
# layers that use another one's tensors, one of them behind it, one in front of it.
ROUTED = moe(6, 3, 16, 1.7, identity=2, groups=(4, 2), shared=24)
DELTA = delta(4, 2, 16, 24, 3, 5, 7)
CONFIG_S = {
    "architecture": "Tobadra", "vocab": 90, "width": 48, "norm": {"eps": 2e-5}, "canon": {"taps": 4}, "logit_scale": 0.7,
    "layers": [
        layer(DELTA, ROUTED, weights_of=3),
        layer(attention(6, 2, 16, 24, 21, 0.3, 500.0, 12), dense(40)),
        layer(lightning(3, 16, 24, [0.9, 0.99, 1.0]), None),
        layer(DELTA, ROUTED),
        layer(attention(2, 2, 24, 8, 2, 0.2, 10000.0, 24), moe(4, 1, 24, 1.0)),
        layer(lightning(1, 24, 8, [0.95]), moe(5, 2, 8, 0.5, identity=1)),
        layer(attention(6, 2, 16, 24, 21, 0.3, 500.0, 12), dense(40), weights_of=1),
    ],
}  # fmt: skip
# Widths that the tensor-core products take, heads of 64 and 128, units enough for the sorted form at few tokens.
CONFIG_T = {
    "architecture": "Tobadra", "vocab": 64, "width": 128, "norm": {"eps": 1e-5}, "canon": {"taps": 2}, "logit_scale": 2.0,
    "layers": [
        layer(attention(4, 2, 64, 64, 33, 0.1, 20000.0, 32), moe(12, 2, 32, 1.5, identity=6, groups=(6, 3), shared=64)),
        layer(delta(2, 2, 64, 32, 4, 16, 8), dense(96)),
        layer(lightning(2, 64, 64, [0.96875, 0.998]), moe(8, 3, 64, 2.0, shared=32)),
        layer(attention(2, 1, 128, 128, 70, 0.08, 500.0, 128), dense(64)),
        layer(delta(2, 1, 128, 64, 2, 8, 24), moe(9, 2, 16, 1.0, identity=3, groups=(3, 1))),
    ],
}  # fmt: skip
# Sizes that no fast path takes: a width that is no multiple of 8, odd head widths, one head, one unit, as many choices
# as units, a rotation of two elements, ranks of one, one tap, a window of one token.
CONFIG_U = {
    "architecture": "Tobadra", "vocab": 51, "width": 36, "norm": {"eps": 1e-4}, "canon": {"taps": 1}, "logit_scale": 1.0,
    "layers": [
        layer(attention(1, 1, 10, 6, 1, 0.6, 30.0, 2), moe(1, 1, 9, 1.0)),
        layer(delta(3, 1, 5, 7, 1, 1, 3), dense(17)),
        layer(lightning(3, 6, 5, [0.5, 0.75, 0.999]), moe(3, 4, 7, 0.8, identity=1, shared=5)),
        layer(delta(1, 1, 9, 6, 6, 2, 1), None),
        layer(attention(3, 1, 14, 20, 50, 0.3, 1000.0, 6), None),
    ],
}  # fmt: skip
CONFIGS = {"S": CONFIG_S, "T": CONFIG_T, "U": CONFIG_U}
LENGTHS = {"S": [70, 45, 133, 9, 97, 33, 1, 2], "T": [150, 64, 17, 81, 49, 130], "U": [40, 3, 77, 18, 1, 60]}


def random_ids(seed, count, vocab):
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(count)]


def write_model(folder, raw, seed=31, scale=8.0):
    """Random weights with decays of the delta rule from fast to almost none and convolutions that mostly pass the current
    token; the ranks are left to the tensors' shapes."""
    from mini_engine_b200.config import TobadraConfig
    from mini_engine_b200.config.registry import architecture_for
    from mini_engine_b200.parts.model import declared_weights
    from mini_engine_b200.weights.random_init import random_tensors
    from mini_engine_b200.weights.safetensors_io import write_safetensors

    specs = declared_weights(architecture_for("Tobadra").build_spec(TobadraConfig.from_dict(raw)))
    tensors = random_tensors(specs, seed, torch.bfloat16, scale=scale)
    for name, t in tensors.items():
        if name.endswith("A_log"):
            tensors[name] = (torch.linspace(0.0, -6.0, t.shape[0]) + t.float()).to(torch.bfloat16)
        elif name.endswith(".conv"):
            tensors[name][:, -1] += 0.75
            tensors[name][:, :-1] *= 3.0
        elif name.endswith("canon1"):
            tensors[name] *= 3.0
    silent = json.loads(json.dumps(raw))
    for entry in silent["layers"]:
        entry["mixer"].pop("decay_rank", None), entry["mixer"].pop("gate_rank", None)
    (folder / "config.json").write_text(json.dumps(silent))
    write_safetensors(folder / "model.safetensors", tensors)
    return folder


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_model(tmp_path_factory.mktemp(f"tobadra_{name}"), raw) for name, raw in CONFIGS.items()}


_loaded: dict = {}


def load_plain(folder):
    from safetensors.torch import load_file

    if folder not in _loaded:
        weights = {k: v.to(torch.float64) for k, v in load_file(str(Path(folder) / "model.safetensors")).items()}
        _loaded[folder] = weights, json.loads((Path(folder) / "config.json").read_text())
    return _loaded[folder]


def routed_layers(config):
    return [i for i, entry in enumerate(config["layers"]) if (entry.get("mlp") or {}).get("kind") == "moe"]


def expected_logits(folder, requests, routing=None):
    """Plain logits per request.  ``routing`` (request -> layer -> [T, top]) is the engine's choice, followed where the
    plain decision was a close call."""
    weights, config = load_plain(folder)
    out = {}
    for name, toks in requests.items():
        follow = None if routing is None else routing.get(name)
        out[name] = plain.forward(config, weights, toks, follow=follow, close=CLOSE_CALL).float()
    return out


def replay(folder, dtype_name, steps, block_size=16, max_tokens=None, max_live=4, max_step_tokens=512, routing=None):
    """``routing`` (a dict) is filled with what the routed feed-forwards chose: request -> layer -> [T, top]."""
    from mini_engine_b200.csrc import ops
    from mini_engine_b200.engine.replay import Replayer

    replayer = Replayer(folder, DTYPES[dtype_name], max_tokens or schedules.peak_live_tokens(steps), block_size,
                        max_step_tokens=max_step_tokens, max_live=max_live)  # fmt: skip
    layers = routed_layers(json.loads((Path(folder) / "config.json").read_text()))
    calls: list = []
    original = ops.route

    def recording(**kwargs):
        original(**kwargs)
        calls.append(kwargs["chosen"].clone())

    outputs = {}
    ops.route = recording
    try:
        for record in steps:
            calls.clear()
            logits = replayer.step(record)
            if logits is not None:
                outputs[record["step"]] = logits.clone()
            if routing is not None and record["entries"]:
                assert len(calls) == len(layers)
                first = 0
                for item in record["entries"]:
                    count = len(item["tokens"])
                    for index, chosen in zip(layers, calls):
                        routing.setdefault(item["id"], {}).setdefault(index, []).append(chosen[first : first + count].cpu().long())
                    first += count
    finally:
        ops.route = original
    if routing is not None:
        for held in routing.values():
            for index in held:
                held[index] = torch.cat(held[index])
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
    note_error("tobadra " + dtype_name, worst)


def replay_and_compare(folder, dtype_name, steps, requests, **options):
    routing = {} if dtype_name == "bfloat16" else None
    got = replay(folder, dtype_name, steps, routing=routing, **options)
    compare(got, expected_logits(folder, requests, routing), requests, dtype_name)


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


@pytest.mark.parametrize("block_size", [4, 16, 32])
def test_float32_hardly_depends_on_the_cut_or_the_batch(folders, block_size, monkeypatch):
    """In float32 every kernel's sums for a token depend on that token's position alone, except that lightning attention
    runs long portions in chunks whose sums are ordered by the chunk's place in the portion: portions, single tokens, mixed
    batches and other page sizes give the whole prompt's logits up to that rounding, and its very bits when every portion
    walks token by token."""
    from mini_engine_b200.parts import linear_attention

    requests = {name: toks for name, toks in list(requests_for("S").items())[:5]}
    for chunked in (True, False):
        if not chunked:
            monkeypatch.setattr(linear_attention, "CHUNKED_MIN_TOKENS", 1 << 30)
        whole = replay(folders["S"], "float32", schedules.whole(requests), block_size)
        for maker in (schedules.changing_portions, schedules.mixed, lambda r: schedules.tail_one_by_one(r, 40)):
            cut = replay(folders["S"], "float32", maker(requests), block_size)
            for name, toks in requests.items():
                for position in range(len(toks)):
                    a, b = whole[name][position], cut[name][position]
                    if chunked:
                        assert float((a - b).abs().max()) <= 1e-5 * float(a.abs().max()), f"{name} position {position}"
                    else:
                        assert torch.equal(a, b), f"{name} position {position}"


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_long_steps_of_many_tokens(folders, dtype_name):
    """A prompt long enough for rows sorted by unit, chunked lightning attention and products with the activation in
    their epilogue, then a batch that brings two long portions side by side and decoded tokens."""
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
    """Three prompt tokens, then 200 tokens one by one: the states and the convolutions' pasts are carried through 200 steps,
    windows pass over decoded tokens and give their pages back."""
    for name in ("S", "T"):
        requests = {"long": random_ids(77, 203, CONFIGS[name]["vocab"])}
        steps = schedules.tail_one_by_one(requests, tail=200)
        for dtype_name in ("float32", "bfloat16"):
            replay_and_compare(folders[name], dtype_name, steps, requests)


def test_pages_and_slots_that_are_used_again_hold_nothing_of_their_past(folders):
    """A pool of four pages and one state slot: the second request gets the first one's pages and its slot, and must see
    neither the keys nor the states nor the convolutions' pasts that they held."""
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
    got = schedules.collect(steps, outputs)
    if dtype_name == "float32":
        compare(got, expected_logits(folders["U"], requests), requests, dtype_name)
    else:  # the process keeps its routing to itself: against the same steps in this process, bit for bit
        here = replay(folders["U"], dtype_name, steps)
        for name, toks in requests.items():
            for position in range(len(toks)):
                assert torch.equal(got[name][position], here[name][position])


def test_the_stream_after_every_layer(folders):
    """The residual stream behind each layer, with the gated and normed output that it is still owed, against the plain
    layers, in float32."""
    from mini_engine_b200.csrc import ops
    from mini_engine_b200.engine.replay import Replayer
    from mini_engine_b200.parts import block as block_module

    weights, config = load_plain(folders["S"])
    toks = random_ids(9, 50, config["vocab"])
    _, want = plain.forward(config, weights, toks, return_layers=True)
    seen = []
    original = block_module.GatedSandwichBlock.forward

    def recording(self, state, ctx, cache):
        original(self, state, ctx, cache)
        x, (weight, eps) = state.x.clone(), state.pending_norm
        ops.sandwich_norm(x=x, pending=state.pending, bias=state.pending_bias, gate=state.pending_gate, gate_bias=state.pending_gate_bias,
                          out_weight=weight, out_eps=eps, weight=weight, eps=eps, out=torch.empty_like(x))  # fmt: skip
        seen.append(x)

    block_module.GatedSandwichBlock.forward = recording
    try:
        Replayer(folders["S"], torch.float32, 64).step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": []}], "end": ["a"]})
    finally:
        block_module.GatedSandwichBlock.forward = original
    assert len(seen) == len(config["layers"])
    for index, got in enumerate(seen):
        assert torch.allclose(got.cpu(), want[index].float(), atol=2e-5 * float(want[index].abs().max())), f"layer {index}"


@pytest.mark.parametrize("kind", ["attention", "lightning", "channel_delta"])
def test_a_model_of_one_mixer(kind, tmp_path):
    """Each mixer as the only one of a model (a cache without page groups among them), long enough for its window or its
    memory, with the tensors used twice."""
    mixers = {"attention": attention(4, 2, 64, 64, 40, 0.15, 3000.0, 64), "lightning": lightning(2, 32, 16, [0.99, 0.8]),
              "channel_delta": delta(2, 1, 32, 16, 4, 8, 8)}  # fmt: skip
    raw = {"architecture": "Tobadra", "vocab": 100, "width": 64, "norm": {"eps": 1e-5}, "canon": {"taps": 3}, "logit_scale": 1.5,
           "layers": [layer(mixers[kind], dense(32)), layer(mixers[kind], dense(32), weights_of=0)]}  # fmt: skip
    folder = write_model(tmp_path, raw, seed=5, scale=12.0)
    requests = {"a": random_ids(1, 300, 100), "b": random_ids(2, 2, 100)}
    for dtype_name in ("float32", "bfloat16"):
        for maker in (schedules.whole, schedules.changing_portions, lambda r: schedules.tail_one_by_one(r, 32)):
            replay_and_compare(folder, dtype_name, maker(requests), requests)


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
        if dtype_name == "bfloat16":
            continue  # a routing decision that rounding turns makes another sequence: float32 carries the comparison
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

    raw = {**CONFIG_T, "layers": [layer(attention(4, 2, 64, 64, 200, 0.1, 20000.0, 32), dense(64)), *CONFIG_T["layers"][1:3]]}
    folder = write_model(tmp_path, raw)
    prompts = [random_ids(90 + i, n, CONFIG_T["vocab"]) for i, n in enumerate((40, 33, 25, 47))]
    params = SamplingParams(max_tokens=30, ignore_eos=True)
    roomy = LLMEngine.from_pretrained(folder, EngineConfig(block_size=16, num_blocks=64, max_model_len=128, max_num_seqs=4, dtype=torch.float32))
    want = roomy.generate(prompts, params)
    tight = LLMEngine.from_pretrained(folder, EngineConfig(block_size=16, num_blocks=11, max_model_len=128, max_num_seqs=4, dtype=torch.float32))
    got = tight.generate(prompts, params)
    assert tight.scheduler.num_preemptions > 0
    assert got == want
