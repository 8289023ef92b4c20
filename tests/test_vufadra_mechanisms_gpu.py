"""The mechanisms of the Vufadra design alone, kernel by kernel, against the plain functions of ``plain_vufadra.py``: dynamic-tanh
norms with the residual sum and the token shift, mixes of neighbouring tokens, normed branches, stretched rotary angles, sigmoid
attention at the edges of its chunks, the generalized delta rule and the recurrence with a bonus."""

from __future__ import annotations

import math

import pytest
import torch

import plain_vufadra as plain
from test_tobadra_mechanisms_gpu import Context, close, cuda, f32, randn

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------ dynamic tanh and its sum


def norm_tensors(g, width, alpha):
    return {"n": 1 + 0.3 * randn(g, width), "n.b": 0.3 * randn(g, width), "n.alpha": torch.tensor(alpha, dtype=torch.float64)}


def as_norm(w, out):
    return f32(w["n"]), f32(w["n.b"]), f32(w["n.alpha"]), out


@pytest.mark.parametrize("width", [36, 50, 1028])
@pytest.mark.parametrize("parts", ["stream", "one", "two", "two_and_bias", "replaced"])
def test_residual_sum_and_two_norms_of_it(width, parts):
    """What is pending of one or two sublayers, with and without a bias, with and without the old stream; one norm and two;
    picked rows leave the stream alone."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(width)
    tokens = 5
    x, first, second, bias = randn(g, tokens, width), randn(g, 3, tokens, width), randn(g, 2, tokens, width), randn(g, width)
    has = dict(stream=(1, 0, 0, 0), one=(1, 1, 0, 0), two=(1, 1, 1, 0), two_and_bias=(1, 1, 1, 1), replaced=(0, 1, 0, 1))[parts]
    whole = has[0] * x + has[1] * first.sum(0) + has[2] * second.sum(0) + has[3] * bias
    a, b = norm_tensors(g, width, 0.7), norm_tensors(g, width, -1.6)
    terms = [f32(t) if h else None for t, h in zip((x, first, second, bias), has)]
    args = dict(zip(("x", "first", "second", "bias"), terms))
    for dtype, tolerance in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3)):
        outs = [torch.empty(tokens, width, dtype=dtype, device="cuda") for _ in range(2)]
        x_out = torch.empty(tokens, width, device="cuda")
        ops.tanh_norms(**args, x_out=x_out, norms=[as_norm(a, outs[0]), as_norm(b, outs[1])])
        close(x_out, whole, 2e-6)
        close(outs[0], plain.dynamic_tanh(whole, a, "n"), tolerance)
        close(outs[1], plain.dynamic_tanh(whole, b, "n"), tolerance)
        rows = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
        picked = torch.empty(3, width, dtype=dtype, device="cuda")
        ops.tanh_norms(**args, x_out=None, norms=[as_norm(b, picked)], rows=rows)
        close(picked, plain.dynamic_tanh(whole, b, "n")[[4, 0, 4]], tolerance)
        # the sum alone, into the right half of wider rows
        joined = torch.full((tokens, 2 * width), 7.0, dtype=dtype, device="cuda")
        ops.sum_rows(**args, out=joined, column=width)
        close(joined[:, width:], whole, tolerance)
        assert float(joined[:, :width].float().min()) == 7.0


CUTS = [((0, 1), (1, 5)), ((0, 2), (1, 1)), ((0, 1), (1, 1)), ((0, 20), (1, 2)), ((0, 17), (1, 20)), ((2, 2),), ((2, 1),), ((2, 4),)]


@pytest.mark.parametrize("width", [36, 50, 1028])
@pytest.mark.parametrize("which", ["norms", "mix"])
def test_the_previous_token_in_portions_of_unequal_requests(width, which):
    """Two requests in one batch, cut into portions (single tokens, two tokens): a portion's first token reads the last h of
    the step before from its slot; a third request starts in the slot that the first one has used."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(width)
    shift, w, other = randn(g, width), norm_tensors(g, width, 0.9), norm_tensors(g, width, 0.4)
    mus = randn(g, 3, width)
    for dtype, tolerance in ((torch.float32, 3e-6), (torch.bfloat16, 6e-3)):
        requests = [randn(g, n, width).to(dtype).double() for n in (41, 29, 7)]
        if which == "norms":
            want = [plain.mix_previous(plain.dynamic_tanh(r, w, "n"), shift) for r in requests]
        else:
            want = [torch.stack([plain.mix_previous(r, mu) for mu in mus]) for r in requests]
        columns = 0 if which == "norms" else 8
        state = torch.full((4, columns + width), 9.0, dtype=torch.float32, device="cuda")
        got, done = [[], [], []], [0, 0, 0]
        for step in CUTS:
            ctx = Context([n for _, n in step], [done[r] for r, _ in step], [[2, 0, 2][r] for r, _ in step])
            rows = torch.cat([requests[r][done[r] : done[r] + n] for r, n in step])
            count = rows.shape[0]
            if which == "norms":
                out, beside = (torch.empty(count, width, dtype=dtype, device="cuda") for _ in range(2))
                ops.tanh_norms(x=f32(0.5 * rows), first=f32(torch.stack((0.25 * rows, 0.25 * rows))), second=None, bias=None,
                               x_out=torch.empty(count, width, device="cuda"), norms=[as_norm(w, out), as_norm(other, beside)],
                               shift=f32(shift), state=state, ctx=ctx)  # fmt: skip
                close(beside, plain.dynamic_tanh(rows, other, "n"), tolerance)  # the second norm is not shifted
            else:
                out = torch.empty(3, count, width, dtype=dtype, device="cuda")
                ops.token_mix(h=cuda(rows, dtype), mu=f32(mus), ctx=ctx, state=state, out=out, state_column=8)
            first = 0
            for r, n in step:
                got[r].append(out[..., first : first + n, :].cpu())
                done[r], first = done[r] + n, first + n
        for r in range(3):
            close(torch.cat(got[r], dim=-2), want[r], tolerance)


@pytest.mark.parametrize("which", ["norms", "mix"])
def test_the_previous_token_in_a_long_step(which):
    """Enough tokens that a thread takes a run of them: entries that start and end inside a run, entries of one and two
    tokens, entries that go on from their past beside fresh ones."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(4)
    width, cut = 40, [300, 1, 2, 5, 8, 260, 3]
    shift, w = randn(g, width), norm_tensors(g, width, 1.2)
    requests = [randn(g, 20 + n, width).float().double() for n in cut]
    state = torch.full((8, width), 9.0, dtype=torch.float32, device="cuda")

    def run(rows, ctx):
        out = torch.empty(1, *rows.shape, dtype=torch.float32, device="cuda")
        if which == "norms":
            ops.tanh_norms(x=f32(rows), first=None, second=None, bias=None, x_out=None, norms=[as_norm(w, out[0])], shift=f32(shift), state=state, ctx=ctx)
        else:
            ops.token_mix(h=f32(rows), mu=f32(shift.view(1, -1)), ctx=ctx, state=state, out=out)
        return out[0]

    inner = (lambda r: plain.dynamic_tanh(r, w, "n")) if which == "norms" else (lambda r: r)
    for starts in ([20] * 7, [20, 0, 20, 0, 20, 0, 0]):
        for slot, (r, first) in enumerate(zip(requests, starts)):
            if first:
                run(r[:first], Context([first], [0], [slot]))
        out = run(torch.cat([r[s : s + n] for r, s, n in zip(requests, starts, cut)]), Context(cut, starts, list(range(7))))
        # a request that starts in the middle of these rows sees zeros in front of it
        want = torch.cat([plain.mix_previous(inner(r), shift)[s : s + n] if s else plain.mix_previous(inner(r[:n]), shift) for r, s, n in zip(requests, starts, cut)])
        close(out, want, 3e-6)
        for slot, (r, s, n) in enumerate(zip(requests, starts, cut)):
            close(state[slot], inner(r)[s + n - 1], 3e-6)


@pytest.mark.parametrize("width", [36, 50, 1028, 12288])
def test_normed_branches_joined(width):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(width)
    tokens, eps = 4, (0.2, 0.7)
    parts = [randn(g, s, tokens, width) * scale for s, scale in ((3, 0.1), (1, 9.0))]
    weights = [1 + 0.3 * randn(g, width) for _ in parts]
    out = torch.empty(tokens, width, device="cuda")
    ops.branch_norm_sum([(f32(p), factor, f32(w), e) for p, factor, w, e in zip(parts, (0.5, 0.25), weights, eps)], out)
    want = sum(factor * plain.rms_norm(p.sum(0), w, e) for p, factor, w, e in zip(parts, (0.5, 0.25), weights, eps))
    close(out, want, 3e-6)


# --------------------------------------------------------------------------------------- attention


@pytest.mark.parametrize("rot", [
    {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 2.0}},
    {"base": 500.0, "dims": 6, "scaling": {"factor": 2.5, "original": 90, "fast": 40.0, "slow": 0.5}},
    {"base": 3000.0, "dims": 20, "scaling": {"factor": 1.0, "original": 64, "fast": 3.0, "slow": 3.0}},
    {"base": 700.0, "dims": 2},
])  # fmt: skip
def test_stretched_angles_and_their_amplitude(rot):
    from mini_engine_b200.csrc import ops
    from mini_engine_b200.parts.rotary import RotaryEncoding

    rope = RotaryEncoding("", 0, head_dim=41, theta=rot["base"], rotary_dim=rot["dims"], double_angles=True, yarn=rot.get("scaling"))
    freq, amplitude = plain.frequencies(rot)
    positions = torch.tensor([0, 1, 77, 1111, 99991, 1000003], dtype=torch.int32)
    out = torch.empty(6, rot["dims"] // 2, 2, dtype=torch.float32, device="cuda")
    ops.rope_table(cuda(rope.inv_freq()), cuda(positions), out, rope.amplitude)
    angle = positions.double().view(-1, 1) * torch.tensor(freq, dtype=torch.float64)
    want = amplitude * torch.stack((torch.cos(angle), torch.sin(angle)), dim=-1)
    assert float((out.cpu().double() - want).abs().max()) < 1e-6


class Cached:
    """One request's keys and values in pages out of order, its queries through the attention kernel that the sizes choose."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, page, total, **options):
        self.__dict__.update(dtype=dtype, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, page=page, options=options)
        count = -(-total // page)
        order = torch.randperm(2 * count, generator=torch.Generator().manual_seed(7))[:count]
        self.table = order.to(torch.int32)
        self.k_pages = torch.full((2 * count + 1, kv_heads, page, dim), 3.0, dtype=dtype, device="cuda")
        self.v_pages = torch.full((2 * count + 1, kv_heads, page, vdim), 3.0, dtype=dtype, device="cuda")

    def step(self, q, k, v, first, released=0):
        """Rows of the tokens from ``first`` on; pages wholly below position ``released`` have been given back."""
        from test_kernels_gpu import fake_context

        from mini_engine_b200.csrc import ops

        tokens = q.shape[0]
        positions = torch.arange(first, first + tokens)
        pages, offsets = self.table[positions // self.page].long(), positions % self.page
        self.k_pages[pages.cuda(), :, offsets.cuda()] = cuda(k, self.dtype)
        self.v_pages[pages.cuda(), :, offsets.cuda()] = cuda(v, self.dtype)
        table = self.table.clone()
        table[: released // self.page] = -1
        out = torch.full((tokens, self.heads * self.vdim), float("nan"), dtype=self.dtype, device="cuda")
        data = dict(new_counts=[tokens], lengths=[first + tokens], entry_of=torch.zeros(tokens, dtype=torch.int32).cuda(),
                    positions=cuda(positions.to(torch.int32)))  # fmt: skip
        ops.paged_attention(
            q=cuda(q.reshape(tokens, -1), self.dtype), k_pages=self.k_pages, v_pages=self.v_pages, block_table=cuda(table.view(1, -1)),
            ctx=fake_context(data), out=out, heads=self.heads, kv_heads=self.kv_heads, head_dim=self.dim, window=0, value_dim=self.vdim,
            **self.options,
        )  # fmt: skip
        return out.cpu()


SIZES = [(6, 2, 16, 24, 16), (3, 1, 11, 6, 4), (4, 4, 64, 64, 16), (6, 2, 64, 64, 4), (4, 2, 128, 128, 16), (3, 1, 128, 128, 32), (10, 1, 128, 128, 16)]


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,page", SIZES)
@pytest.mark.parametrize("chunk", [1, 16, 40, 129, 500])
@pytest.mark.parametrize("weights", ["sigmoid", "softmax"])
@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_chunked_attention_with_keys_at_the_edges_of_chunks(heads, kv_heads, dim, vdim, page, chunk, weights, dtype_name):
    """Keys just inside and just outside a query's chunk stand out: the chunk's first key and the last key of the chunk in front
    of it are the direction of that query, scaled up, so that an edge that is one token off shows.  Whole prompts (the tcgen05
    kernel, blocks that span several chunks), portions down to two tokens, decoded tokens (split and gathered); pages of
    earlier chunks are gone."""
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype_name]
    g = torch.Generator().manual_seed(dim + chunk)
    total, scale = 300, 1.0 / math.sqrt(dim)
    q, k, v = randn(g, total, heads, dim), randn(g, total, kv_heads, dim), randn(g, total, kv_heads, vdim)
    bias = randn(g, heads) - 2.0
    for n, i in enumerate(range(chunk, total, max(29, chunk // 3))):
        j = i // chunk * chunk - n % 2  # inside: the chunk's first key; outside: the key in front of it
        head = (5 * n) % heads
        k[j, head // (heads // kv_heads)] = q[i, head] * (7.0 / (scale * float(q[i, head].norm()) ** 2))
    q, k, v = (t.to(dtype).double() for t in (q, k, v))

    def at(seen):
        if weights == "sigmoid":
            return plain.sigmoid_attention(q, k, v, scale, bias, seen).reshape(total, -1)
        spread = lambda t: t.repeat_interleave(heads // kv_heads, dim=1)  # noqa: E731
        scores = torch.einsum("ihd,jhd->hij", q, spread(k)) * scale
        probabilities = torch.softmax(scores.masked_fill(seen == 0, -math.inf), dim=-1)
        return torch.einsum("hij,jhd->ihd", probabilities, spread(v)).reshape(total, -1)

    seen = plain.chunk_mask(total, chunk)
    want = at(seen.double())
    if 1 < chunk < total:  # the edges matter: chunks that start one token off are another result
        i, j = torch.arange(total).view(-1, 1), torch.arange(total).view(1, -1)
        for off in (1, -1):
            moved = (j <= i) & ((i + off) // chunk == (j + off) // chunk)
            assert float((at(moved.double()) - want).abs().max()) > 0.05 * float(want.abs().max())
    tolerance = 5e-6 if dtype_name == "float32" else 1.5e-2
    options = dict(scale=scale, chunk=chunk, sigmoid_bias=f32(bias) if weights == "sigmoid" else None)
    for cuts in ([0, total], [0, 2, 4, 50, 51, 118, 119, 160, 290, *range(291, total + 1)]):
        run = Cached(dtype, heads, kv_heads, dim, vdim, page, total, **options)
        got = [run.step(q[a:b], k[a:b], v[a:b], a, released=a // chunk * chunk) for a, b in zip(cuts, cuts[1:])]
        close(torch.cat(got), want, tolerance)


@pytest.mark.parametrize("place", [0, 15, 16, 37, 899])
@pytest.mark.parametrize("dim,vdim", [(24, 16), (64, 64), (128, 128)])
@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_a_far_key_that_stands_out(place, dim, vdim, dtype_name):
    """Nine hundred keys whose weights are next to nothing and one whose score stands out (the first token, a page's last and
    first slot, far back, the query itself): the last query's output is that key's value, decoded and at a prompt's end."""
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype_name]
    g = torch.Generator().manual_seed(3)
    total = 900
    q, k, v = 0.02 * randn(g, total, 1, dim), 0.02 * randn(g, total, 1, dim), randn(g, total, 1, vdim)
    q[-1] = randn(g, 1, dim)
    k[place] = q[-1] * (24.0 / float(q[-1].norm()) ** 2)
    q, k, v = (t.to(dtype).double() for t in (q, k, v))
    bias = f32(torch.tensor([-16.0]))
    want = plain.sigmoid_attention(q, k, v, 1.0, torch.tensor([-16.0]), plain.chunk_mask(total, total).double())[-1, 0]
    assert float((want - v[place, 0]).abs().max()) < 2e-2 * float(v.abs().max())
    for cuts in ([0, total], [0, total - 1, total]):
        run = Cached(dtype, 1, 1, dim, vdim, 16, total, scale=1.0, chunk=1000, sigmoid_bias=bias)
        got = torch.cat([run.step(q[a:b], k[a:b], v[a:b], a) for a, b in zip(cuts, cuts[1:])])
        close(got[-1], want, 2e-5 if dtype_name == "float32" else 2e-2)


def test_sigmoid_weights_far_below_and_above_a_half():
    """Biases of -30 and +30 and scores of hundreds: weights of 1e-13 and of one, nothing overflows."""
    g = torch.Generator().manual_seed(8)
    total, heads, dim = 200, 2, 128
    q, k, v = (randn(g, total, heads, dim).bfloat16().double() for _ in range(3))
    for bias, scale in ((-30.0, 0.01), (30.0, 0.01), (0.0, 8.0)):
        want = plain.sigmoid_attention(q, k, v, scale, torch.full((heads,), bias), plain.chunk_mask(total, total).double()).reshape(total, -1)
        for cuts in ([0, total], [0, 3, total - 1, total]):
            run = Cached(torch.bfloat16, heads, heads, dim, dim, 16, total, scale=scale, chunk=256, sigmoid_bias=f32(torch.full((heads,), bias)))
            got = torch.cat([run.step(q[a:b], k[a:b], v[a:b], a) for a, b in zip(cuts, cuts[1:])])
            if bias < 0:  # beside values of one such weights are nothing
                assert float(got.float().abs().max()) < 1e-5
            else:
                close(got, want, 1.5e-2)


# ------------------------------------------------------------------------------------- recurrences

STATE_SIZES = [(2, 16, 8), (3, 24, 40), (1, 6, 5), (2, 64, 64), (2, 128, 128), (1, 200, 36), (1, 257, 12), (1, 512, 64)]


def state_inputs(rule, heads, dim, vdim, tokens):
    g = torch.Generator().manual_seed(dim + heads)
    q, k = randn(g, tokens, heads * dim), randn(g, tokens, heads * dim)
    v, z, rate = randn(g, tokens, heads * vdim), randn(g, tokens, heads * dim), randn(g, tokens, heads * dim)
    decay_bias, channel = (randn(g, heads * dim) - 2.0 if rule == "bonus" else randn(g, heads * dim)), randn(g, heads * dim)
    return q, k, v, z, rate, decay_bias, channel


def plain_states(rule, heads, dim, vdim, q, k, v, z, rate, decay_bias, channel, decay_scale):
    heads_of = lambda t, n: t.view(t.shape[0], heads, n)  # noqa: E731
    if rule == "removal":
        decay = torch.exp(-decay_scale * plain.sigmoid(z + decay_bias))
        return plain.removal_recurrence(heads_of(q, dim), heads_of(k, dim), heads_of(v, vdim), heads_of(decay, dim), heads_of(plain.sigmoid(rate + channel), dim))
    decay = torch.exp(-torch.exp(z + decay_bias))
    return plain.bonus_recurrence(heads_of(q, dim), heads_of(k, dim), heads_of(v, vdim), heads_of(decay, dim), channel.view(heads, dim))


class StateRun:
    def __init__(self, rule, heads, dim, vdim, inputs, decay_scale=0.6):
        self.__dict__.update(rule=rule, heads=heads, dim=dim, vdim=vdim, inputs=inputs, decay_scale=decay_scale)
        self.state = torch.full((5, heads * dim * vdim + 4), 7.0, dtype=torch.float32, device="cuda")

    def step(self, spans, slots, chunk_min=0):
        """``spans``: (first, count) per entry, all of the same sequence."""
        from mini_engine_b200.csrc import ops

        q, k, v, z, rate, decay_bias, channel = self.inputs
        take = lambda t: torch.cat([t[a : a + n] for a, n in spans])  # noqa: E731
        rows = torch.cat((take(k), take(v), take(rate), take(q)), dim=1)
        sums = f32(torch.stack((0.25 * rows, 0.75 * rows)))
        logits = f32(take(z).unsqueeze(0))
        wide, tall = self.heads * self.dim, self.heads * self.vdim
        count = rows.shape[0]
        row, numbers = ops.state_rule_floats(self.rule, self.dim, self.vdim)
        held = torch.empty(count, self.heads * row, device="cuda"), torch.empty(count, self.heads * numbers, device="cuda")
        sizes = dict(heads=self.heads, dim=self.dim, vdim=self.vdim)
        ops.state_prepare(
            rule=self.rule, k=(sums, 0), v=(sums, wide), rate=(sums, wide + tall) if self.rule == "removal" else None, q=(sums, 2 * wide + tall),
            logits=(logits, 0), decay_bias=f32(decay_bias), channel=f32(channel), rows=held[0], scalars=held[1], decay_scale=self.decay_scale,
            unit_eps=1e-6, **sizes,
        )  # fmt: skip
        out = torch.empty(count, self.heads * self.vdim, device="cuda")
        ctx = Context([n for _, n in spans], [a for a, _ in spans], slots)
        records = None
        if chunk_min:
            records = torch.full((count // ops.STATE_CHUNK + len(spans), self.heads * ops.state_record_floats(self.rule, self.dim)), float("nan"), device="cuda")
        ops.state_walk(rule=self.rule, rows=held[0], scalars=held[1], ctx=ctx, state=self.state, out=out, chunk_min=chunk_min, records=records, **sizes)
        return out.cpu()


@pytest.mark.parametrize("rule", ["removal", "bonus"])
@pytest.mark.parametrize("heads,dim,vdim", STATE_SIZES)
def test_states_whole_in_portions_token_by_token_and_side_by_side(rule, heads, dim, vdim):
    """Whole against the plain loop (from a slot that held something else), the state it leaves; portions and single tokens
    from the carried state are the same bits; two entries of one batch at different places of the sequence."""
    tokens = 70
    inputs = state_inputs(rule, heads, dim, vdim, tokens)
    if rule == "removal":  # keys of a few units, so that a removal of rates near one stays a contraction
        inputs = (inputs[0], inputs[1] / math.sqrt(dim), *inputs[2:])
    run = StateRun(rule, heads, dim, vdim, inputs)
    want, state = plain_states(rule, heads, dim, vdim, *inputs, 0.6)
    whole = run.step([(0, tokens)], [0])
    close(whole, want.reshape(tokens, -1), 2e-5)
    close(run.state[0, : heads * dim * vdim].view(heads, vdim, dim), state.transpose(1, 2), 2e-5)
    assert float(run.state[0, heads * dim * vdim :].min()) == 7.0  # what lies behind the states is not theirs
    cuts = [0, 1, 2, 4, 20, 37, 38, tokens]
    assert torch.equal(torch.cat([run.step([(a, b - a)], [1]) for a, b in zip(cuts, cuts[1:])]), whole)
    assert torch.equal(run.state[0], run.state[1])
    run.step([(0, 33)], [2])
    both = run.step([(0, 2), (33, 37)], [3, 2])
    assert torch.equal(both[:2], whole[:2]) and torch.equal(both[2:], whole[33:])
    assert torch.equal(run.state[2], run.state[0])


@pytest.mark.parametrize("rule", ["removal", "bonus"])
@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 8), (3, 24, 40), (1, 4, 4), (2, 64, 64), (2, 128, 128), (1, 100, 36), (3, 48, 48), (1, 32, 68)])
@pytest.mark.parametrize("decays", ["mixed", "strong", "none"])
def test_states_in_chunks(rule, heads, dim, vdim, decays):
    """Long entries in chunks of 16 tokens: whole, from a carried state, whole chunks and a rest of one token and of fifteen,
    beside entries that walk and beside each other, with decays that leave nothing of a channel within a token, and with none."""
    tokens = 150
    q, k, v, z, rate, decay_bias, channel = state_inputs(rule, heads, dim, vdim, tokens)
    z, scale = {"mixed": (2.0 * z, 0.6), "strong": (z + (3.0 if rule == "bonus" else 9.0), 40.0), "none": (z - 60.0, 0.6)}[decays]
    if rule == "removal":
        k = k / math.sqrt(dim)
    inputs = (q, k, v, z, rate, decay_bias, channel)
    run = StateRun(rule, heads, dim, vdim, inputs, decay_scale=scale)
    want, state = plain_states(rule, heads, dim, vdim, *inputs, scale)
    want = want.reshape(tokens, -1)
    states_of = lambda slot: run.state[slot, : heads * dim * vdim].view(heads, vdim, dim)  # noqa: E731
    for cuts in ([0, tokens], [0, 49, 97, tokens], [0, 5, 38, 101, 103, tokens], [0, 33, 112, tokens]):
        run.state.fill_(7.0)
        got = torch.cat([run.step([(a, b - a)], [1], chunk_min=33) for a, b in zip(cuts, cuts[1:])])
        close(got, want, 3e-5)
        close(states_of(1), state.transpose(1, 2), 3e-5)
        assert float(run.state[0].min()) == 7.0 and float(run.state[1, heads * dim * vdim :].min()) == 7.0
    # in one batch: a single token, a long entry, a walking portion, another long entry
    run.step([(0, 60)], [0], chunk_min=33)
    run.step([(0, 20)], [2], chunk_min=33)
    got = run.step([(60, 1), (0, tokens), (20, 32), (0, 35)], [0, 3, 2, 4], chunk_min=33)
    for rows, first in ((got[:1], 60), (got[1 : 1 + tokens], 0), (got[1 + tokens : 33 + tokens], 20), (got[33 + tokens :], 0)):
        close(rows, want[first : first + rows.shape[0]], 3e-5)
    close(states_of(3), state.transpose(1, 2), 3e-5)


def test_a_key_is_removed_channel_by_channel_hundreds_of_tokens_later():
    """A value stored under a key stays for hundreds of tokens of other keys, is read back, is then removed at a rate per
    channel by writing zero under the same key, and what the rates left is read."""
    heads, dim, vdim, tokens = 1, 32, 8, 400
    g = torch.Generator().manual_seed(0)
    q, v = torch.zeros(tokens, dim, dtype=torch.float64), torch.zeros(tokens, vdim, dtype=torch.float64)
    k = torch.zeros(tokens, dim, dtype=torch.float64)
    k[:, 16:] = randn(g, tokens, 16)  # the other keys live in other channels
    key = torch.cat((randn(g, 16), torch.zeros(16, dtype=torch.float64)))
    for t in (0, 300):
        k[t] = key
    v[0], q[250], q[399] = randn(g, vdim), key, key
    v[1:250] = randn(g, 249, vdim)
    z = torch.full((tokens, dim), -40.0, dtype=torch.float64)  # no decay
    rate, channel = torch.zeros(tokens, dim, dtype=torch.float64), torch.linspace(-3.0, 3.0, dim, dtype=torch.float64)
    inputs = (q, k, v, z, rate, torch.zeros(dim, dtype=torch.float64), channel)
    want, _ = plain_states("removal", heads, dim, vdim, *inputs, 0.6)
    got = StateRun("removal", heads, dim, vdim, inputs).step([(0, tokens)], [0])
    close(got[250], v[0] * float(key @ key), 1e-4)
    close(got, want.reshape(tokens, -1), 2e-5)
    left = float((key * key * (1.0 - plain.sigmoid(channel))).sum())
    close(got[399], v[0] * left, 1e-4)


def test_the_current_token_counts_through_its_bonus_alone():
    """Bonus zero: a token does not see itself; a bonus of minus the key's square takes it out; the next token sees it whole."""
    heads, dim, vdim, tokens = 2, 20, 12, 3
    q, k, v, z, rate, decay_bias, channel = state_inputs("bonus", heads, dim, vdim, tokens)
    for bonus in (0.0 * channel, channel, 5.0 + channel):
        inputs = (q, k, v, z, rate, decay_bias, bonus)
        want, _ = plain_states("bonus", heads, dim, vdim, *inputs, 1.0)
        got = StateRun("bonus", heads, dim, vdim, inputs).step([(0, tokens)], [0])
        close(got, want.reshape(tokens, -1), 5e-6)
        if float(bonus.abs().max()) == 0.0:
            assert float(got[0].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_low_rank_sums_behind_tanh(dtype):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(1)
    proj = randn(g, 3, 7, 20)
    out = torch.empty(7, 9 * (2 if dtype == torch.bfloat16 else 1), dtype=dtype, device="cuda")
    ops.split_halves(f32(proj), 4, 9, out, activate=True)
    want = torch.tanh(proj.sum(0)[:, 4:13])
    got = out.cpu().double()
    close(got[:, :9] + got[:, 9:] if dtype == torch.bfloat16 else got, want, 2e-5 if dtype == torch.bfloat16 else 2e-6)


@pytest.mark.parametrize("gate", ["silu", "sigmoid"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,vdim", [(3, 20), (2, 64), (4, 128), (1, 7)])
def test_finish_with_a_weight_of_every_head(gate, dtype, heads, vdim):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(2)
    tokens, eps = 9, 0.2
    o, gates, weight = randn(g, tokens, heads, vdim), randn(g, 2, tokens, 4 + heads * vdim), 1 + 0.3 * randn(g, heads * vdim)
    out = torch.empty(tokens, heads * vdim, dtype=dtype, device="cuda")
    ops.gla_finish(o=f32(o).view(tokens, -1), proj=f32(gates), gate_column=4, weight=f32(weight), eps=eps, out=out, heads=heads, vdim=vdim, gate=gate)
    activation = plain.silu if gate == "silu" else plain.sigmoid
    want = plain.rms_norm(o, None, eps).reshape(tokens, -1) * weight * activation(gates.sum(0)[:, 4:])
    close(out, want, 2e-6 if dtype == torch.float32 else 5e-3)
