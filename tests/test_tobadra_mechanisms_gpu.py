"""The mechanisms of the Tobadra design alone, kernel by kernel, against the plain functions of ``plain_tobadra.py``: the
gated sublayer between two norms, the convolution in front of a mixer, attention with rotated values at the edges of its
window, lightning attention, the gated delta rule with its convolutions, the router, the units' products."""

from __future__ import annotations

import math
import random

import pytest
import torch

import plain_tobadra as plain

pytestmark = pytest.mark.gpu


def cuda(t, dtype=None):
    return None if t is None else t.to(device="cuda", dtype=dtype or t.dtype).contiguous()


def f32(t):
    return cuda(t, torch.float32)


def close(got, want, tolerance):
    want = want.double()
    error = float((got.cpu().double() - want).abs().max()) / max(float(want.abs().max()), 1e-30)
    assert error <= tolerance, f"relative error {error:.3g}"


class Context:
    """What the kernels' bindings read of a step: entry ``b`` brings ``counts[b]`` tokens from position ``starts[b]``."""

    def __init__(self, counts, starts, slots):
        self.num_entries = len(counts)
        cu = [0]
        for n in counts:
            cu.append(cu[-1] + n)
        self.cu_tokens = torch.tensor(cu, dtype=torch.int32, device="cuda")
        self.entry_of_token = torch.tensor([b for b, n in enumerate(counts) for _ in range(n)], dtype=torch.int32, device="cuda")
        self.state_slots = torch.tensor(slots, dtype=torch.int32, device="cuda")
        self.fresh = torch.tensor([1 if s == 0 else 0 for s in starts], dtype=torch.int32, device="cuda")


def randn(g, *shape):
    return torch.randn(*shape, generator=g, dtype=torch.float64)


# ------------------------------------------------------------------- sublayers between two norms


@pytest.mark.parametrize("hidden", [36, 50, 1000, 4096])
@pytest.mark.parametrize("splits,gate_splits", [(1, 1), (3, 2), (8, 8), (9, 1)])
@pytest.mark.parametrize("parts", ["all", "no_bias", "no_gate"])
def test_gate_norm_residual_sum_and_next_norm(hidden, splits, gate_splits, parts):
    """Bias before the gate, gate before the norm behind the sublayer, that norm before the sum; both norms have an eps
    that matters.  With rows picked, the stream stays as it was."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(hidden + splits)
    tokens, out_eps, eps = 5, 0.3, 0.07
    x, y, gate = randn(g, tokens, hidden), randn(g, splits, tokens, hidden), randn(g, gate_splits, tokens, hidden)
    bias, gate_bias, w_out, w = randn(g, hidden), randn(g, hidden), 1 + 0.1 * randn(g, hidden), 1 + 0.1 * randn(g, hidden)
    has_bias, has_gate = parts != "no_bias", parts != "no_gate"
    whole = y.sum(0) + (bias if has_bias else 0)
    if has_gate:
        whole = whole * plain.sigmoid(gate.sum(0) + gate_bias)
    stream = x + plain.rms_norm(whole, w_out, out_eps)
    normed = plain.rms_norm(stream, w, eps)
    args = dict(pending=f32(y), bias=f32(bias) if has_bias else None, gate=f32(gate) if has_gate else None,
                gate_bias=f32(gate_bias) if has_gate else None, out_weight=f32(w_out), out_eps=out_eps, weight=f32(w), eps=eps)  # fmt: skip
    for dtype, tolerance in ((torch.float32, 3e-6), (torch.bfloat16, 5e-3)):
        held = f32(x)
        rows = torch.tensor([3, 0, 3], dtype=torch.int32, device="cuda")
        picked = torch.empty(3, hidden, dtype=dtype, device="cuda")
        ops.sandwich_norm(x=held, out=picked, rows=rows, **args)
        assert torch.equal(held, f32(x))
        close(picked, normed[[3, 0, 3]], tolerance)
        out = torch.empty(tokens, hidden, dtype=dtype, device="cuda")
        ops.sandwich_norm(x=held, out=out, **args)
        close(held, stream, 3e-6)
        close(out, normed, tolerance)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 16])
@pytest.mark.parametrize("width", [36, 50, 1028])
def test_input_convolution_in_portions_of_unequal_requests(taps, width):
    """Two requests in one batch, cut into portions (single tokens, two tokens, longer than the taps): each portion reaches
    into the tokens in front of it through its slot; a third request starts in the slot that the first one has used."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(taps * 100 + width)
    w = randn(g, width, taps)
    requests = [randn(g, 41, width), randn(g, 29, width), randn(g, 7, width)]
    for dtype, tolerance in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        requests = [r.to(dtype).double() for r in requests]
        want = [r + plain.causal_conv(r, w) for r in requests]
        state = torch.full((4, taps - 1, width), 9.0, dtype=torch.float32, device="cuda") if taps > 1 else None
        got = [[], [], []]
        steps = [((0, 1), (1, 5)), ((0, 2), (1, 1)), ((0, 1), (1, 1)), ((0, 20), (1, 2)), ((0, 17), (1, 20)), ((2, 2),), ((2, 1),), ((2, 4),)]
        done = [0, 0, 0]
        for step in steps:
            ctx = Context([n for _, n in step], [done[r] for r, _ in step], [[2, 0, 2][r] for r, _ in step])
            h = cuda(torch.cat([requests[r][done[r] : done[r] + n] for r, n in step]), dtype)
            out = torch.empty_like(h)
            ops.input_convolution(h=h, taps=f32(w.T), ctx=ctx, state=state, out=out)
            first = 0
            for r, n in step:
                got[r].append(out[first : first + n].cpu())
                done[r], first = done[r] + n, first + n
        for r in range(3):
            close(torch.cat(got[r]), want[r], tolerance)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_input_convolution_of_a_long_step(taps):
    """Enough tokens that a thread takes a run of them: entries that start and end inside a run, entries shorter than the
    taps, entries that go on from their past beside fresh ones."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(taps)
    width, cut = 40, [300, 1, 2, 5, 8, 260, 3]
    w, requests = randn(g, width, taps), [randn(g, 20 + n, width).float().double() for n in cut]
    state = torch.full((8, taps - 1, width), 9.0, dtype=torch.float32, device="cuda") if taps > 1 else None
    for starts in ([20] * 7, [20, 0, 20, 0, 20, 0, 0]):
        for r, first in zip(requests, starts):  # what came before, request by request
            if first:
                slot = next(i for i, x in enumerate(requests) if x is r)
                ops.input_convolution(h=f32(r[:first]), taps=f32(w.T), ctx=Context([first], [0], [slot]), state=state, out=f32(r[:first]))
        h = torch.cat([r[s : s + n] for r, s, n in zip(requests, starts, cut)])
        out = torch.empty(h.shape, dtype=torch.float32, device="cuda")
        ops.input_convolution(h=f32(h), taps=f32(w.T), ctx=Context(cut, starts, list(range(7))), state=state, out=out)
        want = torch.cat([(r + plain.causal_conv(r, w))[s : s + n] for r, s, n in zip(requests, starts, cut)])
        close(out, want, 3e-6)
        if taps > 1:
            for slot, (r, s, n) in enumerate(zip(requests, starts, cut)):
                held = torch.cat((torch.zeros(taps - 1, width, dtype=torch.float64), r))[s + n : s + n + taps - 1]
                assert torch.equal(state[slot].cpu(), held.float())


# ------------------------------------------------------------------- attention with rotated values


def test_angles_in_double_precision():
    from mini_engine_b200.parts.rotary import RotaryEncoding
    from mini_engine_b200.csrc import ops

    rope = RotaryEncoding("", 0, head_dim=64, theta=10000.0, double_angles=True)
    positions = torch.tensor([0, 1, 77, 1111, 99991, 1000003], dtype=torch.int32)
    out = torch.empty(6, 32, 2, dtype=torch.float32, device="cuda")
    ops.rope_table(cuda(rope.inv_freq()), cuda(positions), out)
    angle = positions.double().view(-1, 1) * 10000.0 ** (-2.0 * torch.arange(32, dtype=torch.float64) / 64)
    want = torch.stack((torch.cos(angle), torch.sin(angle)), dim=-1)
    assert float((out.cpu().double() - want).abs().max()) < 5e-7


def angle_table(positions, base, dims):
    angle = positions.double().view(-1, 1) * torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    return f32(torch.stack((torch.cos(angle), torch.sin(angle)), dim=-1))


class AttentionRun:
    """One request's rows through the store kernel, the attention kernel that the sizes choose and the turn back."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, base, dims, window, scale, page, total, seed=5):
        self.__dict__.update(dtype=dtype, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, base=base, dims=dims, window=window,
                             scale=scale, page=page)  # fmt: skip
        count = -(-total // page)
        order = torch.randperm(2 * count, generator=torch.Generator().manual_seed(seed))[:count]
        self.table = order.to(torch.int32)
        self.k_pages = torch.full((2 * count + 1, kv_heads, page, dim), 3.0, dtype=dtype, device="cuda")
        self.v_pages = torch.full((2 * count + 1, kv_heads, page, vdim), 3.0, dtype=dtype, device="cuda")

    def step(self, rows, bias, first):
        from test_kernels_gpu import fake_context

        from mini_engine_b200.csrc import ops

        tokens = rows.shape[0]
        positions = torch.arange(first, first + tokens)
        slots = (self.table[positions // self.page] * self.page + positions % self.page).to(torch.int32)
        values = angle_table(positions, self.base, self.vdim)
        q = torch.empty(tokens, self.heads * self.dim, dtype=self.dtype, device="cuda")
        ops.qkv_rope_unit_store(
            qkv=f32(torch.stack((0.25 * rows, 0.75 * rows))), heads=self.heads, kv_heads=self.kv_heads, head_dim=self.dim,
            value_dim=self.vdim, bias=f32(bias), cos_sin=angle_table(positions, self.base, self.dims), unit_norm_eps=None, q_out=q,
            page_size=self.page, slot_mapping=cuda(slots), k_pages=self.k_pages, v_pages=self.v_pages, value_cos_sin=values,
        )  # fmt: skip
        out = torch.full((tokens, self.heads * self.vdim), float("nan"), dtype=self.dtype, device="cuda")
        data = dict(new_counts=[tokens], lengths=[first + tokens], entry_of=torch.zeros(tokens, dtype=torch.int32).cuda(),
                    positions=cuda(positions.to(torch.int32)))  # fmt: skip
        ops.paged_attention(
            q=q, k_pages=self.k_pages, v_pages=self.v_pages, block_table=cuda(self.table.view(1, -1)), ctx=fake_context(data), out=out,
            heads=self.heads, kv_heads=self.kv_heads, head_dim=self.dim, scale=self.scale, window=self.window, value_dim=self.vdim,
        )  # fmt: skip
        ops.turn_heads_back(out, values, self.heads)
        return out.cpu()


SIZES = [(6, 2, 16, 24, 12), (3, 1, 10, 6, 2), (4, 4, 40, 36, 40), (4, 2, 64, 64, 32), (8, 1, 128, 128, 128)]


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims", SIZES)
@pytest.mark.parametrize("window", [1, 17, 33, 300])
@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_attention_with_rotated_values_and_keys_at_the_window_edge(heads, kv_heads, dim, vdim, dims, window, dtype_name):
    """Every 23rd key, just inside and just outside some query's window, is the direction of that query, scaled up: its score
    stands out, so that a window that is one token off shows.  The whole prompt, portions (two tokens, across pages),
    and decoded tokens; in bfloat16 the sizes of 64 and 128 take the tensor-core kernels."""
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype_name]
    g = torch.Generator().manual_seed(dim + window)
    total, base, scale = 170, 300.0, 1.0 / math.sqrt(dim)
    width = (heads + kv_heads) * dim + kv_heads * vdim
    rows, bias = 0.5 * randn(g, total, width), 0.2 * randn(g, width)
    split = lambda r: (r[:, : heads * dim].view(total, heads, dim), r[:, heads * dim : (heads + kv_heads) * dim].view(total, kv_heads, dim),
                       r[:, (heads + kv_heads) * dim :].view(total, kv_heads, vdim))  # fmt: skip
    q, k, v = split(rows + bias)
    p = torch.arange(total)
    q = plain.rotate(q, p, base, dims)
    unturn = lambda x, at: plain.rotate(x.view(1, 1, -1), torch.tensor([at]), base, dims, back=True).view(-1)  # noqa: E731
    for n, i in enumerate(range(window, total, 23)):  # the query at i: its window's first key is i - window + 1
        for j in ((i - window + 1,), (i - window,))[n % 2]:
            head = (7 * n) % heads
            wanted = q[i, head] * (6.0 / (scale * float(q[i, head].norm()) ** 2))  # rotated key: the score is about 6
            group = head // (heads // kv_heads)
            start = heads * dim + group * dim
            rows[j, start : start + dim] = unturn(wanted, j) - bias[start : start + dim]
    q, k, v = split(rows + bias)
    q, k = plain.rotate(q, p, base, dims), plain.rotate(k, p, base, dims)
    at = lambda size: plain.attention_heads(q * scale, k, v, 1.0, base, size).reshape(total, -1)  # noqa: E731
    want = at(window)
    for off in (window - 1, window + 1):  # the edges matter: a window that is one token off is another result
        if off >= 1 and off < total:
            assert float((at(off) - want).abs().max()) > 0.05 * float(want.abs().max())
    tolerance = 3e-6 if dtype_name == "float32" else 2e-2
    for cuts in ([0, total], [0, 2, 4, 50, 51, 118, 119, 160, *range(161, total + 1)]):
        run = AttentionRun(dtype, heads, kv_heads, dim, vdim, base, dims, window, scale, 16, total)
        got = torch.cat([run.step(rows[a:b], bias, a) for a, b in zip(cuts, cuts[1:])])
        close(got, want, tolerance)


@pytest.mark.parametrize("place", [0, 15, 16, 37, 399])
@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(24, 16), (64, 64)])
def test_a_far_key_that_stands_out_brings_its_value_turned_by_the_distance(place, dtype_name, dim, vdim):
    """Four hundred keys and one whose score stands out (the first token, a page's last and first slot, far back, the query
    itself): the output of the last query is that key's value, turned by the distance between the two."""
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype_name]
    g = torch.Generator().manual_seed(3)
    total, base, scale = 400, 50.0, 1.0
    rows = 0.05 * randn(g, total, 2 * dim + vdim)
    rows[-1, :dim] = randn(g, dim)
    q = plain.rotate(rows[-1:, :dim].view(1, 1, dim), torch.tensor([total - 1]), base, dim)
    key = q * (20.0 / float(q.norm()) ** 2)
    rows[place, dim : 2 * dim] = plain.rotate(key, torch.tensor([place]), base, dim, back=True).view(-1)
    rows[place, 2 * dim :] = randn(g, vdim)
    run = AttentionRun(dtype, 1, 1, dim, vdim, base, dim, 0, scale, 16, total)
    got = run.step(rows[:-1], torch.zeros(2 * dim + vdim), 0), run.step(rows[-1:], torch.zeros(2 * dim + vdim), total - 1)
    turned = plain.rotate(rows[place, 2 * dim :].view(1, 1, vdim), torch.tensor([place - total + 1]), base, vdim).view(-1)
    close(got[1][0], turned, 1e-4 if dtype_name == "float32" else 3e-2)
    if place not in (total - 1,):
        assert float((turned - rows[place, 2 * dim :]).abs().max()) > 0.1


# --------------------------------------------------------------------------- lightning attention


@pytest.mark.parametrize("heads,dim,vdim", [(2, 16, 8), (3, 24, 40), (1, 6, 5), (2, 64, 64), (2, 192, 32), (1, 256, 128)])
def test_lightning_whole_in_portions_and_token_by_token(heads, dim, vdim):
    """silu on q, k and v (no other scale), a decay per head (one of them 1), the norm over all heads together with its
    weight, the sigmoid gate: whole against the plain loop; portions and single tokens from the carried state the same
    bits; in chunks of 64 tokens from zero and from a carried state; the slot held another request's state before."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(dim + heads)
    tokens, eps = 150, 1e-3
    decay = [0.9, 1.0, 0.5][:heads]
    widths = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim}
    columns, column = {}, 0
    for key, n in widths.items():
        columns[key], column = column, column + n
    proj = randn(g, tokens, column)
    weight = 1 + 0.1 * randn(g, heads * vdim)
    part = {key: proj[:, columns[key] : columns[key] + n] for key, n in widths.items()}
    q, k = (plain.silu(part[n]).view(tokens, heads, dim) for n in "qk")
    o, want_state = plain.lightning_recurrence(q, k, plain.silu(part["v"]).view(tokens, heads, vdim), decay)
    want = plain.rms_norm(o.reshape(tokens, -1), weight, eps) * plain.sigmoid(part["g"])
    state = torch.full((4, heads, dim, vdim), 7.0, dtype=torch.float32, device="cuda")

    def run(first, count, slot, chunk_min=0):
        rows = proj[first : first + count]
        sums = f32(torch.stack((0.25 * rows, 0.75 * rows)))
        raw = torch.empty(count, heads * vdim, dtype=torch.float32, device="cuda")
        prepared = torch.empty(count, heads * 3 * dim, dtype=torch.float32, device="cuda")
        scratch = torch.empty((count // 64 + 1, heads, dim, vdim), dtype=torch.float32, device="cuda") if chunk_min else None
        ops.retention_scan(proj=sums, columns=columns, cos_sin=None, decay=f32(torch.tensor(decay)), k_scale=1.0,
                           ctx=Context([count], [first], [slot]), state=state, out=raw, prepared=prepared, heads=heads, dim=dim, vdim=vdim,
                           chunk_min=chunk_min, chunk_state=scratch, silu=True)  # fmt: skip
        out = torch.empty(count, heads * vdim, dtype=torch.float32, device="cuda")
        ops.gla_finish(o=raw, proj=sums, gate_column=columns["g"], weight=f32(weight), eps=eps, out=out, heads=heads, vdim=vdim,
                       gate="sigmoid", scope="projection")  # fmt: skip
        return out.cpu()

    whole = run(0, tokens, 0)
    close(whole, want, 2e-5)
    close(state[0], want_state, 2e-5)
    cuts = [0, 2, 3, 20, 21, 85, tokens]
    assert torch.equal(torch.cat([run(a, b - a, 1) for a, b in zip(cuts, cuts[1:])]), whole) and torch.equal(state[0], state[1])
    if ops.retention_chunked_supports(dim, vdim):
        for cuts in ([0, 150], [0, 70, 150], [0, 5, 69, 150]):
            close(torch.cat([run(a, b - a, 2, chunk_min=33) for a, b in zip(cuts, cuts[1:])]), want, 3e-5)
            close(state[2], want_state, 3e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_finish_with_a_norm_per_head_and_a_sigmoid_gate(dtype):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(2)
    tokens, heads, vdim, eps = 9, 3, 20, 0.2
    o, gates, weight = randn(g, tokens, heads, vdim), randn(g, 2, tokens, 5 + heads * vdim), 1 + 0.1 * randn(g, vdim)
    out = torch.empty(tokens, heads * vdim, dtype=dtype, device="cuda")
    ops.gla_finish(o=f32(o).view(tokens, -1), proj=f32(gates), gate_column=5, weight=f32(weight), eps=eps, out=out, heads=heads, vdim=vdim,
                   gate="sigmoid")  # fmt: skip
    want = plain.rms_norm(o, weight, eps).reshape(tokens, -1) * plain.sigmoid(gates.sum(0)[:, 5:])
    close(out, want, 2e-6 if dtype == torch.float32 else 5e-3)


# --------------------------------------------------------------------------------- the delta rule


class DeltaRun:
    """A delta-rule mixer's two kernels on given sums (with ``halves``: two partial sums that meet in the kernels)."""

    def __init__(self, heads, qk_heads, dim, vdim, taps, slots=4, halves=True):
        self.__dict__.update(heads=heads, qk_heads=qk_heads, dim=dim, vdim=vdim, taps=taps, halves=halves)
        self.channels = 2 * qk_heads * dim + heads * vdim
        self.width = -(-(self.channels + heads) // 4) * 4
        self.columns = {"q": 0, "k": qk_heads * dim, "v": 2 * qk_heads * dim, "beta": self.channels}
        self.matrix = heads * dim * vdim
        self.state = torch.full((slots, self.matrix + (taps - 1) * self.channels), 5.0, dtype=torch.float32, device="cuda")

    def step(self, proj, second, conv, a_log, dt_bias, counts, starts, slots):
        from mini_engine_b200.csrc import ops

        tokens, sizes = proj.shape[0], dict(heads=self.heads, qk_heads=self.qk_heads, dim=self.dim, vdim=self.vdim)
        ctx = Context(counts, starts, slots)
        new = lambda *shape: torch.full(shape, float("nan"), dtype=torch.float32, device="cuda")  # noqa: E731
        qk, gv, scalars = new(tokens, self.qk_heads * 2 * self.dim), new(tokens, self.heads * (self.dim + self.vdim)), new(tokens, self.heads * 2)
        halves = lambda t: f32(torch.stack((0.25 * t, 0.75 * t)) if self.halves else t.unsqueeze(0))  # noqa: E731
        ops.delta_prepare(proj=halves(proj), columns=self.columns, second=halves(second), conv=f32(conv.T), a_log=f32(a_log),
                          dt_bias=f32(dt_bias), ctx=ctx, state=self.state, matrix=self.matrix, qk=qk, gv=gv, scalars=scalars,
                          q_scale=self.dim**-0.5, unit_eps=1e-6, **sizes)  # fmt: skip
        out = new(tokens, self.heads * self.vdim)
        ops.delta_scan(qk=qk, gv=gv, scalars=scalars, ctx=ctx, state=self.state, out=out, **sizes)
        return out.cpu()

    def matrices(self, slot):
        return self.state[slot, : self.matrix].view(self.heads, self.vdim, self.dim).transpose(1, 2).cpu()

    def plain(self, proj, second, conv, a_log, dt_bias):
        """The same from the plain functions: the projections are handed in as identities."""
        c = self.columns
        w = {"a1": torch.eye(second.shape[1], dtype=torch.float64), "a2": torch.eye(second.shape[1], dtype=torch.float64),
             "A_log": a_log, "dt_bias": dt_bias}  # fmt: skip
        eye = torch.eye(self.width + second.shape[1], dtype=torch.float64)
        spans = {"q": (0, c["k"]), "k": (c["k"], c["v"]), "v": (c["v"], c["beta"]), "b": (c["beta"], c["beta"] + self.heads)}
        for name, (a, b) in spans.items():
            w[name] = eye[a:b]
            if name != "b":
                w[name + ".conv"] = conv[a:b]
        w["a1"] = eye[self.width :]
        m = {"heads": self.heads, "kv_heads": self.qk_heads, "dim": self.dim, "vdim": self.vdim}
        out, state = plain.delta_recurrence(*plain.delta_inputs(torch.cat((proj, second), dim=1), w, "", m))
        return out.reshape(proj.shape[0], -1), state


DELTA_SIZES = [(4, 2, 16, 12, 4), (3, 1, 5, 7, 2), (2, 2, 64, 64, 3), (2, 1, 128, 40, 4), (1, 1, 192, 33, 1), (2, 2, 36, 128, 4),
               (1, 1, 260, 8, 2), (3, 3, 1, 1, 5), (5, 5, 128, 128, 4)]  # fmt: skip


@pytest.mark.parametrize("heads,qk_heads,dim,vdim,taps", DELTA_SIZES)
def test_delta_rule_whole_in_portions_and_token_by_token(heads, qk_heads, dim, vdim, taps):
    """Convolutions, unit q and k, decays from fast to almost none, the correction: whole against the plain loop; then
    portions (two tokens, one, longer) from the carried state and past inputs in a slot that held another request's, the
    same bits; then both requests side by side in one batch, one decoding while the other brings a portion."""
    g = torch.Generator().manual_seed(dim + vdim)
    run = DeltaRun(heads, qk_heads, dim, vdim, taps)
    lengths = (90, 47)
    data = [(randn(g, n, run.width), randn(g, n, heads * dim)) for n in lengths]
    conv, a_log = randn(g, run.channels, taps), torch.linspace(-7.0, 0.5, heads, dtype=torch.float64)
    dt_bias = randn(g, heads * dim)
    rest = (conv, a_log, dt_bias)
    wants = [run.plain(p, s, *rest) for p, s in data]
    whole = [run.step(p, s, *rest, [n], [0], [r]) for r, ((p, s), n) in enumerate(zip(data, lengths))]
    for r in range(2):
        close(whole[r], wants[r][0], 3e-5)
        close(run.matrices(r), wants[r][1], 3e-5)
    p, s = data[0]
    cuts = [0, 1, 3, 4, 5, 40, 42, 43, 90]
    pieces = [run.step(p[a:b], s[a:b], *rest, [b - a], [a], [3]) for a, b in zip(cuts, cuts[1:])]
    assert torch.equal(torch.cat(pieces), whole[0]) and torch.equal(run.state[3], run.state[0])
    # both at once, in other slots, the first one token by token
    got, done = [[], []], [0, 0]
    run.state[2:].fill_(-3.0)
    for counts in [(30, 2), (1, 20), (1, 1), (1, 24), (57, 0)]:
        here = [r for r in range(2) if counts[r]]
        take = lambda which: torch.cat([data[r][which][done[r] : done[r] + counts[r]] for r in here])  # noqa: E731
        out = run.step(take(0), take(1), *rest, [counts[r] for r in here], [done[r] for r in here], [2 + r for r in here])
        first = 0
        for r in here:
            got[r].append(out[first : first + counts[r]])
            first, done[r] = first + counts[r], done[r] + counts[r]
    for r in range(2):
        assert torch.equal(torch.cat(got[r]), whole[r])


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("heads,qk_heads,dim,vdim,halves", [(2, 1, 16, 40, True), (1, 1, 130, 9, False), (2, 2, 100, 128, True),
                                                            (2, 1, 64, 192, False), (3, 1, 128, 128, False)])  # fmt: skip
def test_delta_rule_over_a_long_step(taps, heads, qk_heads, dim, vdim, halves):
    """Enough tokens that a warp takes a run of them: entries that start and end inside a run, entries shorter than the
    taps, entries that go on from their past: the very bits of the same tokens in short steps."""
    g = torch.Generator().manual_seed(taps)
    run = DeltaRun(heads, qk_heads, dim, vdim, taps, slots=12, halves=halves)
    cut = [300, 1, 2, 5, 8, 260]
    starts = [20, 20, 0, 20, 0, 20]
    data = [(randn(g, 20 + n, run.width), randn(g, 20 + n, heads * dim)) for n in cut]
    rest = (randn(g, run.channels, taps), torch.linspace(-6.0, 0.5, heads, dtype=torch.float64), randn(g, heads * dim))
    wants = []
    for slot, ((p, s), first, n) in enumerate(zip(data, starts, cut)):
        if first:
            for where in (slot, slot + 6):
                run.step(p[:first], s[:first], *rest, [first], [0], [where])
        short = [run.step(p[a:b], s[a:b], *rest, [b - a], [a], [slot + 6]) for a, b in zip(range(first, first + n, 100), [*range(first + 100, first + n, 100), first + n])]
        wants.append(torch.cat(short))
    take = lambda which: torch.cat([d[which][f : f + n] for d, f, n in zip(data, starts, cut)])  # noqa: E731
    out = run.step(take(0), take(1), *rest, cut, starts, list(range(6)))
    assert torch.equal(out, torch.cat(wants)) and torch.equal(run.state[:6], run.state[6:])
    close(out[: cut[0]], run.plain(*data[0], *rest)[0][20:], 3e-5)


@pytest.mark.parametrize("dim,vdim", [(16, 8), (64, 64), (128, 96)])
def test_delta_rule_remembers_and_replaces(dim, vdim):
    """Straight into the recurrence: hardly any decay, beta near 1.  A value written under one key is read back 400 tokens
    later; written again under the same key it is replaced and not added to; a decay on that key's channel alone takes
    it away."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(dim)
    tokens = 403
    k = torch.zeros(tokens, 1, dim, dtype=torch.float64)
    k[:, 0, 2:] = randn(g, tokens, dim - 2)
    k = k / k.norm(dim=-1, keepdim=True)  # the others' keys do not touch channels 0 and 1
    for t in (0, 1, 200):  # a first value under channel 0, one under channel 1, a second one under channel 0
        k[t, 0] = 0.0
        k[t, 0, 1 if t == 1 else 0] = 1.0
    v = randn(g, tokens, 1, vdim)
    beta, decay = torch.full((tokens, 1), 1.0, dtype=torch.float64), torch.ones(tokens, 1, dim, dtype=torch.float64)
    q = k.clone()
    q[401, 0], q[402, 0] = 0.0, 0.0
    q[401, 0, 0] = q[402, 0, 1] = 1.0
    beta[401:] = 0.0  # the last two tokens only read
    for forget in (False, True):
        if forget:
            decay[300, 0, 1] = 0.25
        want, _ = plain.delta_recurrence(q, k, v, beta, decay)
        assert torch.allclose(want[401, 0], v[200, 0]) and torch.allclose(want[402, 0], v[1, 0] * (0.25 if forget else 1.0))
        out = torch.empty(tokens, vdim, dtype=torch.float32, device="cuda")
        ops.delta_scan(qk=f32(torch.cat((q, k), dim=-1)), gv=f32(torch.cat((decay, v), dim=-1)),
                       scalars=f32(torch.stack((beta, (q * k).sum(-1)), dim=-1)), ctx=Context([tokens], [0], [0]),
                       state=torch.empty(1, dim * vdim, dtype=torch.float32, device="cuda"), out=out, heads=1, qk_heads=1, dim=dim, vdim=vdim)  # fmt: skip
        close(out, want.view(tokens, vdim), 2e-5)


def test_low_rank_sums_as_two_halves():
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(4)
    proj = randn(g, 3, 6, 20)
    want = proj.float().double().sum(0)[:, 4:15]
    out = torch.empty(6, 22, dtype=torch.bfloat16, device="cuda")
    ops.split_halves(f32(proj), 4, 11, out)
    halves = out.cpu().double()
    close(halves[:, :11] + halves[:, 11:], want, 2e-5)
    close(halves[:, :11], want, 5e-3)
    whole = torch.empty(6, 11, dtype=torch.float32, device="cuda")
    ops.split_halves(f32(proj), 4, 11, whole)
    close(whole, want, 1e-6)


# ------------------------------------------------------------------------------------ routed units


def run_route(h, router, correction, spec, shared=None):
    from mini_engine_b200.csrc import ops

    tokens, held, top = h.shape[0], spec["experts"], spec["top"]
    rows = router if shared is None else torch.cat((router, shared))
    new = lambda *shape, dtype=torch.float32: torch.full(shape, -7, dtype=dtype, device="cuda")  # noqa: E731
    dense, chosen, weight = new(tokens, held), new(tokens, top, dtype=torch.int32), new(tokens, top)
    identity = new(tokens) if spec.get("identity") else None
    gate = new(tokens) if shared is not None else None
    groups = spec.get("groups") or {"count": 1, "keep": 1}
    ops.route(h=cuda(h), router=f32(rows), weights=dense, chosen=chosen, chosen_weight=weight, top=top, group_count=groups["count"],
              group_keep=groups["keep"], weight_scale=spec.get("scale", 1.0), scoring="softmax_all", correction=f32(correction),
              identity_weight=identity, shared_gate=gate)  # fmt: skip
    back = lambda t: None if t is None else t.cpu().double()  # noqa: E731
    return chosen.cpu().long(), back(weight), back(dense), back(identity), back(gate)


@pytest.mark.parametrize("experts,identity,top,groups", [(6, 2, 3, (4, 2)), (5, 0, 5, None), (1, 1, 1, None), (1, 1, 2, (2, 2)), (7, 5, 2, (3, 1)),
                                                         (60, 4, 8, (8, 3)), (300, 20, 6, (40, 4))])  # fmt: skip
def test_router_with_a_correction_groups_and_units_without_tensors(experts, identity, top, groups):
    g = torch.Generator().manual_seed(experts)
    tokens, hidden, units = 40, 44, experts + identity
    spec = {"experts": experts, "identity": identity, "top": top, "scale": 2.25, "groups": groups and {"count": groups[0], "keep": groups[1]}}
    h, router, shared = randn(g, tokens, hidden).float(), randn(g, units, hidden), randn(g, 1, hidden)
    correction = 0.3 * randn(g, units) - 0.2  # many choice scores are negative
    want, want_weight = plain.route(h.double(), {"router": router, "correction": correction}, "", spec)
    chosen, weight, dense, passed, gate = run_route(h, router, correction, spec, shared)
    assert torch.equal(chosen, want)
    close(weight, want_weight, 1e-5)
    spread = torch.zeros(tokens, units, dtype=torch.float64).scatter_(1, want, want_weight)
    close(dense, spread[:, :experts], 1e-5)
    if identity:
        assert torch.allclose(passed, spread[:, experts:].sum(-1), atol=1e-5)
    close(gate, plain.sigmoid(h.double() @ shared.T)[:, 0], 1e-5)
    if units > 2 and units > top:
        assert not torch.equal(run_route(h, router, torch.zeros(units), spec)[0], want)  # the correction decides


def test_a_long_step_routes_every_token_as_a_short_one():
    g = torch.Generator().manual_seed(9)
    spec = {"experts": 10, "identity": 2, "top": 3, "scale": 1.5, "groups": {"count": 4, "keep": 2}}
    h, router, correction, shared = randn(g, 1101, 72).float(), randn(g, 12, 72), 0.3 * randn(g, 12), randn(g, 1, 72)
    whole = run_route(h, router, correction, spec, shared)
    pieces = [run_route(h[a : a + 300], router, correction, spec, shared) for a in range(0, 1101, 300)]
    for i in range(5):
        assert torch.equal(whole[i], torch.cat([p[i] for p in pieces]))
    assert torch.equal(whole[0], plain.route(h.double(), {"router": router, "correction": correction}, "", spec)[0])


def test_units_of_other_groups_count_as_minus_infinity_and_not_zero():
    """All choice scores are negative and one group holds the best unit: the second choice comes from that group too,
    although the other group's units would be larger than what remains in it."""
    h = torch.ones(1, 4)
    router = torch.zeros(6, 4, dtype=torch.float64)  # the softmax is 1 / 6 everywhere
    correction = torch.tensor([-0.5, -5.0, -6.0, -0.6, -0.7, -0.8], dtype=torch.float64)
    spec = {"experts": 6, "top": 2, "scale": 1.0, "groups": {"count": 2, "keep": 1}}
    chosen, weight, *_ = run_route(h, router, correction, spec)
    assert chosen.tolist() == [[0, 1]] and torch.allclose(weight, torch.full((1, 2), 1 / 6, dtype=torch.float64))
    # a group is worth its best unit, not the sum of its two best: with sums the other group would win
    assert plain.route(h.double(), {"router": router, "correction": correction}, "", spec)[0].tolist() == [[0, 1]]


@pytest.mark.parametrize("kind,function", [("gelu_erf", plain.gelu_erf), ("gelu_tanh", plain.gelu_tanh)])
@pytest.mark.parametrize("units,inter", [(3, 8), (5, 7), (1, 64)])
def test_activation_of_units_side_by_side(kind, function, units, inter):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(inter)
    sums, weight = 2 * randn(g, 3, 11, units * inter), torch.rand(11, units, generator=g, dtype=torch.float64)
    weight[0] = 0.0
    want = function(sums.sum(0))
    for dtype, tolerance in ((torch.float32, 2e-6), (torch.bfloat16, 5e-3)):
        out = torch.empty(11, units * inter, dtype=dtype, device="cuda")
        ops.activation(f32(sums), out, kind)
        close(out, want, tolerance)
        ops.activation(f32(sums), out, kind, group_weight=f32(weight))
        close(out, want * weight.repeat_interleave(inter, dim=1), tolerance)
        assert not out[0].any()


@pytest.mark.parametrize("kind,function", [("gelu_erf", plain.gelu_erf), ("gelu_tanh", plain.gelu_tanh), ("relu_squared", lambda z: torch.relu(z) ** 2),
                                           ("silu", plain.silu), ("relu", torch.relu)])  # fmt: skip
@pytest.mark.parametrize("tokens,outs,inner", [(129, 200, 72), (1100, 328, 136), (2048, 6144, 64)])
def test_products_with_an_activation_in_the_epilogue(kind, function, tokens, outs, inner):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(tokens)
    x, w = randn(g, tokens, inner).to(torch.bfloat16), (2 * randn(g, outs, inner) / inner**0.5).to(torch.bfloat16)
    act = torch.full((tokens, outs), float("nan"), dtype=torch.bfloat16, device="cuda")
    ops.gemm_tensor_core_activated(ops.GemmPlan(cuda(w)), cuda(x), act, kind)
    close(act, function(x.double() @ w.double().T), 6e-3)


@pytest.mark.parametrize("activation", [None, "gelu_erf"])
def test_grouped_products_without_a_gate(activation):
    """Rows sorted by unit: units of many tiles, of one row and without any; choices that have no tensors get no row."""
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(8)
    tokens, top, units, inner, outs = 300, 2, 5, 64, 72
    chosen = torch.randint(0, 3, (tokens, top), generator=g, dtype=torch.int32)
    chosen[7, 1], chosen[:40, 0] = 4, 5  # unit 3 has no row; 5 and above are units without tensors
    capacity = -(-(tokens * top + units * 127) // 128) * 128
    new = lambda *shape: torch.empty(shape, dtype=torch.int32, device="cuda")  # noqa: E731
    row_of, token_of, block_unit = new(tokens, top), new(capacity), new(capacity // 128)
    ops.sort_by_unit(chosen=cuda(chosen), units=units, pad=128, row_of=row_of, token_of=token_of, unit_of_block=block_unit)
    assert (row_of.cpu()[chosen >= units] == -1).all() and (row_of.cpu()[chosen < units] >= 0).all()
    x, w = randn(g, tokens, inner).to(torch.bfloat16), randn(g, units, outs, inner).to(torch.bfloat16)
    rows = torch.empty(capacity, inner, dtype=torch.bfloat16, device="cuda")
    ops.gather_rows(cuda(x), token_of, rows)
    out = torch.zeros(capacity, outs, dtype=torch.float32 if activation is None else torch.bfloat16, device="cuda")
    ops.gemm_tensor_core_grouped(ops.GemmPlan(cuda(w).view(units * outs, inner)), rows, out, block_unit, outs, outs, activation=activation)
    out = out.cpu().double()
    for t in range(0, tokens, 7):
        for c in range(top):
            if int(chosen[t, c]) < units:
                want = x[t].double() @ w[int(chosen[t, c])].double().T
                want = want if activation is None else plain.gelu_erf(want)
                assert torch.allclose(out[int(row_of[t, c])], want, atol=6e-3 * float(want.abs().max()))


@pytest.mark.parametrize("width", [36, 50, 1024])
@pytest.mark.parametrize("with_identity,with_shared,with_gate", [(True, True, True), (True, False, False), (False, True, True), (False, True, False)])
def test_the_outputs_of_a_tokens_units_meet(width, with_identity, with_shared, with_gate):
    from mini_engine_b200.csrc import ops

    g = torch.Generator().manual_seed(width)
    tokens, top = 13, 3
    h, shared = randn(g, tokens, width).to(torch.bfloat16), randn(g, 2, tokens, width)
    identity, gate = randn(g, tokens), torch.rand(tokens, generator=g, dtype=torch.float64)
    identity[::3] = 0.0
    rest = torch.zeros(tokens, width, dtype=torch.float64)
    if with_identity:
        rest = rest + identity.view(-1, 1) * h.double()
    if with_shared:
        rest = rest + (gate.view(-1, 1) if with_gate else 1.0) * shared.sum(0)
    common = dict(h=cuda(h), identity_weight=f32(identity) if with_identity else None, shared=f32(shared) if with_shared else None,
                  shared_gate=f32(gate) if with_gate else None)  # fmt: skip
    out = torch.empty(tokens, width, dtype=torch.float32, device="cuda")
    routed = randn(g, 4, tokens, width)
    ops.moe_finish(out=out, routed=f32(routed), **common)
    close(out, routed.sum(0) + rest, 2e-6)
    rows, weight = randn(g, tokens * top, width), randn(g, tokens, top)
    row_of = torch.tensor(random.Random(1).sample(range(tokens * top), tokens * top), dtype=torch.int32).view(tokens, top)
    row_of[4, 0] = row_of[9, 2] = -1  # choices without a row
    want = rest.clone()
    for t in range(tokens):
        for c in range(top):
            if row_of[t, c] >= 0:
                want[t] += weight[t, c] * rows[row_of[t, c]]
    ops.moe_finish(out=out, sorted_out=f32(rows), row_of=cuda(row_of), weight=f32(weight), **common)
    close(out, want, 2e-6)
