"""Lurisun on the GPU against the plain implementation (tests/plain_lurisun.py, float64, whole sequences).

First the new kernels alone (attention with sigmoid weights and with chunks on every attention kernel; keys that are filed
as values too; the pair embedding; the input convolution; the decayed memory whole, in portions, token by token and in
chunks side by side), then every mechanism alone as a one-layer model, then whole models through the step function in
every way of cutting the work, in 32-bit and in bfloat16; then window and chunk edges and far keys made to stand out,
states that are lost on purpose, long decoding, used-again pages and slots, generation through the engine, and the programs
in bin/.
"""
import json
import os
import subprocess
import sys
import types

import numpy as np
import pytest
import torch

import helpers
import lurisun_cases as lu
import plain_lurisun as pl

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-4, "bfloat16": 4e-2}
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def _rel(a, b):
    return float((a.double().cpu() - b.double().cpu()).abs().max()) / max(float(b.double().abs().max()), 1e-30)


# ---- the kernels alone -----------------------------------------------------------------------------------------------

def _paged(keys, values, P, dtype):
    """keys [n, G, D], values [n, G, D] of ONE request filed into pages in a shuffled order; (pages, block table)."""
    n, G, D = keys.shape
    n_pages = -(-n // P)
    order = torch.randperm(n_pages + 3, generator=torch.Generator().manual_seed(n))[:n_pages]
    pages = torch.zeros(n_pages + 3, 2, G, P, D)
    for j in range(n):
        pages[order[j // P], 0, :, j % P] = keys[j]
        pages[order[j // P], 1, :, j % P] = values[j]
    return pages.to(dtype).to(DEV), order.to(torch.int32).view(1, -1).to(DEV)


def _rows_ctx(rows, table):
    """A step that holds `rows` (consecutive positions of one request), single rows as a decode step."""
    T = len(rows)
    single = T == 1
    ctx = types.SimpleNamespace(
        positions=torch.tensor(rows, dtype=torch.int32, device=DEV), row_req=torch.zeros(T, dtype=torch.int32, device=DEV),
        block_tables=[table], max_kv_len=rows[-1] + 1, n_rows=T, n_dec_rows=T if single else 0, n_pre_rows=0 if single else T,
        dec_rows=None, pre_rows=None, n_tiles=0, n_wide=0)
    if not single:
        ints = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
        ctx.pre_rows = torch.arange(T, dtype=torch.int32, device=DEV)
        tiles, wide = list(range(0, T, 64)), list(range(0, T, 128))
        ctx.tile_row0, ctx.tile_nrows, ctx.n_tiles = ints(tiles), ints([min(64, T - b) for b in tiles]), len(tiles)
        ctx.wide_row0, ctx.wide_nrows, ctx.n_wide = ints(wide), ints([min(128, T - b) for b in wide]), len(wide)
    return ctx


def _softmax_gqa(q, k, v, scale, mask):
    r = q.shape[1] // k.shape[1]
    return pl.softmax_attend(q, k.repeat_interleave(r, 1), v.repeat_interleave(r, 1), scale, mask)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,P,chunk,window,sigmoid", [
    (4, 2, 16, 4, 9, None, True), (3, 3, 32, 16, 20, None, True), (8, 2, 64, 64, 100, None, True), (4, 1, 64, 64, None, None, True),
    (4, 4, 128, 64, 130, None, True), (2, 1, 64, 64, None, 40, True), (6, 2, 24, 8, 1, None, True), (16, 1, 128, 64, 64, None, True),
    (4, 2, 256, 64, 90, None, True), (4, 2, 64, 64, 70, None, False), (6, 2, 16, 8, 33, None, False), (20, 1, 64, 64, 77, None, True),
    (8, 2, 128, 64, 128, None, False), (34, 1, 32, 16, 50, None, False)])
@pytest.mark.parametrize("fast", [True, False])
def test_attention_with_chunks_and_sigmoid_weights(dtype, H, G, D, P, chunk, window, sigmoid, fast, monkeypatch):
    """Rows of a prompt portion in the middle of a request and single decode rows, on the tensor-core kernels and on the
    generic one."""
    from kungfu_b200 import ops
    monkeypatch.setattr(ops, "use_fast_attention", fast)
    g = torch.Generator().manual_seed(H * D + (chunk or 0))
    n, tdt = 300, DTYPES[dtype]
    q, k, v = (torch.randn(n, h, D, generator=g).to(tdt).double() for h in (H, G, G))
    bias = torch.randn(H, generator=g) - 1.0
    scale = 2.0 / D ** 0.5
    mask = pl.chunk_mask(n, chunk) & pl.window_mask(n, window)
    ref = pl.sigmoid_attend(q, k, v, scale, bias, mask) if sigmoid else _softmax_gqa(q, k, v, scale, mask)
    pages, table = _paged(k, v, P, tdt)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    c = chunk or 64
    for rows in (list(range(140, 300)), [299], [150], [c * (200 // c)], [c * (200 // c) - 1], list(range(0, 70)), [5, 6]):
        out = torch.empty(len(rows), H * D, dtype=tdt, device=DEV)
        ops.paged_attention(q[rows].to(tdt).reshape(len(rows), H * D).to(DEV), out, _rows_ctx(rows, table), cache, H, G, D, scale, 0.0,
                            window, chunk=chunk, sigmoid_bias=bias.to(DEV) if sigmoid else None)
        torch.cuda.synchronize()
        ops.raise_on_device_error(torch.device(DEV))
        assert _rel(out.view(len(rows), H, D), ref[rows]) < (2e-5 if dtype == "float32" else 2e-2), (rows[0], len(rows))


@pytest.mark.parametrize("H,G,D,chunk,sigmoid", [(4, 2, 64, 900, True), (4, 1, 128, 600, True), (2, 2, 64, None, True),
                                                 (4, 4, 256, 700, True), (4, 2, 128, 800, False)])
@pytest.mark.parametrize("plan", [None, (4, 0), (3, 2), (8, 0)])
def test_long_contexts_whose_keys_are_cut_into_runs(H, G, D, chunk, sigmoid, plan, monkeypatch):
    """Short portions and single rows at a context of 1,500 tokens on the tensor-core kernels: the prompt kernel cuts a
    tile's keys into several runs (planned, and forced to 3, 4 and 8), the decode kernel into several splits; sums of
    weights that are not normalized are added up once each.  Portions that straddle a chunk's edge are among them."""
    from kungfu_b200 import ops
    monkeypatch.setattr(ops, "prefill_plan_override", plan)
    slow_before = ops.fallback_count()
    g = torch.Generator().manual_seed(H * D + (chunk or 0))
    n, P = 1500, 64
    q, k, v = (torch.randn(n, h, D, generator=g).to(torch.bfloat16).double() for h in (H, G, G))
    bias = torch.randn(H, generator=g) - 3.0
    scale = 2.0 / D ** 0.5
    mask = pl.chunk_mask(n, chunk)
    ref = pl.sigmoid_attend(q, k, v, scale, bias, mask) if sigmoid else _softmax_gqa(q, k, v, scale, mask)
    pages, table = _paged(k, v, P, torch.bfloat16)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    c = chunk or 1024
    for rows in (list(range(1400, 1437)), list(range(1100, 1400)), list(range(c - 20, c + 20)), [1499], [c], [c - 1]):
        out = torch.empty(len(rows), H * D, dtype=torch.bfloat16, device=DEV)
        ops.paged_attention(q[rows].to(torch.bfloat16).reshape(len(rows), H * D).to(DEV), out, _rows_ctx(rows, table), cache, H, G, D,
                            scale, 0.0, None, chunk=chunk, sigmoid_bias=bias.to(DEV) if sigmoid else None)
        torch.cuda.synchronize()
        ops.raise_on_device_error(torch.device(DEV))
        assert _rel(out.view(len(rows), H, D), ref[rows]) < 2e-2, (rows[0], len(rows))
    assert ops.fallback_count() == slow_before                      # every launch ran a tensor-core kernel


@pytest.mark.parametrize("level", [-60.0, -12.0, 0.0, 40.0])
def test_sigmoid_weights_of_any_size(level):
    """Scores far below and far above zero on the tensor-core kernels: weights near 0 keep their relative size down to
    2^-30, weights near 1 are 1."""
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(1)
    n, D, P = 200, 64, 64
    q, k, v = (torch.randn(n, 1, D, generator=g).to(torch.bfloat16).double() for _ in range(3))
    bias = torch.tensor([level])
    ref = pl.sigmoid_attend(q, k, v, 0.25, bias, pl.chunk_mask(n, None))
    pages, table = _paged(k, v, P, torch.bfloat16)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    for rows in (list(range(60, 200)), [199]):
        out = torch.empty(len(rows), D, dtype=torch.bfloat16, device=DEV)
        ops.paged_attention(q[rows].to(torch.bfloat16).reshape(len(rows), D).to(DEV), out, _rows_ctx(rows, table), cache, 1, 1, D, 0.25,
                            0.0, None, sigmoid_bias=bias.to(DEV))
        torch.cuda.synchronize()
        got = out.view(len(rows), 1, D).double().cpu()
        if level > -50:
            assert _rel(got, ref[rows]) < 2e-2
        else:
            assert float(got.abs().max()) < 1e-6


def _step_ctx(rows_of_reqs, slots, pad_rows=0, starts_at=None):
    """A hand-made step: request r has rows_of_reqs[r] consecutive rows from position starts_at[r] and state slot slots[r]
    (an idle request slot has 0 rows); `pad_rows` padding rows (request -1) at the end."""
    starts, row_req, pos, at = [], [], [], 0
    for r, n in enumerate(rows_of_reqs):
        starts.append(at)
        row_req += [r] * n
        pos += list(range((starts_at or [0] * 99)[r], (starts_at or [0] * 99)[r] + n))
        at += n
    row_req += [-1] * pad_rows
    pos += [0] * pad_rows
    bufs = {}
    ints = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    return types.SimpleNamespace(
        n_reqs=len(rows_of_reqs), n_rows=len(row_req), row_req=ints(row_req), positions=ints(pos), req_row_start=ints(starts),
        req_n_rows=ints(rows_of_reqs), req_state_slot=ints(slots), decode_only=max(rows_of_reqs) == 1,
        buf=lambda tag, shape, dt: bufs.setdefault((tag, tuple(shape), dt), torch.empty(shape, dtype=dt, device=DEV)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,rows", [(64, [5, 1, 0, 3]), (30, [1, 1, 1, 1]), (1536, [2, 40, 1, 7])])
def test_pair_embedding(dtype, W, rows):
    """Requests at their first token and in the middle, an idle slot, padding rows; factors beyond 32 bits together."""
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(W)
    V, buckets, mp, mc = 50000, 997, 1000003, 65537
    table, pair = (torch.randn(n, W, generator=g).to(DTYPES[dtype]) for n in (V, buckets + 1))
    slots, starts = [2, 0, 1, 3], [0, 17, 0, 5]
    prev = torch.tensor([[49999], [1], [7], [31234]], dtype=torch.int32)
    T = sum(rows)
    tokens = torch.randint(0, V, (T + 2,), generator=g, dtype=torch.int32)
    want, after, at = [], prev.clone(), 0
    for r, n in enumerate(rows):
        before = int(prev[slots[r], 0])
        for i in range(n):
            tok = int(tokens[at])
            b = buckets if starts[r] + i == 0 else (before * mp + tok * mc) % buckets
            want.append(table[tok].double() * 1.5 + pair[b].double())
            before, at = tok, at + 1
        if n:
            after[slots[r], 0] = before
    dev_prev, out = prev.to(DEV), torch.full((T + 2, W), 9.0, device=DEV)
    ops.embed_pair(tokens.to(DEV), table.to(DEV), pair.to(DEV), 1.5, mp, mc, dev_prev, out, _step_ctx(rows, slots, 2, starts))
    torch.cuda.synchronize()
    assert _rel(out[:T], torch.stack(want)) < 1e-6 and float(out[T:].abs().max()) == 0.0
    assert torch.equal(dev_prev.cpu(), after)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6, 8])
@pytest.mark.parametrize("W", [64, 30, 2048])
def test_input_convolution_in_portions(dtype, taps, W):
    """Requests of unequal length fed in portions of changing size (1 to 700 rows, several requests per step, with
    padding rows): the result does not depend on how they are cut; steps of single rows also run the kernel that does the
    residual sum and the convolution together."""
    from kungfu_b200 import ops
    tdt = DTYPES[dtype]
    tol = 1e-5 if dtype == "float32" else 1e-2
    g = torch.Generator().manual_seed(taps * W)
    lengths = [40, 900, 9]
    h = [torch.randn(n, W, generator=g) for n in lengths]
    w = (0.5 * torch.randn(W, taps, generator=g)).to(tdt)
    ref = [pl.input_convolution(x.double(), w) for x in h]
    state = torch.zeros(4, max(taps - 1, 1), W, device=DEV)
    slots, done, step = [3, 0, 2], [0, 0, 0], 0
    sizes = ([1, 2, 1], [2, 1, 3], [3, 700, 1], [1, 1, 1], [5, 90, 1], [20, 2, 2])
    while min(d - n for d, n in zip(done, lengths)) < 0:
        rows = [min(s, n - d) for s, n, d in zip(sizes[step % len(sizes)], lengths, done)]
        step += 1
        x = torch.cat([h[r][done[r]:done[r] + n] for r, n in enumerate(rows)] + [torch.ones(2, W)])
        ctx = _step_ctx(rows, slots, 2)
        out = torch.zeros(x.shape[0], W, dtype=tdt, device=DEV)
        single = max(rows) == 1
        if single:
            branch, weight = torch.randn(x.shape[0], W, generator=g), (1.0 + 0.2 * torch.randn(W, generator=g)).to(tdt)
            res = x - (pl.rms(branch.double(), 1e-5) * weight.double()).float()
            res_dev = res.to(DEV)
            ran = ops.add_rmsnorm_conv(branch.to(DEV), weight.to(DEV), 1e-5, res_dev, w.to(DEV), state if taps > 1 else None, out, ctx)
            assert ran == (taps <= 4)
            if ran:
                assert _rel(res_dev, x) < 1e-5
        if not single or taps > 4:
            ops.input_conv(x.to(DEV), w.to(DEV), state if taps > 1 else None, out, ctx)
        torch.cuda.synchronize()
        at = 0
        for r, n in enumerate(rows):
            if n:
                assert _rel(out[at:at + n], ref[r][done[r]:done[r] + n]) < tol, (step, r, n)
            at += n
            done[r] += n
    assert float(state[1].abs().max()) == 0.0


def _memory_reference(q, k, v, decay, S):
    """The plain recurrence from a state: (results, state after)."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=torch.float64)
    S = S.clone().double()
    a = torch.tensor(decay, dtype=torch.float64)[:, None, None]
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


@pytest.mark.parametrize("kind", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,dv", [(2, 8, 12), (3, 40, 50), (1, 4, 6), (4, 64, 64), (2, 128, 32), (1, 200, 24), (2, 6, 7), (2, 256, 40),
                                    (5, 96, 72), (3, 128, 128)])
def test_decayed_memory_from_earlier_states(kind, H, d, dv, monkeypatch):
    """Requests with earlier tokens in their states and a fresh one, an idle request slot and padding rows: results and
    states after a step of unequal portions, after the same rows one by one, and (bfloat16) after the same step with
    every way of walking chunks.  float32: raw projections, the activation applied inside."""
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(H * d + dv)
    rows, slots = [700, 1, 0, 130, 64], [2, 0, -1, 3, 1]
    T = sum(rows)
    width = 2 * H * d + H * dv
    ld = width + (-width) % 8
    raw = torch.randn(T + 2, ld, generator=g)
    act = "silu" if kind == "float32" else None
    if kind == "bfloat16":
        raw = pl.silu(raw).to(torch.bfloat16)
    used = pl.silu(raw.double()) if act else raw.double()
    decay = [1.0, 0.0, 0.97, 0.5, 0.9995][:H] if H > 1 else [0.99]
    S0 = torch.randn(4, H, d, dv, generator=g)
    S0[3] = 0.0
    powers = ops.decay_powers(decay).to(DEV)
    q0, k0, v0 = 0, H * d, 2 * H * d

    def check(S, out, tol):
        at = 0
        for r, n in enumerate(rows):
            if n == 0:
                continue
            x = used[at:at + n]
            ref, after = _memory_reference(x[:, q0:k0].view(n, H, d), x[:, k0:v0].view(n, H, d), x[:, v0:width].view(n, H, dv), decay,
                                           S0[slots[r]])
            assert _rel(out[at:at + n].view(n, H, dv), ref) < tol, r
            assert _rel(S[slots[r]], after) < tol, r
            at += n

    ways = [dict(decay_chunks=False)] if kind == "float32" else [dict(decay_chunks=False), dict(decay_chunks=True), dict(use_tensor_cores=True)]
    for way in ways:
        for name, value in way.items():
            monkeypatch.setattr(ops, name, value)
        S, out = S0.clone().to(DEV), torch.zeros(T + 2, H * dv, device=DEV)
        ops.decay_memory(raw.to(DEV), q0, k0, v0, act, powers, S, out, H, d, dv, _step_ctx(rows, slots, 2))
        torch.cuda.synchronize()
        check(S, out, 1e-4)
        assert float(out[T:].abs().max()) == 0.0
    if kind == "bfloat16":
        wide = raw.float()                                     # decoding reads 32-bit rows in the engine; here both
    S, out = S0.clone().to(DEV), torch.zeros(T, H * dv, device=DEV)
    starts = [sum(rows[:r]) for r in range(5)]
    for step in range(max(rows)):
        live = [r for r in range(5) if step < rows[r]]
        pick = torch.tensor([starts[r] + step for r in live])
        o = torch.zeros(len(live), H * dv, device=DEV)
        src = raw if (kind == "float32" or step % 2) else wide
        ops.decay_memory(src[pick].contiguous().to(DEV), q0, k0, v0, act, powers, S, o, H, d, dv,
                         _step_ctx([1] * len(live), [slots[r] for r in live]))
        out[pick.to(DEV)] = o
    torch.cuda.synchronize()
    check(S, out, 1e-4)


def test_decayed_memory_chunks_side_by_side_run_and_leave_the_state(monkeypatch):
    """One long prompt of few heads: the step is cut into chunks (three launches), also when its length is a multiple of
    the chunk, one more, or one less; `writes` off leaves the state as it was."""
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(3)
    H, d, dv, decay = 2, 64, 64, [0.999, 0.9]
    powers = ops.decay_powers(decay).to(DEV)
    for n in (512, 513, 767, 768, 1100):
        raw = pl.silu(torch.randn(n, H * (2 * d + dv), generator=g)).to(torch.bfloat16)
        S0 = torch.randn(2, H, d, dv, generator=g)
        x = raw.double()
        ref, after = _memory_reference(x[:, :H * d].view(n, H, d), x[:, H * d:2 * H * d].view(n, H, d), x[:, 2 * H * d:].view(n, H, dv),
                                       decay, S0[1])
        for writes in (True, False):
            S, out = S0.clone().to(DEV), torch.zeros(n, H * dv, device=DEV)
            before = ops.launch_count()
            ops.decay_memory(raw.to(DEV), 0, H * d, 2 * H * d, None, powers, S, out, H, d, dv, _step_ctx([n], [1]), writes=writes)
            assert ops.launch_count() - before == 3
            torch.cuda.synchronize()
            assert _rel(out.view(n, H, dv), ref) < 1e-4 and _rel(S[1], after if writes else S0[1]) < 1e-4
            assert torch.equal(S[0].cpu(), S0[0])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("nh,nkv,dk,rot,P", [(4, 2, 16, 8, 4), (3, 3, 8, 8, 8), (8, 2, 64, 32, 64), (2, 1, 20, 0, 16), (4, 4, 128, 128, 64)])
def test_keys_as_projected_are_filed_as_values(dtype, nh, nkv, dk, rot, P):
    """q|k with biases -> norms over the whole projections and rotation for queries and keys; the values are the biased
    keys, neither normed nor turned.  Two requests in the middle of their sequences and a padding row."""
    from kungfu_b200 import ops
    tdt = DTYPES[dtype]
    tol = 1e-5 if dtype == "float32" else 1e-2
    g = torch.Generator().manual_seed(nh * dk)
    positions, row_req = [5, 6, 7, 8, 9, 10, 11, 30, 0], [0] * 7 + [1, -1]
    T, D, C = len(positions), ops.attention_head_size(dk), (nh + nkv) * dk
    proj = torch.randn(T, C + (-C) % 4, generator=g)
    bias = (0.3 * torch.randn(C, generator=g)).to(tdt)
    wq, wk = ((1 + 0.3 * torch.randn(n * dk, generator=g)).to(tdt) for n in (nh, nkv))
    pos = torch.tensor(positions)
    half = 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    ang = pos.double()[:, None] * half[None, :]
    table = torch.arange(2 * (40 // P + 2), dtype=torch.int32).view(2, -1).flip(1).contiguous().to(DEV)
    ctx = types.SimpleNamespace(positions=pos.to(torch.int32).to(DEV), row_req=torch.tensor(row_req, dtype=torch.int32, device=DEV), block_tables=[table])
    x = proj[:, :C].double() + bias.double()
    q = pl.rotate_halves((pl.rms(x[:, :nh * dk], 1e-5) * wq.double()).view(T, nh, dk), pos, 50.0, rot)
    k = pl.rotate_halves((pl.rms(x[:, nh * dk:], 1e-5) * wk.double()).view(T, nkv, dk), pos, 50.0, rot)
    v = x[:, nh * dk:].view(T, nkv, dk)
    pages = torch.full((table.numel(), 2, nkv, P, D), 7.0, dtype=tdt, device=DEV)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    q_out = torch.full((T, nh * D), 7.0, dtype=tdt, device=DEV)
    ops.rownorm_rope_append(proj.to(DEV), 0, bias.to(DEV), wq.to(DEV), wk.to(DEV), 1e-5, torch.cos(ang).float().to(DEV) if rot else None,
                            torch.sin(ang).float().to(DEV) if rot else None, rot, False, 1.0, nh, nkv, dk, dk, ctx, cache, q_out,
                            values_are_keys=True)
    torch.cuda.synchronize()
    assert _rel(q_out.view(T, nh, D)[:8, :, :dk], q[:8]) < tol and float(q_out[8].abs().max()) == 0.0
    for t in range(8):
        page = int(table[row_req[t], positions[t] // P])
        kk, vv = pages[page, 0, :, positions[t] % P], pages[page, 1, :, positions[t] % P]
        assert _rel(kk[:, :dk], k[t]) < tol and _rel(vv[:, :dk], v[t]) < tol
        if D > dk:
            assert float(kk[:, dk:].abs().max()) == 0.0 and float(vv[:, dk:].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,n", [(3, 511), (5, 512), (2, 1030), (3, 4096), (2, 6000)])
def test_norm_over_all_heads_and_gate(dtype, T, n):
    from kungfu_b200 import ops
    tdt = DTYPES[dtype]
    g = torch.Generator().manual_seed(n)
    o, gate = torch.randn(T, n, generator=g), torch.randn(T, n + 8, generator=g)
    w = (1 + 0.3 * torch.randn(n, generator=g)).to(tdt)
    out = torch.empty(T, n, dtype=tdt, device=DEV)
    ops.head_norm_gate(o.to(DEV), w.to(DEV), 1e-5, gate.to(DEV), 8, "sigmoid", out, 1, n)
    ref = pl.rms(o.double(), 1e-5) * w.double() * torch.sigmoid(gate[:, 8:].double())
    assert _rel(out, ref) < (1e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,n,col0", [(1, 5, 0), (3, 35, 7), (7, 64, 12), (300, 2048, 256)])
def test_gate_per_element(dtype, T, n, col0):
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(n)
    x, gate = torch.randn(T, n, generator=g).to(DTYPES[dtype]), torch.randn(T, col0 + n + 4, generator=g)
    out = torch.empty(T, n, dtype=DTYPES[dtype], device=DEV)
    ops.element_gate(x.to(DEV), gate.to(DEV), col0, out)
    ref = x.double() * torch.sigmoid(gate[:, col0:col0 + n].double())
    assert _rel(out, ref) < (1e-6 if dtype == "float32" else 5e-3)


# ---- models ------------------------------------------------------------------------------------------------------------

def _runner(folder, dtype, page, max_tokens, max_requests=4, graphs=True, ctx=2048):
    from kungfu_b200 import api
    cfg, model = api.load_model(folder, dtype=dtype, device=DEV)
    return api.make_runner(cfg, model, dtype=dtype, device=DEV, page_size=page, max_tokens=max_tokens,
                           max_requests=max_requests, max_context=ctx, cuda_graphs=graphs)


def _plain(cfg, tensors, toks):
    """(exact logits, logits with the plain implementation rounding to bfloat16 where a 16-bit path may), both float32."""
    exact = pl.forward(cfg, tensors, toks).float()
    with pl.rounded_to_bfloat16():
        return exact, pl.forward(cfg, tensors, toks).float()


def _quantiles(errs):
    errs = sorted(errs)
    n = len(errs)
    return errs[n // 2], errs[min(n - 1, (n * 19) // 20)], errs[-1]


def _check(got, ref, tol, noisy=None):
    """32-bit: the largest difference of any logit against the largest logit, below `tol` at every place.  bfloat16: the
    yardstick is the model itself: `noisy` holds the plain implementation's logits with its 16-bit roundings switched on.
    The median of the framework's per-place errors must stay within twice the yardstick's, the 95th percentile and the
    largest error within three times, with a floor of tol / 8."""
    assert got
    if tol < 1e-2:
        scale = max(float(r.abs().max()) for r in ref.values())
        worst = max(float((row - ref[rid][pos]).abs().max()) for (rid, pos), row in got.items()) / scale
        assert worst < tol, f"rel err {worst:.3e}"
        return
    assert noisy is not None
    rel = lambda a, b: float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt())
    mine = _quantiles([rel(row, ref[rid][pos]) for (rid, pos), row in got.items()])
    yard = _quantiles([rel(noisy[rid][pos], ref[rid][pos]) for (rid, pos) in got])
    for m, y, what, factor in zip(mine, yard, ("median", "95 %", "largest"), (2.0, 3.0, 3.0)):
        assert m < max(factor * y, tol / 8), f"rel err {what} {m:.3e}, rounding alone {y:.3e}"


ONE_LAYER = {
    "chunks": lu.config(64, 200, [lu.layer("attention", lu.attention(4, 2, 16, 0.3, chunk=37, rot_dims=8, base=100.0))]),
    "chunks_wide": lu.config(128, 200, [lu.layer("attention", lu.attention(6, 2, 64, 0.1, chunk=70, rot_dims=64))]),
    "no_mask": lu.config(64, 200, [lu.layer("attention", lu.attention(3, 1, 40, 0.2, rot_dims=2))]),
    "many_heads": lu.config(64, 200, [lu.layer("attention", lu.attention(18, 1, 16, 0.3, chunk=50))]),
    "lightning": lu.config(64, 200, [lu.layer("lightning", lu.lightning(3, 8, 12, [0.99, 0.5, 0.999]))]),
    "lightning_wide": lu.config(128, 200, [lu.layer("lightning", lu.lightning(2, 128, 64, [0.995, 0.9]))]),
    "lightning_odd": lu.config(64, 200, [lu.layer("lightning", lu.lightning(2, 9, 5, [0.9, 0.7]))]),
    "latent": lu.config(64, 200, [lu.layer("latent_attention", lu.latent(3, 8, 6, 20, 12, 0.4, window=29))]),
    "latent_wide": lu.config(256, 200, [lu.layer("latent_attention", lu.latent(20, 32, 24, 100, 48, 0.15, window=66))]),
    # a latent whose stored head is above the largest the tensor-core kernels take: the generic kernel in both element types
    "latent_huge": lu.config(128, 200, [lu.layer("latent_attention", lu.latent(2, 16, 12, 290, 20, 0.2, window=40))]),
    "dense": lu.config(64, 200, [lu.layer("attention", lu.attention(1, 1, 8, 0.5), 88)], logit_scale=0.3),
    "taps": lu.config(64, 200, [lu.layer("lightning", lu.lightning(1, 8, 8, [0.0]), 24)], taps=8),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mechanism_alone_as_a_one_layer_model(which, dtype, tmp_path):
    cfg = ONE_LAYER[which]
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=7, sharp=1.5)
    reqs = {"a": helpers.random_tokens(150, cfg["vocab"], 1), "b": helpers.random_tokens(9, cfg["vocab"], 2)}
    tensors = helpers.read_tensors(folder)
    both = {rid: _plain(cfg, tensors, toks) for rid, toks in reqs.items()}
    ref, noisy = {r: b[0] for r, b in both.items()}, {r: b[1] for r, b in both.items()}
    for steps in (helpers.trace_whole(reqs), helpers.trace_chunks(reqs), helpers.trace_decode_tail(reqs, 8)):
        runner = _runner(folder, dtype, 64, helpers.trace_max_tokens(steps, 64))
        _check(helpers.run_trace_with_runner(runner, steps), ref, TOL[dtype], noisy)


def test_residual_after_every_layer(tmp_path):
    """The 32-bit residual stream after each layer against the plain one."""
    from kungfu_b200.engine import StepEntry
    cfg = lu.LU_A
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=11)
    toks = helpers.random_tokens(40, cfg["vocab"], 3)
    after = []
    pl.forward(cfg, helpers.read_tensors(folder), toks, after)
    runner = _runner(folder, "float32", 4, 64, graphs=False)
    runner.cache.add_request("a")
    kept = []
    runner.model.after_layer = lambda i, x: kept.append(x[:len(toks)].detach().clone())
    try:
        runner.step([StepEntry("a", toks, [len(toks) - 1])])
    finally:
        runner.model.after_layer = None
    assert len(kept) == len(after)
    for i, x in enumerate(kept):
        assert x.dtype == torch.float32 and _rel(x, after[i]) < 1e-4, i


NOISY = {}          # per model of the fixture below: request -> the plain implementation's logits with 16-bit roundings


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    cases = dict(lu.CASES)
    cases["E"] = (lu.LU_E, [3, 130, 64, 270, 65, 17], 64)
    for name, (cfg, lengths, page) in cases.items():
        folder = lu.write_model(str(tmp_path_factory.mktemp(name) / "m"), cfg, seed=21)
        reqs = {f"r{i}": helpers.random_tokens(n, cfg["vocab"], 300 + i) for i, n in enumerate(lengths)}
        tensors = helpers.read_tensors(folder)
        both = {rid: _plain(cfg, tensors, toks) for rid, toks in reqs.items()}
        out[name] = (folder, cfg, reqs, {r: b[0] for r, b in both.items()}, page)
        NOISY[name] = {r: b[1] for r, b in both.items()}
    return out


def _steps(mode, reqs):
    return {"whole": helpers.trace_whole, "tail": lambda r: helpers.trace_decode_tail(r, 32),
            "chunks": helpers.trace_chunks, "mixed": lambda r: helpers.trace_mixed(r, seed=5)}[mode](reqs)


@pytest.mark.parametrize("name", ["A", "B", "C", "D", "E"])
@pytest.mark.parametrize("mode", ["whole", "tail", "chunks", "mixed"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_modes_match_plain(models, name, mode, dtype):
    """Whole prompts, most of a prompt then token by token, portions of 2 to 11 tokens, and mixed batches of up to four
    unequal requests with pools so small that pages and state slots are used again."""
    from kungfu_b200 import ops
    folder, cfg, reqs, ref, page = models[name]
    steps = _steps(mode, reqs)
    runner = _runner(folder, dtype, page, helpers.trace_max_tokens(steps, page))
    got = helpers.run_trace_with_runner(runner, steps)
    assert len(got) == sum(len(t) for t in reqs.values())
    _check(got, ref, TOL[dtype], NOISY[name])
    ops.raise_on_device_error(torch.device(DEV))
    assert runner.cache.n_live == 0
    if mode == "mixed":
        assert any(n > g.pool.n_pages for n, g in zip(runner.cache.pages_handed_out(), runner.cache.groups))
        assert len(reqs) > runner.cache.max_requests           # state slots served more requests than there are slots


@pytest.mark.parametrize("name,page", [("A", 4), ("E", 64)])
def test_batch_of_unequal_requests_equals_each_alone(models, name, page):
    """32-bit: the logits of a request must not depend on what else is in its step."""
    from kungfu_b200.engine import StepEntry
    folder, cfg, reqs, ref, _ = models[name]
    runner = _runner(folder, "float32", page, 1024, graphs=False)
    alone = {}
    for rid, toks in reqs.items():
        runner.cache.add_request(rid)
        alone[rid] = runner.step([StepEntry(rid, toks, [len(toks) - 1])])[0].clone()
        runner.cache.release(rid)
    some = list(reqs)[:4]
    for rid in some:
        runner.cache.add_request(rid)
    together = runner.step([StepEntry(rid, reqs[rid], [len(reqs[rid]) - 1]) for rid in some]).clone()
    for i, rid in enumerate(some):
        scale = float(ref[rid].abs().max())
        assert float((together[i] - alone[rid]).abs().max()) / scale < 2e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B", "E"])
def test_long_decoding_from_captured_graphs(models, name, dtype):
    """A short prompt and then 300 tokens one by one (the decode steps replay from a CUDA graph after the second); the
    windows and chunks of both models pass over decoded tokens only, and the memories carry their state all the way."""
    folder, cfg, _, _, page = models[name]
    toks = helpers.random_tokens(310, cfg["vocab"], 9)
    exact, noisy = _plain(cfg, helpers.read_tensors(folder), toks)
    steps = helpers.trace_decode_tail({"a": toks}, 300)
    runner = _runner(folder, dtype, page, 384)
    got = helpers.run_trace_with_runner(runner, steps)
    _check(got, {"a": exact}, TOL[dtype], {"a": noisy})
    assert any(s.get("graph") is not None for s in runner._graphs.values())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_walks_its_chunks_side_by_side(dtype, tmp_path):
    """700 tokens whole, then in two portions and a tail: long enough for the memories' chunks to be walked side by side
    and for the prompt attention's keys to fill several tiles."""
    cfg = lu.config(128, 120, [lu.layer("lightning", lu.lightning(2, 64, 64, [0.999, 0.95]), 64),
                               lu.layer("attention", lu.attention(2, 1, 64, 0.15, chunk=300, rot_dims=32), 64)], taps=4)
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=2)
    toks = helpers.random_tokens(700, 120, 5)
    exact, noisy = _plain(cfg, helpers.read_tensors(folder), toks)
    for sizes in ((700,), (560, 130, 1, 2, 7)):
        steps = helpers.trace_chunks({"a": toks}, sizes=sizes)
        runner = _runner(folder, dtype, 64, 768)
        _check(helpers.run_trace_with_runner(runner, steps), {"a": exact}, TOL[dtype], {"a": noisy})


def _echo_model(folder, kind, reach, seed):
    """A one-layer model without a feed-forward in which token 250 + 2k + 1 "calls" token 250 + 2k: the keys' matrix is
    the queries' matrix behind a fixed shuffle of the input's elements and the caller's embedding is the callee's
    shuffled the same way, so the caller's query equals the callee's key and meets it with the largest score there is.
    The convolution and the pair table are zero, so a token is its embedding alone.  `kind` 'chunks': sigmoid weights with
    a bias that leaves every other key next to nothing; 'window': the latent mixer with a scale that makes its softmax sharp."""
    if kind == "chunks":
        cfg = lu.config(64, 300, [lu.layer("attention", lu.attention(2, 2, 32, 0.5, chunk=reach, rot_dims=8))])
    else:
        cfg = lu.config(64, 300, [lu.layer("latent_attention", lu.latent(2, 32, 16, 48, 48, 0.7, window=reach))])
    t, p = lu.draw_tensors(cfg, seed), "l0.mix."
    shuffle = torch.cat([torch.roll(torch.arange(32), 5), 32 + torch.roll(torch.arange(32), 11)])
    a, b = ("q", "k") if kind == "chunks" else ("dq", "dkv")
    t[p + b] = torch.zeros_like(t[p + a])
    t[p + b][:, shuffle] = t[p + a]                                  # W_k h = W_q (h taken in shuffled order)
    for n in (a + ".norm", b + ".norm"):
        t[p + n] = torch.ones_like(t[p + n])
    if kind == "chunks":
        for n in ("q.b", "k.b"):
            t[p + n] = torch.zeros_like(t[p + n])
        t[p + "pb"] = torch.full_like(t[p + "pb"], -11.0)
    else:
        t[p + "uk"] = t[p + "uq"].clone()
    t["l0.canon1"], t["bigram"] = torch.zeros_like(t["l0.canon1"]), torch.zeros_like(t["bigram"])
    for callee in range(250, 300, 2):
        t["embed"][callee][shuffle] = t["embed"][callee + 1]         # the callee's row, shuffled, is the caller's
    lu.write_tensors(folder, cfg, t)
    return cfg, t


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,reach", [("window", 40), ("window", 64), ("window", 129), ("chunks", 40), ("chunks", 64), ("chunks", 100)])
def test_keys_at_window_and_chunk_edges_stand_out(kind, reach, dtype, tmp_path):
    """Pairs of a callee and its caller are planted just inside and just outside: `reach - 1` and `reach` apart for a
    window; for chunks at the first and last place of one chunk (seen), and at the last place of a chunk and the first of
    the next (not seen, though they are neighbours), in the prompt and among the tokens decoded one by one, at page
    borders too.  The plain implementation itself shows that each planted key decides its row or does not touch it."""
    folder = str(tmp_path / "m")
    cfg, tensors = _echo_model(folder, kind, reach, seed=3)
    n = 6 * reach + 150
    toks = [t % 250 for t in helpers.random_tokens(n, 250, 5)]
    plants = []                                   # (callee's place, caller's place, seen?)
    if kind == "chunks":
        c = reach
        wanted = [(0, c - 1, True), (c, 2 * c - 2, True), (2 * c - 1, 2 * c, False), (2 * c + 1, 3 * c - 1, True), (3 * c - 2, 3 * c + 1, False),
                  (4 * c, 5 * c - 1, True), (5 * c, 6 * c - 1, True), (6 * c - 2, 6 * c, False)]
    else:
        wanted, at = [], 2
        for k in range(10):
            wanted.append((at, at + (reach - 1 if k % 2 == 0 else reach), k % 2 == 0))
            at += reach // 2 + 7 + (62 - at % 64 if k == 3 else 0)     # one plant starts right before a page border
    for k, (callee, caller, seen) in enumerate(wanted):
        if caller < n and not any({callee, caller} & set(p[:2]) for p in plants):
            toks[callee], toks[caller] = 250 + 2 * k, 251 + 2 * k
            plants.append((callee, caller, seen))
    assert sum(p[2] for p in plants) >= 3 and sum(not p[2] for p in plants) >= 3
    ref = pl.forward(cfg, tensors, toks)
    scale = float(ref.abs().max())
    for first, second, seen in plants:
        moved = list(toks)
        moved[first] = 7
        delta = float((pl.forward(cfg, tensors, moved)[second] - ref[second]).abs().max()) / scale
        assert (delta > 0.05) if seen else (delta == 0.0), (first, second, seen, delta)
    noisy = _plain(cfg, tensors, toks)[1]
    middle = sorted(p[0] for p in plants)[len(plants) // 2]
    tail = n - (middle + 1)                                    # decoding starts between the two of a middle plant
    reqs = {"a": toks}
    for steps in (helpers.trace_whole(reqs), helpers.trace_decode_tail(reqs, tail), helpers.trace_chunks(reqs)):
        runner = _runner(folder, dtype, 64, helpers.trace_max_tokens(steps, 64))
        got = helpers.run_trace_with_runner(runner, steps)
        _check(got, {"a": ref.float()}, TOL[dtype], {"a": noisy})
        for first, second, seen in plants:
            assert float((got[("a", second)] - ref[second].float()).abs().max()) / scale < TOL[dtype], (first, second, seen)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["chunks", "window"])
def test_a_key_hundreds_of_tokens_back_carries_the_row(kind, dtype, tmp_path):
    """A reach of 1,000 tokens: a callee at place 3 (and others at page borders) and its caller 500 to 700 places later, in
    the prompt and in decoding.  Losing that one key among hundreds changes the row by far more than the tolerance."""
    folder = str(tmp_path / "m")
    cfg, tensors = _echo_model(folder, kind, 1000, seed=4)
    n = 720
    toks = [t % 250 for t in helpers.random_tokens(n, 250, 6)]
    plants = [(3, 520), (63, 600), (64, 655), (0, 700), (128, 719)]
    for k, (a, b) in enumerate(plants):
        toks[a], toks[b] = 250 + 2 * k, 251 + 2 * k
    ref = pl.forward(cfg, tensors, toks)
    scale = float(ref.abs().max())
    for a, b in plants:
        moved = list(toks)
        moved[a] = 7
        assert float((pl.forward(cfg, tensors, moved)[b] - ref[b]).abs().max()) / scale > 0.05
    reqs = {"a": toks}
    noisy = _plain(cfg, tensors, toks)[1]
    for steps in (helpers.trace_whole(reqs), helpers.trace_decode_tail(reqs, 130), helpers.trace_chunks(reqs, sizes=(97, 2, 130, 31))):
        runner = _runner(folder, dtype, 64, helpers.trace_max_tokens(steps, 64))
        got = helpers.run_trace_with_runner(runner, steps)
        _check(got, {"a": ref.float()}, TOL[dtype], {"a": noisy})
        for a, b in plants:
            assert float((got[("a", b)] - ref[b].float()).abs().max()) / scale < TOL[dtype], (a, b)


def test_states_are_carried_and_a_lost_one_shows(tmp_path):
    """A memory with decays near one: the first token still moves the row 300 tokens later (the plain implementation says
    by how much), through portions and single tokens.  Zeroing the memory, the convolution's tail or the token before
    between two steps moves the next logits by far more than the tolerance."""
    from kungfu_b200.engine import StepEntry
    cfg = lu.config(64, 200, [lu.layer("lightning", lu.lightning(2, 16, 16, [0.9995, 0.999]))])
    folder = lu.write_model(str(tmp_path / "m"), cfg, seed=8)
    t = helpers.read_tensors(folder)
    toks = helpers.random_tokens(320, 200, 4)
    ref = pl.forward(cfg, t, toks)
    scale = float(ref.abs().max())
    moved = list(toks)
    moved[0] = (toks[0] + 1) % 200
    assert float((pl.forward(cfg, t, moved)[300:] - ref[300:]).abs().max()) / scale > 2e-3
    for steps in (helpers.trace_whole({"a": toks}), helpers.trace_decode_tail({"a": toks}, 40), helpers.trace_chunks({"a": toks})):
        runner = _runner(folder, "float32", 64, 384)
        _check(helpers.run_trace_with_runner(runner, steps), {"a": ref.float()}, TOL["float32"])
    for which in ("memory", "tail", "token", None):
        for n_next in (1, 5):                                    # the fused decode kernel, and the portion's kernel
            runner = _runner(folder, "float32", 64, 384, graphs=False)
            runner.cache.add_request("a")
            runner.step([StepEntry("a", toks[:200], [])])
            memory, tail = runner.cache.storage[0]
            store = {"memory": memory, "tail": tail, "token": runner.cache.storage[1]}.get(which)
            if store is not None:
                store.zero_()
            out = runner.step([StepEntry("a", toks[200:200 + n_next], [0])])
            err = float((out[0].cpu() - ref[200].float()).abs().max()) / scale
            assert (err > 20 * TOL["float32"]) if which else (err < TOL["float32"]), (which, n_next, err)


def test_pages_and_slots_of_finished_requests_are_used_again_and_start_clean(models):
    """Small pools and ONE state slot: requests follow one another through the same pages and the same slot of the
    memories, tails and tokens; each is cut in two portions, the first of two tokens."""
    from kungfu_b200.engine import StepEntry
    folder, cfg, reqs, ref, page = models["B"]
    runner = _runner(folder, "float32", page, 2 * 64, max_requests=1, graphs=False)
    for rid in ("r3", "r2", "r5", "r3"):
        toks = reqs[rid]
        runner.cache.add_request(rid)
        a = runner.step([StepEntry(rid, toks[:2], [0, 1])]).cpu()
        b = runner.step([StepEntry(rid, toks[2:], [len(toks) - 3])]).cpu()
        runner.cache.release(rid)
        scale = float(ref[rid].abs().max())
        assert float((a[0] - ref[rid][0]).abs().max()) / scale < TOL["float32"]
        assert float((a[1] - ref[rid][1]).abs().max()) / scale < TOL["float32"]
        assert float((b[0] - ref[rid][len(toks) - 1]).abs().max()) / scale < TOL["float32"]
    assert any(n > g.pool.n_pages for n, g in zip(runner.cache.pages_handed_out(), runner.cache.groups))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_generate_through_the_entry_point(models, dtype):
    """Greedy generation through Engine (scheduler, portions under a token budget, tokens drawn on the device, graphs)
    against the plain implementation's best token at every place, near ties aside."""
    import kungfu_b200
    from kungfu_b200.sampling import Sampling
    folder, cfg, reqs, _, page = models["E"]
    tensors = helpers.read_tensors(folder)
    eng = kungfu_b200.Engine(folder, dtype=dtype, device=DEV, ctx=512, batch=64, parallel=4, page_size=page,
                             max_tokens_in_cache=1024)
    prompts = [reqs["r1"], reqs["r0"], reqs["r4"], reqs["r5"], reqs["r2"]]
    outs = eng.generate(prompts, Sampling(temperature=0.0), max_tokens=12, ignore_eos=True)
    margin = 1e-3 if dtype == "float32" else 5e-2
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        logits = pl.forward(cfg, tensors, list(p) + list(o))[len(p) - 1:-1]      # one pass: every place sees what was drawn
        top = torch.topk(logits, 2, dim=-1).values
        for i, tok in enumerate(o):
            if float(top[i, 0] - top[i, 1]) > margin * float(logits[i].abs().max()):
                assert int(torch.argmax(logits[i])) == tok, i


def test_programs_in_bin(models, tmp_path):
    """bin/trace_run replays a trace of a Lurisun folder; bin/kungfu inspects the folder, completes a prompt and times
    the model."""
    folder, cfg, reqs, ref, page = models["A"]
    steps = helpers.trace_mixed(reqs, seed=2)
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", str(helpers.trace_max_tokens(steps, 64))],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=900)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    at = {rid: 0 for rid in reqs}
    scale = max(float(r.abs().max()) for r in ref.values())
    for s in steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        k = 0
        for e in s["entries"]:
            for w in e["want"]:
                assert float(np.abs(rows[k] - ref[e["id"]][at[e["id"]] + w].numpy()).max()) / scale < TOL["float32"]
                k += 1
            at[e["id"]] += len(e["tokens"])
    kungfu = os.path.join(ROOT, "bin", "kungfu")
    p = subprocess.run([sys.executable, kungfu, "inspect", folder, "--json"], capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    doc = json.loads(p.stdout)
    assert doc["architecture"] == "Lurisun" and doc["layers"] == 3 and not doc["missing"] and not doc["unexpected"]
    assert len(doc["states"]) == 3
    p = subprocess.run([sys.executable, kungfu, "generate", "--model", folder, "--ids", json.dumps(reqs["r1"]), "--max-tokens", "5",
                        "--dtype", "float32", "--ignore-eos", "--ctx", "256"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    gen = json.loads(p.stdout.strip().splitlines()[-1])["generated"]
    assert len(gen) == 5
    seq = list(reqs["r1"]) + gen
    logits = pl.forward(cfg, helpers.read_tensors(folder), seq)[len(reqs["r1"]) - 1:-1]
    top = torch.topk(logits, 2, dim=-1).values
    for i, tok in enumerate(gen):
        if float(top[i, 0] - top[i, 1]) > 1e-3 * float(logits[i].abs().max()):
            assert int(torch.argmax(logits[i])) == tok
    p = subprocess.run([sys.executable, kungfu, "bench", "--model", folder, "--pp", "40", "--tg", "6", "--reps", "1", "--ctx", "256"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
