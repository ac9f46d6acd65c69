"""Fovosun on the GPU against the plain implementation (tests/plain_fovosun.py, float64, whole sequences).

First the new kernels alone (the streams' update and reading; the preparation of queries and keys of two maps, whole, in
portions and row by row; both maps on every attention kernel and their difference; the router whose winners share a
softmax; turned queries and keys of the decayed memory), then every mechanism alone as a one-layer model, then whole
models through the step function in every way of cutting the work, in 32-bit and in bfloat16; then window edges and far
keys made to stand out, states that are lost on purpose, long decoding, used-again pages and slots, generation through the
engine, and the programs in bin/.
"""
import json
import os
import subprocess
import sys
import types

import numpy as np
import pytest
import torch

import fovosun_cases as fo
import helpers
import plain_fovosun as pl

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
@pytest.mark.parametrize("n,W,T", [(1, 64, 3), (2, 30, 5), (3, 328, 200), (4, 2048, 40), (5, 101, 2), (6, 96, 7), (7, 64, 4), (8, 512, 9),
                                   (16, 36, 5), (11, 7, 3), (3, 4100, 2)])
def test_streams_update_and_reading(dtype, n, W, T):
    """The update alone, the update with the next sublayer's reading, and the reading alone of some rows."""
    from kungfu_b200 import ops
    tdt = DTYPES[dtype]
    tol = 1e-5 if dtype == "float32" else 6e-3
    g = torch.Generator().manual_seed(n * W)
    x, y = torch.randn(T, n, W, generator=g), torch.randn(T, W, generator=g)
    mix, out_w, in_w = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
    w = (1 + 0.3 * torch.randn(W, generator=g)).to(tdt)
    want = pl.scatter_streams(x.double().transpose(0, 1), y.double(), mix, out_w)
    normed = pl.rms(pl.gather_streams(want, in_w), 1e-5) * w.double()
    for nxt in (False, True):
        dev, out = x.to(DEV), torch.full((T, W), 9.0, dtype=tdt, device=DEV)
        kw = dict(next_weights=in_w.to(DEV), next_norm=w.to(DEV), next_eps=1e-5, next_out=out) if nxt else {}
        ops.streams_step(dev, y.to(DEV), mix.to(DEV), out_w.to(DEV), **kw)
        torch.cuda.synchronize()
        assert _rel(dev.transpose(0, 1), want) < 1e-5
        if nxt:
            assert _rel(out, normed) < tol
    rows = [T - 1, 0, T // 2]
    out = torch.empty(3, W, dtype=tdt, device=DEV)
    ops.streams_norm(x.to(DEV), in_w.to(DEV), w.to(DEV), 1e-5, out, torch.tensor(rows, dtype=torch.int32, device=DEV))
    ref = pl.rms(pl.gather_streams(x.double().transpose(0, 1), in_w), 1e-5) * w.double()
    assert _rel(out, ref[rows]) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_embedding_starts_every_stream(dtype):
    from kungfu_b200 import ops
    table = torch.randn(50, 36, generator=torch.Generator().manual_seed(1)).to(DTYPES[dtype])
    toks = [3, 49, 0, 3]
    out = torch.empty(4, 5, 36, device=DEV)
    ops.embed(torch.tensor(toks, dtype=torch.int32, device=DEV), table.to(DEV), 1.75, out)
    assert _rel(out, (table.double()[toks] * 1.75)[:, None, :].expand(4, 5, 36)) < 1e-6


MAP_SHAPES = [  # H, G, d, dv, taps, rot, temperature, biased, page
    (6, 2, 32, 64, 3, 0, (0.6, 16), False, 64), (5, 1, 32, 48, 0, 32, None, True, 64), (2, 2, 8, 20, 4, 8, (0.3, 1), True, 8),
    (6, 3, 16, 16, 2, 8, None, False, 16), (3, 1, 9, 7, 3, 4, (1.1, 3), True, 4), (2, 1, 64, 128, 4, 64, (0.4, 100), False, 64),
    (1, 1, 104, 40, 1, 16, None, False, 64), (2, 2, 136, 100, 3, 136, (0.2, 7), True, 64), (2, 1, 6, 30, 8, 2, None, False, 16),
    (4, 4, 20, 12, 5, 16, (0.7, 9), True, 32), (2, 1, 24, 300, 2, 12, None, False, 16)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("lengths,sizes", [([37, 25], [(1, 2), (5, 1), (1, 1), (1, 1), (2, 9), (1, 1), (11, 3)]),
                                           ([690, 205], [(1, 2), (550, 7), (1, 1), (3, 190), (9, 2)])])
@pytest.mark.parametrize("H,G,d,dv,taps,rot,temp,biased,P", MAP_SHAPES)
def test_queries_and_keys_of_two_maps_in_portions(dtype, H, G, d, dv, taps, rot, temp, biased, P, lengths, sizes):
    """Two requests fed in portions of changing size (single rows also move the convolution's tail in the same kernel where
    they can): every query row is its map's query in its own half and zero elsewhere, the stored key is both maps side by
    side, the value is filed once, tails are zero, and a padding row leaves nothing."""
    from kungfu_b200 import ops
    from kungfu_b200.parts.latent import latent_head_size
    tdt = DTYPES[dtype]
    tol = 2e-5 if dtype == "float32" else 1e-2
    g = torch.Generator().manual_seed(H * d + dv + taps)
    C, D = 2 * (H + G) * d + G * dv, latent_head_size(max(2 * d, dv))
    ld = C + (-C) % 4
    slots = [2, 0]
    raw = [torch.randn(n, ld, generator=g) for n in lengths]
    bias = (0.4 * torch.randn(C, generator=g)).to(tdt) if biased else None
    conv = (0.6 * torch.randn(C, taps, generator=g)).to(tdt) if taps else None
    want = []
    for x in raw:
        u = x[:, :C].double() + (bias.double() if biased else 0.0)
        u = pl.causal_convolution(u, conv) if taps else u
        n, pos = u.shape[0], torch.arange(u.shape[0])
        q, k = u[:, :2 * H * d].reshape(n, 2 * H, d), u[:, 2 * H * d:2 * (H + G) * d].reshape(n, 2 * G, d)
        q, k = pl.rotate_halves(q, pos, 50.0, rot), pl.rotate_halves(k, pos, 50.0, rot)
        if temp:
            q = q * pl.temperature(pos, *temp)[:, None, None]
        wide = torch.zeros(n, H, 2, D, dtype=torch.float64)
        for m in (0, 1):
            wide[:, :, m, m * d:(m + 1) * d] = q.view(n, H, 2, d)[:, :, m]
        want.append((wide.view(n, 2 * H, D), k.reshape(n, G, 2 * d), u[:, 2 * (H + G) * d:].reshape(n, G, dv)))
    table = torch.arange(2 * (max(lengths) // P + 2), dtype=torch.int32).view(2, -1).flip(1).contiguous()
    pages = torch.full((table.numel(), 2, G, P, D), 7.0, dtype=tdt, device=DEV)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    state = torch.zeros(3, max(taps - 1, 1), C, device=DEV)
    half = 50.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1))
    done, step, inline_seen = [0, 0], 0, False
    while min(a - b for a, b in zip(done, lengths)) < 0:
        rows = [min(s, n - a) for s, n, a in zip(sizes[step % len(sizes)], lengths, done)]
        step += 1
        x = torch.cat([raw[r][done[r]:done[r] + n] for r, n in enumerate(rows)] + [torch.ones(1, ld)])
        ctx = _step_ctx(rows, slots, 1, done)
        ctx.block_tables = [table.to(DEV)]
        ang = ctx.positions.cpu().double()[:, None] * half[None, :]
        cos, sin = (f(ang).float().to(DEV) if rot else None for f in (torch.cos, torch.sin))
        q = torch.full((x.shape[0], 2 * H * D), 7.0, dtype=tdt, device=DEV)
        proj = x.to(DEV)
        moved = ops.qkv_prepare(proj, 0, bias.to(DEV) if biased else None, conv.to(DEV) if taps else None, state if taps > 1 else None,
                                None, None, 1e-5, cos, sin, rot, False, H, G, d, dv, ctx, cache, q, commit_inline=max(rows) == 1,
                                parts=2, temperature=temp)
        inline_seen = inline_seen or moved
        if taps > 1 and not moved:
            ops.short_conv_commit(proj, 0, bias.to(DEV) if biased else None, C, taps, state, ctx, w_dtype=tdt)
        torch.cuda.synchronize()
        at = 0
        for r, n in enumerate(rows):
            if n:
                assert _rel(q[at:at + n].view(n, 2 * H, D), want[r][0][done[r]:done[r] + n]) < tol, (step, r)
                zero = (want[r][0][done[r]:done[r] + n] == 0).to(DEV)
                assert float((q[at:at + n].view(n, 2 * H, D).float() * zero).abs().max()) == 0.0
            at += n
            done[r] += n
        assert float(q[at:].abs().max()) == 0.0
    pages = pages.cpu()
    for r, n in enumerate(lengths):
        at = torch.arange(n)
        kk, vv = (pages[table[r, at // P].long(), i, :, at % P] for i in (0, 1))
        assert _rel(kk[..., :2 * d], want[r][1]) < tol and _rel(vv[..., :dv], want[r][2]) < tol, r
        assert float(kk[..., 2 * d:].abs().sum()) == 0.0 and float(vv[..., dv:].abs().sum()) == 0.0
    assert inline_seen == (taps > 1 and d % 4 == 0 and dv % 4 == 0 and rot % 8 == 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("interleaved,rot,norm", [(False, 16, True), (True, 16, True), (False, 0, False), (False, 4, True)])
def test_preparation_of_one_map_with_norms(dtype, interleaved, rot, norm):
    """The same kernels for ordinary heads: norms per head, both pairings, on vectors of four and element by element."""
    from kungfu_b200 import ops
    tdt = DTYPES[dtype]
    g = torch.Generator().manual_seed(rot)
    H, G, d, dv, T, P = 3, 1, 24, 16, 11, 16
    C = (H + G) * d + G * dv
    x, wq, wk = torch.randn(T, C, generator=g), *((1 + 0.3 * torch.randn(d, generator=g)).to(tdt) for _ in range(2))
    ctx = _step_ctx([T], [0], 0, [5])
    ctx.block_tables = [torch.tensor([[1, 0]], dtype=torch.int32, device=DEV)]
    pos = torch.arange(5, 5 + T)
    q, k = x[:, :H * d].double().view(T, H, d), x[:, H * d:(H + G) * d].double().view(T, G, d)
    if norm:
        q, k = pl.rms(q, 1e-5) * wq.double(), pl.rms(k, 1e-5) * wk.double()
    perm = torch.arange(d)
    if interleaved:                                          # pairs (2i, 2i + 1) are halves of a reordered head
        perm[:rot] = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])
    back = torch.argsort(perm)
    q, k = (pl.rotate_halves(t[..., perm], pos, 50.0, rot)[..., back] for t in (q, k))
    ang = pos.double()[:, None] * (50.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1)))[None, :]
    pages = torch.zeros(2, 2, G, P, 32, dtype=tdt, device=DEV)
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    out = torch.empty(T, H * 32, dtype=tdt, device=DEV)
    ops.qkv_prepare(x.to(DEV), 0, None, None, None, wq.to(DEV) if norm else None, wk.to(DEV) if norm else None, 1e-5,
                    torch.cos(ang).float().to(DEV) if rot else None, torch.sin(ang).float().to(DEV) if rot else None, rot, interleaved,
                    H, G, d, dv, ctx, cache, out)
    tol = 2e-5 if dtype == "float32" else 1e-2
    assert _rel(out.view(T, H, 32)[..., :d], q) < tol
    stored = torch.stack([pages[1 if p < P else 0, 0, :, p % P, :d] for p in pos.tolist()])
    assert _rel(stored, k) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv,P,window", [(6, 2, 32, 64, 64, None), (5, 1, 32, 48, 64, 70), (8, 1, 16, 24, 16, 33), (9, 1, 64, 128, 64, 40),
                                               (2, 2, 64, 40, 64, 1), (3, 3, 10, 30, 8, None), (2, 1, 128, 256, 64, 100), (2, 1, 140, 60, 64, 50)])
@pytest.mark.parametrize("fast", [True, False])
def test_both_maps_on_the_attention_kernels_and_their_difference(dtype, H, G, d, dv, P, window, fast, monkeypatch):
    """Portions in the middle of a request and single rows; groups of up to 18 query rows per key head."""
    from kungfu_b200 import ops
    from kungfu_b200.parts.latent import latent_head_size
    monkeypatch.setattr(ops, "use_fast_attention", fast)
    g = torch.Generator().manual_seed(H * d + dv)
    n, tdt, D = 300, DTYPES[dtype], latent_head_size(max(2 * d, dv))
    q, k = torch.randn(n, H, 2, d, generator=g).to(tdt).double(), torch.randn(n, G, 2, d, generator=g).to(tdt).double()
    v, gate = torch.randn(n, G, dv, generator=g).to(tdt).double(), torch.randn(n, H + 3, generator=g)
    scale, lam, diff = 2.0 / d ** 0.5, 0.63, 0.35
    mask = pl.window_mask(n, window)
    maps = [pl.softmax_attend(q[:, :, m], k[:, :, m], v, scale, mask) for m in (0, 1)]
    pad = lambda t: torch.nn.functional.pad(t, (0, D - t.shape[-1]))
    pages, table = _paged(pad(k.reshape(n, G, 2 * d)), pad(v), P, tdt)
    wide = torch.zeros(n, H, 2, D, dtype=torch.float64)
    for m in (0, 1):
        wide[:, :, m, m * d:(m + 1) * d] = q[:, :, m]
    cache = types.SimpleNamespace(pages=pages, page_size=P, group=0, writes=True)
    for rows in (list(range(140, 300)), [299], [150], list(range(0, 70)), [5, 6], [0]):
        T, ctx = len(rows), _rows_ctx(rows, table)
        o = torch.empty(T, 2 * H * D, dtype=tdt, device=DEV)
        ops.paged_attention(wide[rows].reshape(T, 2 * H * D).to(tdt).to(DEV), o, ctx, cache, 2 * H, G, D, scale, 0.0, window)
        torch.cuda.synchronize()
        ops.raise_on_device_error(torch.device(DEV))
        got = o.view(T, H, 2, D)[..., :dv]
        for m in (0, 1):
            assert _rel(got[:, :, m], maps[m][rows]) < (2e-5 if dtype == "float32" else 2e-2), (rows[0], T, m)
        exact = got.double().cpu()
        for gated in (True, False):
            out = torch.empty(T, H * dv, dtype=tdt, device=DEV)
            ops.diff_combine(o, lam, 1.0 - diff, 1e-5, gate[rows].to(DEV) if gated else None, 2, H, dv, D, out, ctx)
            ref = pl.difference(exact[:, :, 0], exact[:, :, 1], lam, diff, 1e-5)
            if gated:
                ref = ref * torch.sigmoid(gate[rows, 2:2 + H].double())[:, :, None]
            assert _rel(out.view(T, H, dv), ref) < (1e-5 if dtype == "float32" else 6e-3)
    ctx.row_req = ctx.row_req - 1                              # a row of padding leaves zeros
    ops.diff_combine(o, lam, 1.0, 1e-5, None, 0, H, dv, D, out, ctx)
    assert float(out.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,top", [(1, 1, 1), (5, 8, 2), (9, 40, 40), (130, 64, 6), (3, 1000, 33)])
def test_router_whose_winners_share_a_softmax(dtype, T, E, top):
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(E)
    z = 3.0 * torch.randn(T, E, generator=g)
    z[0] += 200.0                                              # far from zero: nothing overflows
    b = torch.randn(E, generator=g).to(DTYPES[dtype])
    for bias in (b, None):
        ids, w = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
        ops.moe_route(z.to(DEV), bias.to(DEV) if bias is not None else None, 1, 1, top, 1.5, ids, w, score="softmax_chosen")
        biased = z + (bias.float() if bias is not None else 0.0)
        for t, row in enumerate(pl.route(biased.double(), top)):
            assert ids[t].tolist() == [e for e, _ in row]
            assert max(abs(a - 1.5 * x) for a, (_, x) in zip(w[t].tolist(), row)) < 1e-5


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


@pytest.mark.parametrize("H,d,dv,rot", [(2, 8, 12, 8), (3, 40, 50, 24), (1, 4, 6, 2), (4, 64, 64, 64), (2, 128, 32, 64), (2, 6, 7, 4),
                                        (2, 256, 40, 128), (3, 128, 128, 128), (2, 16, 16, 0), (2, 48, 8, 12)])
def test_turned_queries_and_keys_of_the_memory(H, d, dv, rot):
    """Requests in the middle of their sequences, an idle slot, padding rows: turned as 32-bit rows are read (portions, and
    row by row), and turned beforehand into bfloat16 rows for the tensor cores; results and states."""
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(H * d + dv + rot)
    rows, slots, starts = [150, 1, 0, 70], [2, 0, -1, 1], [0, 17, 0, 301]
    T, width = sum(rows), 2 * H * d + H * dv
    g0 = 8                                                     # q, k, v start behind other columns
    raw = torch.randn(T + 2, g0 + width + (-width) % 4, generator=g)
    decay = [0.97, 0.5, 0.9995, 1.0][:H]
    S0 = torch.randn(3, H, d, dv, generator=g)
    powers = ops.decay_powers(decay).to(DEV)
    q0, k0, v0 = g0, g0 + H * d, g0 + 2 * H * d
    ctx = _step_ctx(rows, slots, 2, starts)
    pos = ctx.positions.cpu()
    ang = pos.double()[:, None] * (70.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / max(rot, 1)))[None, :]
    cos, sin = (f(ang).float().to(DEV) if rot else None for f in (torch.cos, torch.sin))
    x = raw.double()
    q = pl.rotate_halves(x[:, q0:k0].reshape(-1, H, d), pos, 70.0, rot)
    k = pl.rotate_halves(x[:, k0:v0].reshape(-1, H, d), pos, 70.0, rot) * d ** -0.5
    v = x[:, v0:g0 + width].reshape(-1, H, dv)

    def check(S, out, q, k, v, tol):
        at = 0
        for r, n in enumerate(rows):
            if n:
                ref, after = _memory_reference(q[at:at + n], k[at:at + n], v[at:at + n], decay, S0[slots[r]])
                assert _rel(out[at:at + n].view(n, H, dv), ref) < tol and _rel(S[slots[r]], after) < tol, r
            at += n

    turn = dict(cos=cos, sin=sin, rot=rot, key_scale=d ** -0.5)
    S, out = S0.clone().to(DEV), torch.zeros(T + 2, H * dv, device=DEV)
    ops.decay_memory(raw.to(DEV), q0, k0, v0, None, powers, S, out, H, d, dv, ctx, **turn)
    torch.cuda.synchronize()
    check(S, out, q, k, v, 1e-4)
    assert float(out[T:].abs().max()) == 0.0
    S, out = S0.clone().to(DEV), torch.zeros(T, H * dv, device=DEV)
    begin = [sum(rows[:r]) for r in range(4)]
    for step in range(max(rows)):
        live = [r for r in range(4) if step < rows[r]]
        pick = torch.tensor([begin[r] + step for r in live])
        o = torch.zeros(len(live), H * dv, device=DEV)
        t = dict(turn, cos=cos[pick.to(DEV)].contiguous(), sin=sin[pick.to(DEV)].contiguous()) if rot else turn
        ops.decay_memory(raw[pick].contiguous().to(DEV), q0, k0, v0, None, powers, S, o, H, d, dv,
                         _step_ctx([1] * len(live), [slots[r] for r in live]), **t)
        out[pick.to(DEV)] = o
    torch.cuda.synchronize()
    check(S, out, q, k, v, 1e-4)
    packed = torch.zeros(T + 2, width, dtype=torch.bfloat16, device=DEV)
    ops.decay_rotate(raw.to(DEV), q0, k0, v0, cos, sin, rot, d ** -0.5, H, d, dv, packed)
    want = torch.cat([t.reshape(T + 2, -1) for t in (q, k, v)], dim=1)
    assert _rel(packed, want) < 5e-3
    if ops.decay_memory_takes_bfloat16(d, dv, width):
        S, out = S0.clone().to(DEV), torch.zeros(T + 2, H * dv, device=DEV)
        ops.decay_memory(packed, 0, H * d, 2 * H * d, None, powers, S, out, H, d, dv, ctx)
        torch.cuda.synchronize()
        p = packed.double().cpu()
        check(S, out, p[:, :H * d].view(-1, H, d), p[:, H * d:2 * H * d].view(-1, H, d), p[:, 2 * H * d:].view(-1, H, dv), 1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dv", [(3, 20), (2, 600), (4, 64)])
def test_head_norm_without_a_weight(dtype, H, dv):
    from kungfu_b200 import ops
    g = torch.Generator().manual_seed(dv)
    o, gate = torch.randn(6, H * dv, generator=g), torch.randn(6, H * dv + 4, generator=g)
    out = torch.empty(6, H * dv, dtype=DTYPES[dtype], device=DEV)
    ops.head_norm_gate(o.to(DEV), None, 1e-5, gate.to(DEV), 4, "silu", out, H, dv)
    z = gate[:, 4:].double()
    ref = pl.rms(o.double().view(6, H, dv), 1e-5).view(6, -1) * z * torch.sigmoid(z)
    assert _rel(out, ref) < (1e-5 if dtype == "float32" else 6e-3)


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
    "plain_maps": fo.config(64, 200, [fo.layer("attention_2", fo.attention(4, 2, 12, 16, 0.4))]),
    "window": fo.config(64, 200, [fo.layer("attention_2", fo.attention(4, 4, 32, 64, 0.3, window=37, rot=(100.0, 16)))], streams=1),
    "conv_temperature": fo.config(64, 200, [fo.layer("attention", fo.attention(6, 2, 32, 64, 0.2, conv=4, temp=(0.6, 9)))], streams=4),
    "many_heads": fo.config(64, 200, [fo.layer("attention_2", fo.attention(10, 1, 8, 16, 0.5, window=50, rot=(10.0, 8)))]),
    "taps": fo.config(64, 200, [fo.layer("attention", fo.attention(1, 1, 9, 8, 0.5, conv=8, temp=(0.2, 1)))], streams=2),
    "wide_maps": fo.config(128, 200, [fo.layer("attention", fo.attention(2, 1, 128, 200, 0.1, conv=2, temp=(0.3, 64)))]),
    # a stored head above the largest the tensor-core kernels take: the generic kernel in both element types
    "huge_maps": fo.config(64, 200, [fo.layer("attention_2", fo.attention(2, 1, 144, 20, 0.08, window=90, rot=(1000.0, 144)))]),
    "retention": fo.config(64, 200, [fo.layer("retention", fo.retention(3, 8, 12, [0.99, 0.5, 0.999], rot=(20.0, 8)))]),
    "retention_wide": fo.config(128, 200, [fo.layer("retention", fo.retention(2, 128, 64, [0.995, 0.9], rot=(1000.0, 64)))]),
    "retention_odd": fo.config(64, 200, [fo.layer("retention", fo.retention(2, 9, 5, [0.9, 0.7], rot=(50.0, 6)))], streams=5),
    "dense": fo.config(64, 200, [fo.layer("retention", fo.retention(1, 8, 8, [0.0]), fo.dense(88, 0.5))], scale=3.0),
    "mixture": fo.config(64, 200, [fo.layer("retention", fo.retention(1, 8, 8, [0.9]), fo.moe(12, 3, 40, 0.7, (56, 1.4)))]),
    "one_expert": fo.config(64, 200, [fo.layer("retention", fo.retention(1, 8, 8, [0.9]), fo.moe(6, 1, 32, 1.0))], streams=9),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mechanism_alone_as_a_one_layer_model(which, dtype, tmp_path):
    cfg = ONE_LAYER[which]
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=7, sharp=1.5)
    reqs = {"a": helpers.random_tokens(150, cfg["vocab"], 1), "b": helpers.random_tokens(9, cfg["vocab"], 2)}
    tensors = helpers.read_tensors(folder)
    both = {rid: _plain(cfg, tensors, toks) for rid, toks in reqs.items()}
    ref, noisy = {r: b[0] for r, b in both.items()}, {r: b[1] for r, b in both.items()}
    for steps in (helpers.trace_whole(reqs), helpers.trace_chunks(reqs), helpers.trace_decode_tail(reqs, 8)):
        runner = _runner(folder, dtype, 64, helpers.trace_max_tokens(steps, 64))
        _check(helpers.run_trace_with_runner(runner, steps), ref, TOL[dtype], noisy)


def test_residual_after_every_layer(tmp_path):
    """The sum of the 32-bit streams after each layer against the plain one."""
    from kungfu_b200.engine import StepEntry
    cfg = fo.FO_A
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=11)
    toks = helpers.random_tokens(40, cfg["vocab"], 3)
    after = []
    pl.forward(cfg, helpers.read_tensors(folder), toks, after)
    runner = _runner(folder, "float32", 4, 64, graphs=False)
    runner.cache.add_request("a")
    kept = []
    runner.model.after_layer = lambda i, x: kept.append(x[:len(toks)].sum(1))
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
    cases = dict(fo.CASES)
    cases["E"] = (fo.FO_E, [3, 130, 64, 270, 65, 17], 64)
    for name, (cfg, lengths, page) in cases.items():
        folder = fo.write_model(str(tmp_path_factory.mktemp(name) / "m"), cfg, seed=21)
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
    windows of both models pass over decoded tokens only, and the memories carry their state all the way."""
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
    cfg = fo.config(128, 120, [fo.layer("retention", fo.retention(2, 64, 64, [0.999, 0.95], rot=(10000.0, 64)), fo.dense(64)),
                               fo.layer("attention", fo.attention(2, 1, 32, 64, 0.2, conv=4, temp=(0.4, 128)), fo.moe(4, 2, 64))])
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=2)
    toks = helpers.random_tokens(700, 120, 5)
    exact, noisy = _plain(cfg, helpers.read_tensors(folder), toks)
    for sizes in ((700,), (560, 130, 1, 2, 7)):
        steps = helpers.trace_chunks({"a": toks}, sizes=sizes)
        runner = _runner(folder, dtype, 64, 768)
        _check(helpers.run_trace_with_runner(runner, steps), {"a": exact}, TOL[dtype], {"a": noisy})


def _echo_model(folder, window, seed):
    """A one-layer model without a feed-forward in which token 250 + 2k + 1 "calls" token 250 + 2k: the keys' matrix is
    the queries' matrix behind a fixed shuffle of the input's elements and the callee's embedding is the caller's
    shuffled the same way, so the caller's queries equal the callee's keys in both maps and meet them with the largest
    score there is.  With a window: the biased mixer (biases zero), a part of each map turned; without: the mixer with a
    convolution (which passes the current token alone) and a temperature."""
    if window:
        cfg = fo.config(64, 300, [fo.layer("attention_2", fo.attention(2, 2, 32, 64, 0.6, diff=0.3, window=window, rot=(1e6, 8)))])
    else:
        cfg = fo.config(64, 300, [fo.layer("attention", fo.attention(2, 2, 32, 64, 0.6, diff=0.3, conv=3, temp=(0.1, 100)))])
    t, p = fo.draw_tensors(cfg, seed), "l0.mix."
    shuffle = torch.cat([torch.roll(torch.arange(32), 5), 32 + torch.roll(torch.arange(32), 11)])
    t[p + "k"] = torch.zeros_like(t[p + "q"])
    t[p + "k"][:, shuffle] = t[p + "q"]                              # W_k h = W_q (h taken in shuffled order)
    for n in ("q", "k", "v"):
        if window:
            t[p + n + ".b"] = torch.zeros_like(t[p + n + ".b"])
        else:
            t[p + n + ".conv"] = torch.zeros_like(t[p + n + ".conv"])
            t[p + n + ".conv"][:, -1] = 1.0
    for n in ("lq1", "lk1", "lq2", "lk2"):
        t[p + n] = torch.zeros_like(t[p + n])
    t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
    for callee in range(250, 300, 2):
        t["embed"][callee][shuffle] = t["embed"][callee + 1]         # the callee's row, shuffled, is the caller's
    fo.write_tensors(folder, cfg, t)
    return cfg, t


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("reach", [40, 64, 129])
def test_keys_at_window_edges_stand_out(reach, dtype, tmp_path):
    """Pairs of a callee and its caller are planted `reach - 1` apart (seen) and `reach` apart (not seen), in the prompt
    and among the tokens decoded one by one, at page borders too.  The plain implementation itself shows that each planted
    key decides its row or does not touch it."""
    folder = str(tmp_path / "m")
    cfg, tensors = _echo_model(folder, reach, seed=3)
    n = 6 * reach + 150
    toks = [t % 250 for t in helpers.random_tokens(n, 250, 5)]
    plants, at = [], 2                            # (callee's place, caller's place, seen?)
    for k in range(10):
        callee, caller, seen = at, at + (reach - 1 if k % 2 == 0 else reach), k % 2 == 0
        at += reach // 2 + 7 + (62 - at % 64 if k == 3 else 0)         # one plant starts right before a page border
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
@pytest.mark.parametrize("window", [1000, None])
def test_a_key_hundreds_of_tokens_back_carries_the_row(window, dtype, tmp_path):
    """A window of 1,000 tokens, and none: a callee at place 3 (and others at page borders) and its caller 500 to 700 places later, in
    the prompt and in decoding.  Losing that one key among hundreds changes the row by far more than the tolerance."""
    folder = str(tmp_path / "m")
    cfg, tensors = _echo_model(folder, window, seed=4)
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
    by how much), through portions and single tokens.  Zeroing the memory or the convolution's tail between two steps moves
    the next logits by far more than the tolerance."""
    from kungfu_b200.engine import StepEntry
    cfg = fo.config(64, 200, [fo.layer("retention", fo.retention(2, 16, 16, [0.9995, 0.999], rot=(1e5, 8))),
                              fo.layer("attention", fo.attention(2, 1, 16, 32, 0.3, conv=4, temp=(0.4, 30)))])
    folder = fo.write_model(str(tmp_path / "m"), cfg, seed=8)
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
    for which in ("memory", "tail", None):
        for n_next in (1, 5):                                    # the fused decode kernel, and the portion's kernel
            runner = _runner(folder, "float32", 64, 384, graphs=False)
            runner.cache.add_request("a")
            runner.step([StepEntry("a", toks[:200], [])])
            store = {"memory": runner.cache.storage[0], "tail": runner.cache.storage[1]}.get(which)
            if which == "memory":
                (store[0] if isinstance(store, (list, tuple)) else store).zero_()
            elif which == "tail":
                store[1].zero_()
            out = runner.step([StepEntry("a", toks[200:200 + n_next], [0])])
            err = float((out[0].cpu() - ref[200].float()).abs().max()) / scale
            assert (err > 20 * TOL["float32"]) if which else (err < TOL["float32"]), (which, n_next, err)


def test_pages_and_slots_of_finished_requests_are_used_again_and_start_clean(models):
    """Small pools and ONE state slot: requests follow one another through the same pages and the same slot of the
    memories and tails; each is cut in two portions, the first of two tokens."""
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
    """bin/trace_run replays a trace of a Fovosun folder; bin/kungfu inspects the folder, completes a prompt and times
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
    assert doc["architecture"] == "Fovosun" and doc["layers"] == 3 and not doc["missing"] and not doc["unexpected"]
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
