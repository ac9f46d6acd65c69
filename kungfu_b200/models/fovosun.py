"""Fovosun put together from parts.

A Fovosun model keeps several streams of the residual (`parts.StreamsEmbedding`, `parts.StreamsBlock`): every sublayer reads
a weighted sum of them, normed, and its result is mixed into all of them.  A layer's mixer is one of
  attention    differential attention without positions in the scores: a convolution over q, k and v, queries whose
               temperature grows with the position, a gate per head (`parts.DifferentialAttention`);
  attention_2  differential attention with biased projections, rotary pairs (i, i + dims/2) in each map and a sliding
               window (`parts.DifferentialAttention`);
  retention    linear attention with one fixed decay per head, rotated queries and keys, every head normed, a silu gate
               (`parts.LightningAttention` with its options).
The feed-forward is a clamped gated one, a mixture of such experts whose router has a bias and whose winners are weighted
by the softmax over their own logits, with a shared expert (`parts.RoutedExperts`), or absent.  The output is the norm of
the streams' sum and an untied matrix.
Tensor names are those of a Fovosun safetensors file: `embed`, `l<i>.norm1|norm2`, `l<i>.hc1|hc2.in|out|mix`, `l<i>.mix.*`
(attention: q, k, v, q.conv, k.conv, v.conv, lq1, lk1, lq2, lk2, g, o; attention_2: q, q.b, k, k.b, v, v.b, lq1, lk1, lq2,
lk2, o; retention: q, k, v, g, o), `l<i>.mlp.gate|up|down` or `l<i>.mlp.router`, `l<i>.mlp.router.b`,
`l<i>.mlp.e<j>|shared.gate|up|down`, `final.norm`, `head`.
"""
from __future__ import annotations

import torch

from ..config.fovosun import ATTENTION, BIASED_ATTENTION, RETENTION, FovosunConfig
from ..parts import (DecoderModel, DifferentialAttention, GatedFfn, LightningAttention, LmHead, RmsNorm, Rope, RoutedExperts,
                     ShortConv, StreamsBlock, StreamsEmbedding, StreamsMix, StreamsNorm)
from ..weights.store import TensorSpec, WeightStore

MATRIX_STD = 0.02
CONV_STD = 0.3
LAMBDA = ("lq1", "lk1", "lq2", "lk2")


def _attention_rows(m) -> tuple:
    return (("q", 2 * m.heads * m.dim), ("k", 2 * m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim))


def _ffn_specs(p: str, ff: int, W: int) -> list[TensorSpec]:
    return [TensorSpec(p + "gate", (ff, W), MATRIX_STD), TensorSpec(p + "up", (ff, W), MATRIX_STD),
            TensorSpec(p + "down", (W, ff), MATRIX_STD)]


def _streams_specs(cfg: FovosunConfig, p: str, q: int) -> list[TensorSpec]:
    n = cfg.streams
    return [TensorSpec(f"{p}norm{q}", (cfg.width,), 1.0, "norm"), TensorSpec(f"{p}hc{q}.in", (n,), 0.5, "norm"),
            TensorSpec(f"{p}hc{q}.out", (n,), 0.5, "norm"), TensorSpec(f"{p}hc{q}.mix", (n, n), 0.5, "norm")]


def _layer_specs(cfg: FovosunConfig, i: int) -> list[TensorSpec]:
    l, W, p = cfg.layers[i], cfg.width, f"l{i}."
    m, q, f = l.mixer, p + "mix.", l.mlp
    out = _streams_specs(cfg, p, 1)
    if l.type == RETENTION:
        for name, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
            out.append(TensorSpec(q + name, (rows, W), MATRIX_STD))
    else:
        for name, rows in _attention_rows(m):
            out.append(TensorSpec(q + name, (rows, W), MATRIX_STD))
            if l.type == BIASED_ATTENTION:
                out.append(TensorSpec(f"{q}{name}.b", (rows,), MATRIX_STD))
            if m.taps:
                out.append(TensorSpec(f"{q}{name}.conv", (rows, m.taps), CONV_STD, "norm"))
        out += [TensorSpec(q + n, (m.dim,), 0.1, "norm") for n in LAMBDA]
        if l.type == ATTENTION:
            out.append(TensorSpec(q + "g", (m.heads, W), MATRIX_STD))
    out.append(TensorSpec(q + "o", (W, m.heads * m.vdim), MATRIX_STD))
    if f is not None:
        out += _streams_specs(cfg, p, 2)
        if f.kind == "dense":
            out += _ffn_specs(p + "mlp.", f.ffn.ff, W)
        else:
            for e in range(f.experts):
                out += _ffn_specs(f"{p}mlp.e{e}.", f.ffn.ff, W)
            out += [TensorSpec(p + "mlp.router", (f.experts, W), MATRIX_STD), TensorSpec(p + "mlp.router.b", (f.experts,), 0.1, "norm")]
            if f.shared is not None:
                out += _ffn_specs(p + "mlp.shared.", f.shared.ff, W)
    return out


def tensor_specs(cfg: FovosunConfig) -> list[TensorSpec]:
    """Every tensor a Fovosun file holds for `cfg`, with the spread random weights are drawn with."""
    specs = [TensorSpec("embed", (cfg.vocab, cfg.width), MATRIX_STD)]
    for i in range(len(cfg.layers)):
        specs += _layer_specs(cfg, i)
    return specs + [TensorSpec("final.norm", (cfg.width,), 1.0, "norm"), TensorSpec("head", (cfg.vocab, cfg.width), MATRIX_STD)]


def _stack(parts: list[torch.Tensor]) -> torch.Tensor:
    if any(p.numel() == 0 for p in parts) or len({p.dtype for p in parts}) != 1:
        return torch.empty(0)                       # a fault already recorded by the store
    return torch.cat(parts, dim=0).contiguous()


def _taken(w: WeightStore, p: str, rows, suffix: str, *more: int) -> torch.Tensor:
    """The tensors `p<name><suffix>` of `rows` stacked into one matrix (or vector)."""
    names = [p + n + suffix for n, _ in rows]
    out = _stack([w.take(name, (r, *more)) for name, (_, r) in zip(names, rows)])
    w.release(*names)
    return out


def _rope(w: WeightStore, m, ropes: dict) -> Rope | None:
    if not m.rot_dims:
        return None
    key = (m.rot_dims, m.rot_base)                  # mixers with the same rotary constants share one table per step
    if key not in ropes:
        ropes[key] = Rope(m.rot_dims, m.rot_base, w.device)
    return ropes[key]


def _attention(cfg: FovosunConfig, w: WeightStore, kind: str, m, p: str, ropes: dict) -> DifferentialAttention:
    W, rows = cfg.width, _attention_rows(m)
    gated, biased = kind == ATTENTION, kind == BIASED_ATTENTION
    w_in = _taken(w, p, rows + ((("g", m.heads),) if gated else ()), "", W)            # [q | k | v | gate] rows
    bias = _taken(w, p, rows, ".b") if biased else None
    conv = _taken(w, p, rows, ".conv", m.taps) if m.taps else None
    vectors = [w.take(p + n, (m.dim,)) for n in LAMBDA]
    wo = w.take(p + "o", (W, m.heads * m.vdim))
    if w.faulty:
        w.finish()
    return DifferentialAttention(w_in, wo, vectors, n_heads=m.heads, n_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim,
                                 scale=m.scale, diff=m.diff, norm_eps=cfg.norm_eps, window=m.window, position=_rope(w, m, ropes),
                                 bias=bias, conv=ShortConv(conv) if conv is not None else None, temperature=m.temperature,
                                 gated=gated)


def _retention(cfg: FovosunConfig, w: WeightStore, m, p: str, ropes: dict) -> LightningAttention:
    W = cfg.width
    w_in = _taken(w, p, (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)), "", W)
    wo = w.take(p + "o", (W, m.heads * m.vdim))
    if w.faulty:
        w.finish()
    return LightningAttention(w_in, wo, None, m.decay, heads=m.heads, dim=m.dim, vdim=m.vdim, norm_eps=cfg.norm_eps,
                              activation=None, position=_rope(w, m, ropes), key_scale=m.dim ** -0.5, norm_heads=True, gate="silu")


def _ffn_weights(w: WeightStore, p: str, ff: int, W: int) -> tuple:
    return _taken(w, p, (("gate", ff), ("up", ff)), "", W), w.take(p + "down", (W, ff))


def _feed_forward(cfg: FovosunConfig, w: WeightStore, f, p: str):
    W = cfg.width
    if f.kind == "dense":
        gu, down = _ffn_weights(w, p, f.ffn.ff, W)
        if w.faulty:
            w.finish()
        return GatedFfn(gu, down, "clamped_swish", limit=f.ffn.limit)
    gus, downs = zip(*[_ffn_weights(w, f"{p}e{e}.", f.ffn.ff, W) for e in range(f.experts)])
    if w.faulty:
        w.finish()
    w_gate_up, w_down = torch.stack(gus).contiguous(), torch.stack(downs).contiguous()
    w.release(*[f"{p}e{e}.down" for e in range(f.experts)])
    shared = None
    if f.shared is not None:
        gu, down = _ffn_weights(w, p + "shared.", f.shared.ff, W)
        if w.faulty:
            w.finish()
        shared = GatedFfn(gu, down, "clamped_swish", limit=f.shared.limit)
    router, bias = w.take(p + "router", (f.experts, W)), w.take(p + "router.b", (f.experts,))
    if w.faulty:
        w.finish()
    return RoutedExperts(router, bias, w_gate_up, w_down, top=f.top, scale=1.0, limit=f.ffn.limit, shared=shared,
                         score="softmax_chosen")


def build(cfg: FovosunConfig, w: WeightStore) -> DecoderModel:
    W, n = cfg.width, cfg.streams
    table = w.take("embed", (cfg.vocab, W))
    if w.faulty:
        w.finish()

    def sublayer(p: str, q: int) -> tuple:
        """(what sublayer q reads, how its result joins the streams)."""
        norm = RmsNorm(w.take(f"{p}norm{q}", (W,)), cfg.norm_eps)
        weights, out, mix = w.take(f"{p}hc{q}.in", (n,)), w.take(f"{p}hc{q}.out", (n,)), w.take(f"{p}hc{q}.mix", (n, n))
        return StreamsNorm(weights, norm), StreamsMix(mix, out)

    blocks, ropes = [], {}
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        mixer = (_retention(cfg, w, l.mixer, p + "mix.", ropes) if l.type == RETENTION
                 else _attention(cfg, w, l.type, l.mixer, p + "mix.", ropes))
        norm1, mix1 = sublayer(p, 1)
        ffn = norm2 = mix2 = None
        if l.mlp is not None:
            ffn = _feed_forward(cfg, w, l.mlp, p + "mlp.")
            norm2, mix2 = sublayer(p, 2)
        else:                                       # a file may still hold the numbers of a sublayer that does not run
            unused = [s.name for s in _streams_specs(cfg, p, 2) if w.has(s.name)]
            for name in unused:
                w.take(name, w.shape_of(name))
            w.release(*unused)
        if w.faulty:
            w.finish()
        blocks.append(StreamsBlock(norm1, mixer, mix1, norm2, ffn, mix2))
    final_norm = RmsNorm(w.take("final.norm", (W,)), cfg.norm_eps)
    head = w.take("head", (cfg.vocab, W))
    w.finish()
    total = StreamsNorm(torch.ones(n, dtype=torch.float32, device=w.device), final_norm)
    return DecoderModel(StreamsEmbedding(table, n, scale=cfg.embedding_scale), blocks, LmHead(total, head), name=cfg.architecture)
