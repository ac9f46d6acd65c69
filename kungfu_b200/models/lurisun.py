"""Lurisun put together from parts.

A Lurisun model embeds a token and the pair it makes with the token before it (`parts.PairEmbedding`), then runs a list of
blocks whose sublayers read the residual stream itself and whose results are normed before they join it:
`x += norm1(mixer(x + conv(x))); x += norm2(ff(x))`, conv a short causal convolution over time (`parts.SandwichBlock` with
`parts.InputConv` and `parts.NoNorm` in the places of the norms before the sublayers).  A layer's mixer is one of
  latent_attention  attention over a cached latent without positions, queries through a latent of their own, a sliding
                    window and a gate per element of the heads (`parts.LatentAttention`);
  lightning         linear attention with one fixed decay per head, its heads normed together and gated
                    (`parts.LightningAttention`);
  attention         grouped-query attention with biased projections, q and k normed over the whole projection, rotary pairs
                    (i, i + dims/2) on part of each head, the keys as projected for values, chunks of positions instead of a
                    window, and sigmoid weights with a bias per head instead of a softmax (`parts.RowNormAttention`).
The feed-forward is a silu-gated one or absent.  The output is a norm, an untied matrix and a factor on the logits.
Tensor names are those of a Lurisun safetensors file: `embed`, `bigram`, `l<i>.norm1|norm2|canon1`, `l<i>.mix.*` (latent:
dq, dq.norm, uq, dkv, dkv.norm, uk, uv, g, o; lightning: q, k, v, g, o, norm; attention: q, q.b, k, k.b, q.norm, k.norm, pb, o),
`l<i>.mlp.gate|up|down`, `final.norm`, `head`.
"""
from __future__ import annotations

import torch

from ..config.lurisun import LATENT, LIGHTNING, LurisunConfig
from ..parts import (DecoderModel, GatedFfn, InputConv, LatentAttention, LightningAttention, LmHead, NoNorm, PairEmbedding,
                     RmsNorm, Rope, RowNormAttention, SandwichBlock)
from ..weights.store import TensorSpec, WeightStore

MATRIX_STD = 0.02


def _layer_specs(cfg: LurisunConfig, i: int) -> list[TensorSpec]:
    l, W, p = cfg.layers[i], cfg.width, f"l{i}."
    m, q = l.mixer, p + "mix."
    out = [TensorSpec(p + "norm1", (W,), 1.0, "norm"), TensorSpec(p + "canon1", (W, cfg.taps), 0.2)]
    if l.type == LATENT:
        out += [TensorSpec(q + "dq", (m.q_rank, W), MATRIX_STD), TensorSpec(q + "dq.norm", (m.q_rank,), 1.0, "norm"),
                TensorSpec(q + "uq", (m.heads * m.dim, m.q_rank), MATRIX_STD), TensorSpec(q + "dkv", (m.kv_rank, W), MATRIX_STD),
                TensorSpec(q + "dkv.norm", (m.kv_rank,), 1.0, "norm"), TensorSpec(q + "uk", (m.heads * m.dim, m.kv_rank), MATRIX_STD),
                TensorSpec(q + "uv", (m.heads * m.vdim, m.kv_rank), MATRIX_STD), TensorSpec(q + "g", (m.heads * m.vdim, W), MATRIX_STD),
                TensorSpec(q + "o", (W, m.heads * m.vdim), MATRIX_STD)]
    elif l.type == LIGHTNING:
        out += [TensorSpec(q + "q", (m.heads * m.dim, W), MATRIX_STD), TensorSpec(q + "k", (m.heads * m.dim, W), MATRIX_STD),
                TensorSpec(q + "v", (m.heads * m.vdim, W), MATRIX_STD), TensorSpec(q + "g", (m.heads * m.vdim, W), MATRIX_STD),
                TensorSpec(q + "o", (W, m.heads * m.vdim), MATRIX_STD), TensorSpec(q + "norm", (m.heads * m.vdim,), 1.0, "norm")]
    else:
        nq, nk = m.heads * m.dim, m.kv_heads * m.dim
        out += [TensorSpec(q + "q", (nq, W), MATRIX_STD), TensorSpec(q + "q.b", (nq,), MATRIX_STD),
                TensorSpec(q + "k", (nk, W), MATRIX_STD), TensorSpec(q + "k.b", (nk,), MATRIX_STD),
                TensorSpec(q + "q.norm", (nq,), 1.0, "norm"), TensorSpec(q + "k.norm", (nk,), 1.0, "norm"),
                TensorSpec(q + "pb", (m.heads,), 1.0, "norm"), TensorSpec(q + "o", (W, nq), MATRIX_STD)]
    if l.ff:
        out += [TensorSpec(p + "norm2", (W,), 1.0, "norm"), TensorSpec(p + "mlp.gate", (l.ff, W), MATRIX_STD),
                TensorSpec(p + "mlp.up", (l.ff, W), MATRIX_STD), TensorSpec(p + "mlp.down", (W, l.ff), MATRIX_STD)]
    return out


def tensor_specs(cfg: LurisunConfig) -> list[TensorSpec]:
    """Every tensor a Lurisun file holds for `cfg`, with the spread random weights are drawn with."""
    specs = [TensorSpec("embed", (cfg.vocab, cfg.width), MATRIX_STD), TensorSpec("bigram", (cfg.pair.buckets + 1, cfg.width), MATRIX_STD)]
    for i in range(len(cfg.layers)):
        specs += _layer_specs(cfg, i)
    return specs + [TensorSpec("final.norm", (cfg.width,), 1.0, "norm"), TensorSpec("head", (cfg.vocab, cfg.width), MATRIX_STD)]


def _stack(parts: list[torch.Tensor]) -> torch.Tensor:
    if any(p.numel() == 0 for p in parts) or len({p.dtype for p in parts}) != 1:
        return torch.empty(0)                       # a fault already recorded by the store
    return torch.cat(parts, dim=0).contiguous()


def _latent(cfg: LurisunConfig, w: WeightStore, m, p: str) -> LatentAttention:
    W = cfg.width
    mixer = LatentAttention(w.take(p + "uq", (m.heads * m.dim, m.q_rank)), w.take(p + "dkv", (m.kv_rank, W)),
                            w.take(p + "dkv.norm", (m.kv_rank,)), w.take(p + "uk", (m.heads * m.dim, m.kv_rank)),
                            w.take(p + "uv", (m.heads * m.vdim, m.kv_rank)), w.take(p + "o", (W, m.heads * m.vdim)),
                            n_heads=m.heads, dim=m.dim, vdim=m.vdim, rank=m.kv_rank, scale=m.scale, norm_eps=cfg.norm_eps,
                            window=m.window, w_dq=w.take(p + "dq", (m.q_rank, W)), dq_norm=w.take(p + "dq.norm", (m.q_rank,)),
                            w_gate=w.take(p + "g", (m.heads * m.vdim, W)), gate_elements=True)
    w.release(p + "dq", p + "dkv", p + "g", p + "uk", p + "uv")
    return mixer


def _lightning(cfg: LurisunConfig, w: WeightStore, m, p: str) -> LightningAttention:
    W = cfg.width
    rows = (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim))
    w_in = _stack([w.take(p + n, (r, W)) for n, r in rows])
    w.release(*[p + n for n, _ in rows])
    return LightningAttention(w_in, w.take(p + "o", (W, m.heads * m.vdim)), w.take(p + "norm", (m.heads * m.vdim,)), m.decay,
                              heads=m.heads, dim=m.dim, vdim=m.vdim, norm_eps=cfg.norm_eps)


def _attention(cfg: LurisunConfig, w: WeightStore, m, p: str, ropes: dict) -> RowNormAttention:
    W = cfg.width
    nq, nk = m.heads * m.dim, m.kv_heads * m.dim
    rows = (("q", nq), ("k", nk))
    w_in = _stack([w.take(p + n, (r, W)) for n, r in rows])
    bias = _stack([w.take(p + n + ".b", (r,)) for n, r in rows])
    w.release(*[p + n for n, _ in rows], *[p + n + ".b" for n, _ in rows])
    rope = None
    if m.rot_dims:
        key = (m.dim, m.rot_dims, m.rot_base)       # mixers with the same rotary constants share one table per step
        if key not in ropes:
            ropes[key] = Rope(m.dim, m.rot_base, w.device, m.rot_dims)
        rope = ropes[key]
    return RowNormAttention(w_in, w.take(p + "o", (W, nq)), n_heads=m.heads, n_kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.dim,
                            scale=m.scale, position=rope, bias=bias if bias.numel() else None, q_norm=w.take(p + "q.norm", (nq,)),
                            k_norm=w.take(p + "k.norm", (nk,)), norm_eps=cfg.norm_eps, values_are_keys=True, chunk=m.chunk,
                            sigmoid_bias=w.take(p + "pb", (m.heads,)))


def build(cfg: LurisunConfig, w: WeightStore) -> DecoderModel:
    W = cfg.width
    table, pair = w.take("embed", (cfg.vocab, W)), w.take("bigram", (cfg.pair.buckets + 1, W))
    if w.faulty:
        w.finish()
    blocks, ropes = [], {}
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        if l.type == LATENT:
            mixer = _latent(cfg, w, l.mixer, p + "mix.")
        elif l.type == LIGHTNING:
            mixer = _lightning(cfg, w, l.mixer, p + "mix.")
        else:
            mixer = _attention(cfg, w, l.mixer, p + "mix.", ropes)
        conv = w.take(p + "canon1", (W, cfg.taps))
        norm1 = RmsNorm(w.take(p + "norm1", (W,)), cfg.norm_eps)
        ffn = norm2 = None
        if l.ff:
            gate_up = _stack([w.take(p + "mlp.gate", (l.ff, W)), w.take(p + "mlp.up", (l.ff, W))])
            w.release(p + "mlp.gate", p + "mlp.up")
            down = w.take(p + "mlp.down", (W, l.ff))
            norm2 = RmsNorm(w.take(p + "norm2", (W,)), cfg.norm_eps)
            if not w.faulty:
                ffn = GatedFfn(gate_up, down, "silu")
        if w.faulty:
            w.finish()
        blocks.append(SandwichBlock(InputConv(conv), mixer, norm1, NoNorm(W) if ffn is not None else None, ffn, norm2))
    final_norm = RmsNorm(w.take("final.norm", (W,)), cfg.norm_eps)
    head = w.take("head", (cfg.vocab, W))
    w.finish()
    return DecoderModel(PairEmbedding(table, pair, cfg.pair.mul_prev, cfg.pair.mul_cur), blocks,
                        LmHead(final_norm, head, scale=cfg.logit_scale), name=cfg.architecture)
