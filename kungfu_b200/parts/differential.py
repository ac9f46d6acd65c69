"""Differential attention: every head is the difference of two attentions over the same values.

With H heads over G key/value heads (r = H / G), key size d of one map and value size dv, for the input x of a token:

  [q | k | v | g] = x W_in^T (+ bias on q, k, v)             one product over the stacked matrix; q has H * 2 * d rows and k
                                                             G * 2 * d, head by head, map 1 then map 2; g one row per head
  q, k, v <- short causal convolution over time, per channel (`conv`, state: the last taps - 1 projected rows)
  q, k <- rotation of the first rotary elements of every map, pairs (i, i + rot/2)           (`position`)
  q <- q (1 + coef ln(floor((p + 1) / every) + 1)) at position p                             (`temperature`: coef, every)
  a_m,h(i) = sum_j softmax_j(q_m,h(i) . k_m,h/r(j) * scale) v_h/r(j),  m = 1, 2;  causal, optionally a sliding window
  o_h = a_1,h - lambda a_2,h,   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff              one number per mixer
  o_h <- o_h / sqrt(mean(o_h^2) + eps) * (1 - diff) * sigmoid(g_h)                           no weight; `gated`
  y = o W_o^T

Both maps read the same values, so the pages hold one key row [k_1 | k_2] and one value row per key/value head and token:
nothing is stored twice.  A query of map m is a row of 2 d elements that is zero outside map m's half, whose product with
the stored key is q_m . k_m; the attention kernels see 2 H ordinary query heads over G key/value heads of
D = max(2 d, dv) elements (rounded up to a size they have an instance for; tails zero) and read every key and value once
for both maps.  One kernel (`ops.diff_combine`) then takes the difference, norms and gates it.
Scores, softmax, angles, rotation, temperature, lambda, norm and gate are 32-bit.
"""
from __future__ import annotations

import math

import torch

from .. import ops
from .base import Mixer, PagedKV, PositionEncoding, StateBundle, pad_rows, register_mixer
from .conv import ShortConv
from .latent import latent_head_size

MAPS = 2


class DifferentialAttention(Mixer):
    def __init__(self, w_in: torch.Tensor, wo: torch.Tensor, lambda_vectors, *, n_heads: int, n_kv_heads: int, key_dim: int,
                 value_dim: int, scale: float, diff: float, norm_eps: float, window: int | None = None,
                 position: PositionEncoding | None = None, bias: torch.Tensor | None = None, conv: ShortConv | None = None,
                 temperature: tuple | None = None, gated: bool = False):
        """`lambda_vectors`: (lq1, lk1, lq2, lk2), key_dim numbers each; lambda is worked out once, in 64-bit."""
        if n_heads % n_kv_heads:
            raise ValueError(f"n_heads {n_heads} is not a multiple of n_kv_heads {n_kv_heads}")
        self.wo, self.bias, self.conv, self.position = wo, bias, conv, position
        self.n_heads, self.n_kv_heads = int(n_heads), int(n_kv_heads)
        self.key_dim, self.value_dim = int(key_dim), int(value_dim)
        self.head_dim = latent_head_size(max(MAPS * self.key_dim, self.value_dim))
        self.scale, self.diff, self.norm_eps = float(scale), float(diff), float(norm_eps)
        self.window = None if window is None else int(window)
        self.temperature = None if temperature is None else (float(temperature[0]), int(temperature[1]))
        self.gated = bool(gated)
        vectors = [t.detach().to("cpu", torch.float64) for t in lambda_vectors]
        self.lam = self.diff
        if all(t.numel() == self.key_dim for t in vectors):
            lq1, lk1, lq2, lk2 = vectors
            self.lam += math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum()))
        elif any(t.numel() for t in vectors):
            raise ValueError(f"lambda's vectors have {[t.numel() for t in vectors]} numbers, expected {self.key_dim} each")
        self.qkv_width = (self.n_heads + self.n_kv_heads) * MAPS * self.key_dim + self.n_kv_heads * self.value_dim
        self.proj_width = self.qkv_width + (self.n_heads if self.gated else 0)
        self.width = wo.shape[0]
        if w_in.numel() and w_in.shape[0] != self.proj_width:
            raise ValueError(f"stacked projection has shape {tuple(w_in.shape)}, expected {self.proj_width} rows")
        self.w_in = pad_rows(w_in)
        self.proj_width = max(self.proj_width, self.w_in.shape[0])
        if conv is not None and conv.channels != self.qkv_width:
            raise ValueError(f"the convolution has {conv.channels} channels, q|k|v have {self.qkv_width}")
        if position is not None:
            if getattr(position, "interleaved", False) or float(getattr(position, "magnitude", 1.0)) != 1.0:
                raise ValueError("this mixer turns pairs (i, i + rot/2) by cos and sin themselves")
            if position.rotary_dims > self.key_dim:
                raise ValueError(f"{position.rotary_dims} rotary dims for maps of {self.key_dim}")
        ops.check_attention_sizes(MAPS * self.n_heads, self.n_kv_heads, self.head_dim, ops.MAX_GENERIC_HEAD_DIM)

    def state_need(self):
        kv = PagedKV(self.n_kv_heads, self.head_dim, self.window)
        if self.conv is None or self.conv.taps <= 1:
            return kv
        return StateBundle((kv, self.conv.state_need()))

    def forward(self, x, ctx, cache):
        kv, tail = cache if isinstance(cache, tuple) else (cache, None)
        T = x.shape[0]
        nh, nkv, D = self.n_heads, self.n_kv_heads, self.head_dim
        proj = ctx.buf("attn_proj", (T, self.proj_width), torch.float32)
        ops.linear(x, self.w_in, proj)
        cos = sin = None
        rot = 0
        if self.position is not None:
            cos, sin = self.position.rotation(ctx)
            rot = 2 * cos.shape[1]
        q = ctx.buf("attn_q", (T, MAPS * nh * D), ctx.act_dtype)
        conv = self.conv
        moves = tail is not None and tail.writes
        done = ops.qkv_prepare(proj, 0, self.bias, conv.weight if conv else None, tail.state if tail is not None else None, None,
                               None, self.norm_eps, cos, sin, rot, False, nh, nkv, self.key_dim, self.value_dim, ctx, kv, q,
                               commit_inline=moves and bool(getattr(ctx, "decode_only", False)), parts=MAPS,
                               temperature=self.temperature)
        if moves and not done:
            conv.commit(proj, 0, self.bias, ctx, tail)
        o = ctx.buf("attn_o", (T, MAPS * nh * D), ctx.act_dtype)
        ops.paged_attention(q, o, ctx, kv, MAPS * nh, nkv, D, self.scale, 0.0, self.window)
        packed = ctx.buf("attn_gated", (T, nh * self.value_dim), ctx.act_dtype)
        ops.diff_combine(o, self.lam, 1.0 - self.diff, self.norm_eps, proj if self.gated else None, self.qkv_width, nh,
                         self.value_dim, D, packed, ctx)
        y = ctx.buf("branch_out", (T, self.width), torch.float32)
        ops.linear(packed, self.wo, y)
        return y


register_mixer("differential_attention", DifferentialAttention)
