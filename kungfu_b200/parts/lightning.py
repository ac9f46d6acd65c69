"""Linear attention with one fixed decay per head ("lightning attention") as a mixer.

With H heads, key size d and value size dv, for the input x of a token:
  q, k = silu(W_q x), silu(W_k x)  (H d each)      v = silu(W_v x)  (H dv)      g = W_g x  (H dv)
  S_h <- a_h S_h + k_h v_h^T;  o_h = S_h^T q_h       S_h: d x dv, 32-bit, zero at admission; a_h a constant of the model
  o <- o / sqrt(mean over all heads' elements of o^2 + eps) * w * sigmoid(g);  y = W_o o
The state, the recurrence, the norm and the gate are 32-bit; the state is carried per request in the cache manager's state
slots, so a request may be fed in portions of any size.  A prompt portion in bfloat16 takes q, k and v from a product whose
epilogue is the activation (bfloat16 rows the tensor-core walk reads) and g from a second one; everything else takes one
product over the stacked matrix and the activation is applied as the recurrence reads its 32-bit result.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import FixedState, Mixer, pad_rows, register_mixer


class LightningAttention(Mixer):
    def __init__(self, w_in: torch.Tensor, wo: torch.Tensor, norm_weight: torch.Tensor, decay, *, heads: int, dim: int,
                 vdim: int, norm_eps: float, out_tag: str = "branch_out"):
        """`w_in`: the stacked rows [q | k | v | g]; `decay`: one number in [0, 1] per head."""
        decay = [float(a) for a in decay]
        if len(decay) != heads or not all(0.0 <= a <= 1.0 for a in decay):
            raise ValueError(f"expected {heads} decays between 0 and 1, found {decay}")
        if dim > 256:
            raise ValueError(f"key size {dim} is above 256, the most the recurrence keeps in registers")
        self.wo, self.norm_weight = wo, norm_weight
        self.heads, self.dim, self.vdim = int(heads), int(dim), int(vdim)
        self.norm_eps, self.out_tag = float(norm_eps), out_tag
        H, d, dv = self.heads, self.dim, self.vdim
        self.k_col, self.v_col, self.g_col = H * d, 2 * H * d, 2 * H * d + H * dv
        want = self.g_col + H * dv
        if w_in.numel() and w_in.shape[0] != want:
            raise ValueError(f"the input projection has {w_in.shape[0]} rows, expected {want}")
        self.w_in = pad_rows(w_in)
        self.proj_width = max(want, self.w_in.shape[0])
        self.width = wo.shape[0]
        self.powers = ops.decay_powers(decay).to(wo.device)

    def state_need(self):
        return FixedState((self.heads, self.dim, self.vdim), torch.float32)

    def forward(self, x, ctx, cache):
        T = x.shape[0]
        H, d, dv = self.heads, self.dim, self.vdim
        o = ctx.buf("lightning_o", (T, H * dv), torch.float32)
        if (ctx.act_dtype == torch.bfloat16 and not getattr(ctx, "decode_only", False)
                and ops.decay_memory_takes_bfloat16(d, dv, self.g_col)):
            qkv = ctx.buf("lightning_qkv", (T, self.g_col), ctx.act_dtype)
            ops.linear_act(x, self.w_in[:self.g_col], qkv, "silu", ctx)
            gate, g0 = ctx.buf("lightning_gate", (T, self.proj_width - self.g_col), torch.float32), 0
            ops.linear(x, self.w_in[self.g_col:], gate)
            ops.decay_memory(qkv, 0, self.k_col, self.v_col, None, self.powers, cache.state, o, H, d, dv, ctx, writes=cache.writes)
        else:
            gate, g0 = ctx.buf("lightning_proj", (T, self.proj_width), torch.float32), self.g_col
            ops.linear(x, self.w_in, gate)
            ops.decay_memory(gate, 0, self.k_col, self.v_col, "silu", self.powers, cache.state, o, H, d, dv, ctx, writes=cache.writes)
        normed = ctx.buf("lightning_normed", (T, H * dv), ctx.act_dtype)
        ops.head_norm_gate(o, self.norm_weight, self.norm_eps, gate, g0, "sigmoid", normed, 1, H * dv)   # all heads: one head
        y = ctx.buf(self.out_tag, (T, self.width), torch.float32)
        ops.linear(normed, self.wo, y)
        return y


register_mixer("lightning_attention", LightningAttention)
