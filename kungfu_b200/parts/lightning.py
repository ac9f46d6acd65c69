"""Linear attention with one fixed decay per head ("lightning attention") as a mixer.

With H heads, key size d and value size dv, for the input x of a token:
  q, k = silu(W_q x), silu(W_k x)  (H d each)      v = silu(W_v x)  (H dv)      g = W_g x  (H dv)
  S_h <- a_h S_h + k_h v_h^T;  o_h = S_h^T q_h       S_h: d x dv, 32-bit, zero at admission; a_h a constant of the model
  o <- o / sqrt(mean over all heads' elements of o^2 + eps) * w * sigmoid(g);  y = W_o o
The state, the recurrence, the norm and the gate are 32-bit; the state is carried per request in the cache manager's state
slots, so a request may be fed in portions of any size.  A prompt portion in bfloat16 takes q, k and v from a product whose
epilogue is the activation (bfloat16 rows the tensor-core walk reads) and g from a second one; everything else takes one
product over the stacked matrix and the activation is applied as the recurrence reads its 32-bit result.

Options for other models of the kind ("retention" has all of them):
  `activation` None   q, k and v are the projections themselves
  `position`          q and k are turned by it, pairs (i, i + rot/2) of every head's first rotary elements
  `key_scale`         k is multiplied by it, after the rotation
  `norm_heads`        every head's o is divided by its own root mean square instead of all heads' together; `norm_weight`
                      may be None (no weight)
  `gate` 'silu'       silu(g) instead of sigmoid(g)
With a rotation or a key scale a prompt portion in bfloat16 takes everything from one 32-bit product, and one kernel turns,
scales and rounds q, k and v for the tensor-core walk; elsewhere that happens as the recurrence reads them.
"""
from __future__ import annotations

import torch

from .. import ops
from .base import FixedState, Mixer, PositionEncoding, pad_rows, register_mixer


class LightningAttention(Mixer):
    def __init__(self, w_in: torch.Tensor, wo: torch.Tensor, norm_weight: torch.Tensor | None, decay, *, heads: int, dim: int,
                 vdim: int, norm_eps: float, out_tag: str = "branch_out", activation: str | None = "silu",
                 position: PositionEncoding | None = None, key_scale: float = 1.0, norm_heads: bool = False,
                 gate: str = "sigmoid"):
        """`w_in`: the stacked rows [q | k | v | g]; `decay`: one number in [0, 1] per head."""
        if activation not in (None, "silu") or gate not in ("sigmoid", "silu"):
            raise ValueError(f"activation {activation!r} or gate {gate!r} is not known")
        self.activation, self.position, self.key_scale = activation, position, float(key_scale)
        self.norm_heads, self.gate = bool(norm_heads), gate
        if position is not None:
            if getattr(position, "interleaved", False) or float(getattr(position, "magnitude", 1.0)) != 1.0:
                raise ValueError("this mixer turns pairs (i, i + rot/2) by cos and sin themselves")
            if position.rotary_dims > dim:
                raise ValueError(f"{position.rotary_dims} rotary dims for keys of {dim}")
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
        cos = sin = None
        rot = 0
        if self.position is not None:
            cos, sin = self.position.rotation(ctx)
            rot = 2 * cos.shape[1]
        prepared = rot > 0 or self.key_scale != 1.0            # q and k need more than the product's own epilogue
        o = ctx.buf("lightning_o", (T, H * dv), torch.float32)
        rows, act, turn = None, self.activation, dict(cos=cos, sin=sin, rot=rot, key_scale=self.key_scale)
        if (ctx.act_dtype == torch.bfloat16 and not getattr(ctx, "decode_only", False) and not (prepared and act)
                and ops.decay_memory_takes_bfloat16(d, dv, self.g_col)):
            rows, turn = ctx.buf("lightning_qkv", (T, self.g_col), ctx.act_dtype), {}
        if rows is not None and not prepared:
            if act:
                ops.linear_act(x, self.w_in[:self.g_col], rows, act, ctx)
            else:
                ops.linear(x, self.w_in[:self.g_col], rows)
            gate, g0 = ctx.buf("lightning_gate", (T, self.proj_width - self.g_col), torch.float32), 0
            ops.linear(x, self.w_in[self.g_col:], gate)
        else:
            gate, g0 = ctx.buf("lightning_proj", (T, self.proj_width), torch.float32), self.g_col
            ops.linear(x, self.w_in, gate)
            if rows is not None:
                ops.decay_rotate(gate, 0, self.k_col, self.v_col, cos, sin, rot, self.key_scale, H, d, dv, rows)
        ops.decay_memory(gate if rows is None else rows, 0, self.k_col, self.v_col, act if rows is None else None, self.powers,
                         cache.state, o, H, d, dv, ctx, writes=cache.writes, **turn)
        normed = ctx.buf("lightning_normed", (T, H * dv), ctx.act_dtype)
        nh, nd = (H, dv) if self.norm_heads else (1, H * dv)    # all heads together: one head
        ops.head_norm_gate(o, self.norm_weight, self.norm_eps, gate, g0, self.gate, normed, nh, nd)
        y = ctx.buf(self.out_tag, (T, self.width), torch.float32)
        ops.linear(normed, self.wo, y)
        return y


register_mixer("lightning_attention", LightningAttention)
