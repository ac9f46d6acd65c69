"""A plain, slow Lurisun: float64, whole sequences, no cache, one function per mechanism.

Shares nothing with the package.  `cfg` is the dictionary of a config.json, `w` a dictionary name -> tensor.
Notation: W width, H query heads, G key/value heads, d key size, dv value size, r rotated elements of a head.
"""
from __future__ import annotations

import math

import torch

F = torch.float64

# What a 16-bit serving path may round: the inputs of matrix products, queries, keys and values as the attention reads
# them, the attention's weights, the feed-forwards' inner rows.  `ROUND` is applied at those places; the identity by
# default.  `rounded_to_bfloat16()` switches it for a block of code: a yardstick of what 8-bit mantissas alone do.
_EXACT = lambda t: t
ROUND = _EXACT


class rounded_to_bfloat16:
    def __enter__(self):
        global ROUND
        self.saved, ROUND = ROUND, (lambda t: t.to(torch.bfloat16).to(F))

    def __exit__(self, *exc):
        global ROUND
        ROUND = self.saved
        return False


def rms(x, eps: float):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def linear(x, weight, bias=None):
    y = ROUND(x) @ weight.to(F).T
    return y if bias is None else y + bias.to(F)


def silu(x):
    return x / (1.0 + torch.exp(-x))


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


# ---- embedding ----------------------------------------------------------------------------------------------------

def bigram_rows(tokens, mul_prev: int, mul_cur: int, buckets: int) -> list:
    """The row of the bigram table every token adds: the last row for a sequence's first token."""
    rows = []
    for i, t in enumerate(tokens):
        rows.append(buckets if i == 0 else (int(tokens[i - 1]) * mul_prev + int(t) * mul_cur) % buckets)
    return rows


def embedding(tokens, w, cfg):
    b = cfg["embedding"]["bigram"]
    rows = bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"])
    return w["embed"].to(F)[list(tokens)] + w["bigram"].to(F)[rows]


# ---- the convolution of a mixer's input ---------------------------------------------------------------------------

def input_convolution(h, weight):
    """h_t + sum_j weight[:, j] h_(t - taps + 1 + j), zeros before the first row."""
    T, taps = h.shape[0], weight.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] = out[t] + weight[:, j].to(F) * h[s]
    return out


# ---- decayed linear attention -------------------------------------------------------------------------------------

def decayed_memory(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T from zero, o_t = S_t^T q_t;  q, k [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        S = torch.zeros(d, v.shape[-1], dtype=F)
        for t in range(T):
            S = float(decay[h]) * S + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S.T @ q[t, h]
    return out


def lightning(h, w, p: str, m: dict, eps: float):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = ROUND(silu(linear(h, w[p + "q"]))).view(T, H, d)
    k = ROUND(silu(linear(h, w[p + "k"]))).view(T, H, d)
    v = ROUND(silu(linear(h, w[p + "v"]))).view(T, H, dv)
    o = decayed_memory(q, k, v, m["decay"]).reshape(T, H * dv)
    o = rms(o, eps) * w[p + "norm"].to(F) * sigmoid(linear(h, w[p + "g"]))
    return linear(o, w[p + "o"])


# ---- attention ----------------------------------------------------------------------------------------------------

def rotate_halves(x, positions, base: float, r: int):
    """x [T, heads, n]: pairs (i, i + r/2) of the first r elements of every head turned by position * base^(-2i/r)."""
    if r == 0:
        return x
    f = float(base) ** (-2.0 * torch.arange(r // 2, dtype=F) / r)
    ang = positions.to(F)[:, None] * f[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., : r // 2], x[..., r // 2: r]
    out[..., : r // 2] = u * cos - v * sin
    out[..., r // 2: r] = v * cos + u * sin
    return out


def chunk_mask(T: int, size: int | None):
    """Row i sees column j iff j <= i and both stand in the same run of `size` positions, counted from 0."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    m = j <= i
    return m if size is None else m & (i // size == j // size)


def window_mask(T: int, size: int | None):
    """Row i sees column j iff 0 <= i - j < size."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    m = j <= i
    return m if size is None else m & (i - j < size)


def sigmoid_attend(q, k, v, scale: float, bias, mask):
    """Every visible key counts with sigmoid(q . k * scale + bias_h), not normalized.  Head h reads head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    q, k, v = ROUND(q), ROUND(k), ROUND(v)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        g = h // (H // G)
        a = sigmoid((q[:, h] @ k[:, g].T) * scale + float(bias[h]))
        out[:, h] = ROUND(a.masked_fill(~mask, 0.0)) @ v[:, g]
    return out


def softmax_attend(q, k, v, scale: float, mask):
    """q [T, H, d], k [T, H, d], v [T, H, dv]."""
    T, H, _ = q.shape
    q, k, v = ROUND(q), ROUND(k), ROUND(v)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(~mask, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = ROUND(e / e.sum(-1, keepdim=True)) @ v[:, h]
    return out


def attention(h, w, p: str, m: dict, eps: float):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = linear(h, w[p + "q"], w[p + "q.b"])
    k = linear(h, w[p + "k"], w[p + "k.b"])
    v = k.view(T, G, d)                                          # the keys as projected are the values
    q = (rms(q, eps) * w[p + "q.norm"].to(F)).view(T, H, d)
    k = (rms(k, eps) * w[p + "k.norm"].to(F)).view(T, G, d)
    rot = m.get("rot")
    if rot:
        pos = torch.arange(T)
        q, k = (rotate_halves(t, pos, rot["base"], rot["dims"]) for t in (q, k))
    mask = chunk_mask(T, m["mask"]["size"] if m.get("mask") else None)
    o = sigmoid_attend(q, k, v, m["scale"], w[p + "pb"].to(F), mask)
    return linear(o.reshape(T, H * d), w[p + "o"])


def latent_attention(h, w, p: str, m: dict, eps: float):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    cq = rms(linear(h, w[p + "dq"]), eps) * w[p + "dq.norm"].to(F)
    q = linear(cq, w[p + "uq"]).view(T, H, d)
    c = rms(linear(h, w[p + "dkv"]), eps) * w[p + "dkv.norm"].to(F)
    mask = window_mask(T, m["mask"]["size"] if m.get("mask") else None)
    if ROUND is _EXACT:
        k = linear(c, w[p + "uk"]).view(T, H, d)
        v = linear(c, w[p + "uv"]).view(T, H, dv)
        o = softmax_attend(q, k, v, m["scale"], mask)
    else:
        # the same attention in the latent space, as a path that caches c alone has to: q . (U c) = (U^T q) . c, and the
        # values' map applied after the weighted sum.  Exactly equal; what is rounded differs.
        uk, uv = w[p + "uk"].to(F).view(H, d, -1), w[p + "uv"].to(F).view(H, dv, -1)
        ql = torch.einsum("thd,hdr->thr", ROUND(q), uk)
        cs = c[:, None, :].expand(T, H, c.shape[-1])
        ol = ROUND(softmax_attend(ql, cs, cs, m["scale"], mask))
        o = torch.einsum("thr,hvr->thv", ol, uv)
    o = o.reshape(T, H * dv)
    return linear(o * sigmoid(linear(h, w[p + "g"])), w[p + "o"])


# ---- the model ----------------------------------------------------------------------------------------------------

def feed_forward(x, w, p: str):
    return linear(silu(linear(x, w[p + "gate"])) * linear(x, w[p + "up"]), w[p + "down"])


MIXERS = {"lightning": lightning, "attention": attention, "latent_attention": latent_attention}


def forward(cfg: dict, w: dict, tokens, layers_out: list | None = None):
    """Logits [T, vocab] in float64; `layers_out` collects the residual stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = embedding(tokens, w, cfg)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(x, w[p + "canon1"])
        x = x + rms(MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps), eps) * w[p + "norm1"].to(F)
        if layer.get("mlp"):
            x = x + rms(feed_forward(x, w, p + "mlp."), eps) * w[p + "norm2"].to(F)
        if layers_out is not None:
            layers_out.append(x.clone())
    return linear(rms(x, eps) * w["final.norm"].to(F), w["head"]) * float(cfg["logit_scale"])
