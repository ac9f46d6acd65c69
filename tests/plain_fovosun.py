"""A plain, slow Fovosun: float64, whole sequences, no cache, one function per mechanism.

Shares nothing with the package.  `cfg` is the dictionary of a config.json, `w` a dictionary name -> tensor.
Notation: W width, N streams, H query heads, G key/value heads, d query/key size of one map, dv value size.
"""
from __future__ import annotations

import math

import torch

F = torch.float64

# What a 16-bit serving path may round: the inputs of matrix products, queries, keys and values as the attention and the
# retention read them, the attention's weights and each map's result, the feed-forwards' inner rows.  `ROUND` is applied at
# those places; the identity by default.  `rounded_to_bfloat16()` switches it for a block of code: a yardstick of what
# 8-bit mantissas alone do.
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


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


# ---- streams ------------------------------------------------------------------------------------------------------

def gather_streams(xs, weights):
    """sum_s weights[s] xs[s];  xs [N, T, W]."""
    return sum(float(weights[s]) * xs[s] for s in range(xs.shape[0]))


def scatter_streams(xs, y, mix, out):
    """Every stream from the old ones: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    N = xs.shape[0]
    return torch.stack([sum(float(mix[s, t]) * xs[s] for s in range(N)) + float(out[t]) * y for t in range(N)])


# ---- what stands between the projections and the attention --------------------------------------------------------

def causal_convolution(u, weight):
    """y_t = sum_j weight[:, j] u_(t - taps + 1 + j), zeros before the first row;  u [T, C], weight [C, taps]."""
    T, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + weight[:, j].to(F) * u[s]
    return y


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


def temperature(positions, coef: float, every: int):
    """The factor of the query at each position: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1.0 + coef * math.log((int(p) + 1) // every + 1) for p in positions], dtype=F)


# ---- attention ----------------------------------------------------------------------------------------------------

def window_mask(T: int, size: int | None):
    """Row i sees column j iff 0 <= i - j < size (no bound without a size)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    m = j <= i
    return m if size is None else m & (i - j < size)


def softmax_attend(q, k, v, scale: float, mask):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    r = H // k.shape[1]
    q, k, v = ROUND(q), ROUND(k), ROUND(v)
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for h in range(H):
        s = ((q[:, h] @ k[:, h // r].T) * scale).masked_fill(~mask, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = ROUND(ROUND(e) @ v[:, h // r] / e.sum(-1, keepdim=True))
    return out


def difference_weight(lq1, lk1, lq2, lk2, diff: float) -> float:
    """lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    dot = lambda a, b: float((a.to(F) * b.to(F)).sum())
    return math.exp(dot(lq1, lk1)) - math.exp(dot(lq2, lk2)) + diff


def difference(a1, a2, lam: float, diff: float, eps: float):
    """(a1 - lambda a2), every head divided by its root mean square, times 1 - diff."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention(h, w, p: str, m: dict, eps: float):
    """Every step a layer's options name, in order; both kinds of attention layer are this with other options."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (linear(h, w[p + n], w.get(p + n + ".b")) for n in "qkv")
    if m.get("conv"):
        q, k, v = (causal_convolution(t, w[p + n + ".conv"]) for n, t in (("q", q), ("k", k), ("v", v)))
    q, k, v = q.view(T, H, 2, d), k.view(T, G, 2, d), v.view(T, G, dv)
    pos = torch.arange(T)
    rot = m.get("rot")
    maps = []
    for i in (0, 1):
        qi, ki = q[:, :, i], k[:, :, i]
        if rot:
            qi, ki = (rotate_halves(t, pos, rot["base"], rot["dims"]) for t in (qi, ki))
        if m.get("q_temp"):
            qi = qi * temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
        maps.append(softmax_attend(qi, ki, v, m["scale"], window_mask(T, m["mask"]["size"] if m.get("mask") else None)))
    lam = difference_weight(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    o = difference(maps[0], maps[1], lam, m["diff"], eps)
    if p + "g" in w:
        o = o * sigmoid(linear(h, w[p + "g"]))[:, :, None]
    return linear(o.reshape(T, H * dv), w[p + "o"])


# ---- retention ----------------------------------------------------------------------------------------------------

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


def retention(h, w, p: str, m: dict, eps: float):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = linear(h, w[p + "q"]).view(T, H, d), linear(h, w[p + "k"]).view(T, H, d), linear(h, w[p + "v"]).view(T, H, dv)
    rot = m.get("rot")
    if rot:
        q, k = (rotate_halves(t, torch.arange(T), rot["base"], rot["dims"]) for t in (q, k))
    o = rms(decayed_memory(ROUND(q), ROUND(k * d ** -0.5), ROUND(v), m["decay"]), eps).reshape(T, H * dv)
    g = linear(h, w[p + "g"])
    return linear(o * g * sigmoid(g), w[p + "o"])


# ---- feed-forward -------------------------------------------------------------------------------------------------

def clamped_feed_forward(x, w, p: str, limit: float):
    g = torch.clamp(linear(x, w[p + "gate"]), max=limit)
    u = torch.clamp(linear(x, w[p + "up"]), min=-limit, max=limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w[p + "down"])


def route(logits, top: int):
    """Per row: [(expert, weight)] of the `top` largest logits, weights the softmax over those logits alone."""
    rows = []
    for z in logits:
        best = sorted(range(len(z)), key=lambda e: (-float(z[e]), e))[:top]
        ex = [math.exp(float(z[e]) - float(z[best[0]])) for e in best]
        rows.append([(e, x / sum(ex)) for e, x in zip(best, ex)])
    return rows


def mixture(x, w, p: str, f: dict):
    r = f["router"]
    y = torch.zeros(x.shape, dtype=F)
    picks = route(linear(x, w[p + "router"], w[p + "router.b"]), r["top"])
    results = {}
    for e in {e for row in picks for e, _ in row}:
        at = [t for t, row in enumerate(picks) if any(e == i for i, _ in row)]
        results[e] = dict(zip(at, clamped_feed_forward(x[at], w, f"{p}e{e}.", f["expert"]["limit"])))
    for t, row in enumerate(picks):
        for e, weight in row:
            y[t] = y[t] + weight * results[e][t]
    if f.get("shared"):
        y = y + clamped_feed_forward(x, w, p + "shared.", f["shared"]["limit"])
    return y


def feed_forward(x, w, p: str, f: dict):
    return clamped_feed_forward(x, w, p, f["limit"]) if f["kind"] == "dense" else mixture(x, w, p, f)


# ---- the model ----------------------------------------------------------------------------------------------------

MIXERS = {"attention": attention, "attention_2": attention, "retention": retention}


def forward(cfg: dict, w: dict, tokens, layers_out: list | None = None):
    """Logits [T, vocab] in float64; `layers_out` collects the sum of the streams after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"].to(F)[list(tokens)] * float(cfg["embedding"]["scale"])
    xs = torch.stack([x] * cfg["streams"])

    def sublayer(xs, p: str, q: int, run):
        u = gather_streams(xs, w[f"{p}hc{q}.in"])
        y = run(rms(u, eps) * w[f"{p}norm{q}"].to(F))
        return scatter_streams(xs, y, w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"])

    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        xs = sublayer(xs, p, 1, lambda h: MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps))
        if layer.get("mlp"):
            xs = sublayer(xs, p, 2, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]))
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return linear(rms(xs.sum(0), eps) * w["final.norm"].to(F), w["head"])
