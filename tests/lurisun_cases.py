"""Small Lurisun configurations and weights for the tests.

The configurations differ from one another in every size and option: each kind of layer first, last, twice in a row or
absent; as many key/value heads as heads, fewer, or one; rotations of a whole head, of a part and of none; chunks and
windows of one token to more than a page, and layers without a mask; latents that fill their stored head or not, query
latents smaller and larger than the key latent, values wider and narrower than keys; one to five linear-attention heads
with decays of 0, 1 and between, keys wider and narrower than values; convolutions of one to six taps; pair tables of
one row to hundreds; layers without a feed-forward; a logit factor of 1, above and below; widths that are no multiple of
16 bytes.
"""
from __future__ import annotations

import json
import os

import torch


def latent(heads, dim, vdim, kv_rank, q_rank, scale, window=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def attention(heads, kv_heads, dim, scale, chunk=None, rot_dims=0, base=10000.0):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
    return m


def layer(kind, mixer, ff=0):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5, logit_scale=1.0, taps=4, pair=(7, 3, 61)):
    return {"architecture": "Lurisun", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "canon": {"taps": taps}, "embedding": {"bigram": dict(zip(("mul_prev", "mul_cur", "buckets"), pair))},
            "layers": layers}


# every kind of layer, the lightning layer without a feed-forward
LU_A = config(64, 300, [
    layer("attention", attention(4, 2, 24, 0.2, chunk=9, rot_dims=8, base=100.0), 72),
    layer("lightning", lightning(3, 16, 8, [0.5, 0.9, 0.995])),
    layer("latent_attention", latent(3, 8, 12, 20, 28, 0.4, window=7), 40)], eps=1e-6, logit_scale=3.5)

# lightning twice in a row with unlike heads; whole heads turned; a latent wider than its queries' latent, no mask there
LU_B = config(96, 257, [
    layer("lightning", lightning(2, 8, 24, [1.0, 0.7]), 100),
    layer("lightning", lightning(5, 24, 8, [0.99, 0.0, 0.8, 0.999, 0.3]), 36),
    layer("latent_attention", latent(2, 24, 16, 48, 16, 0.2), 64),
    layer("attention", attention(6, 6, 16, 0.25, chunk=33, rot_dims=16))], eps=1e-5, logit_scale=0.4, taps=2, pair=(1, 1, 400))

# rows that are no multiple of 16 bytes (width 100); odd sizes; a chunk and a window of one token; no rotation; no mask
LU_C = config(100, 333, [
    layer("latent_attention", latent(5, 10, 6, 18, 30, 0.3, window=1), 50),
    layer("attention", attention(5, 1, 10, 0.3, chunk=1), 30),
    layer("lightning", lightning(4, 10, 14, [0.95, 0.6, 0.97, 0.2]), 70),
    layer("attention", attention(6, 3, 6, 0.5), 44),
    layer("latent_attention", latent(2, 6, 20, 34, 12, 0.35, window=50))], eps=1e-4, logit_scale=1.0, taps=6, pair=(131, 977, 89))

# the smallest of everything, rows of 60 bytes in bfloat16: one head, one tap, a pair table of two rows
LU_D = config(30, 101, [
    layer("lightning", lightning(1, 4, 6, [0.9]), 18),
    layer("latent_attention", latent(1, 6, 5, 7, 3, 0.7, window=3), 12),
    layer("attention", attention(1, 1, 6, 0.6, chunk=2, rot_dims=2, base=10.0))], logit_scale=2.5, taps=1, pair=(2, 5, 1))

# sizes at which the tensor-core kernels run: rows of 512, heads of 64 to 128 and 256, pages of 64; chunks and windows
# below and above a page
LU_E = config(512, 3000, [
    layer("attention", attention(8, 2, 64, 0.1, chunk=100, rot_dims=32), 640),
    layer("lightning", lightning(4, 128, 64, [0.97, 0.999, 0.8, 0.5]), 384),
    layer("latent_attention", latent(8, 32, 64, 112, 72, 0.15, window=70), 768),
    layer("lightning", lightning(2, 40, 96, [0.9, 0.9995])),
    layer("attention", attention(4, 4, 104, 0.08, chunk=260, rot_dims=104, base=5000.0), 256),
    layer("latent_attention", latent(20, 16, 24, 60, 128, 0.25, window=129), 320),
    layer("lightning", lightning(2, 256, 32, [0.95, 0.99]), 448)], eps=1e-6, logit_scale=1.7, taps=3, pair=(40503, 17, 1009))

CASES = {"A": (LU_A, [5, 17, 23, 40, 11, 30], 4), "B": (LU_B, [1, 31, 40, 70, 9, 50], 8), "C": (LU_C, [3, 50, 64, 29, 77, 2], 16),
         "D": (LU_D, [4, 19, 1, 33, 8, 12], 4)}


def draw_tensors(cfg_dict: dict, seed: int, sharp: float = 1.0) -> dict:
    """Random weights by tensor name (bfloat16), drawn here with torch's generator.  Norm weights lie around one; the
    weights of the norms over q and k around `sharp`, which spreads the scores; the sigmoid's biases lie around -2, so
    that many keys weigh little and few weigh much; filters reach every tap; the two embedding tables are alike in size."""
    from kungfu_b200.api import load_config
    from kungfu_b200 import registry
    cfg = load_config(json.loads(json.dumps(cfg_dict)))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for spec in registry.find(cfg.architecture).tensor_specs(cfg):
        name = spec.name
        x = torch.randn(tuple(spec.shape), generator=g)
        if name.endswith(("q.norm", "k.norm")):
            x = sharp * (1.0 + 0.2 * x)
        elif name.endswith("norm") or name.endswith(("norm1", "norm2")):
            x = 1.0 + 0.2 * x
        elif name.endswith("pb"):
            x = -2.0 + x
        elif name.endswith(".b"):
            x = 0.3 * x
        elif name.endswith("canon1"):
            x = 0.4 * x
        elif name in ("embed", "bigram"):
            x = 0.5 * x
        else:
            x = x / (spec.shape[-1] ** 0.5)                  # projections keep the spread of their input
        out[name] = x.to(torch.bfloat16)
    return out


def write_tensors(folder: str, cfg_dict: dict, tensors: dict) -> str:
    from kungfu_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg_dict, f)
    return folder


def write_model(folder: str, cfg_dict: dict, seed: int, sharp: float = 1.0) -> str:
    return write_tensors(folder, cfg_dict, draw_tensors(cfg_dict, seed, sharp))
