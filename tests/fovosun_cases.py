"""Small Fovosun configurations and weights for the tests.

The configurations differ from one another in every size and option: each kind of layer first, last, twice in a row or
absent; one to sixteen streams; as many key/value heads as heads, fewer, or one; values wider and narrower than one map's
keys, than both maps', and equal; rotations of a whole map, of a part and of none; windows of one token to more than a
page and none; temperatures whose step comes every token to every hundred; convolutions of one to eight taps and none; one
to five retention heads with decays of 0, 1 and between; dense feed-forwards, mixtures of 1 to 9 experts of which 1 to all
are used, with and without a shared expert, unlike limits, and layers without a feed-forward; widths that are no multiple of
16 bytes.
"""
from __future__ import annotations

import json
import os

import torch


def attention(heads, kv_heads, dim, vdim, scale, diff=0.4, conv=0, temp=None, window=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if conv:
        m["conv"] = conv
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def retention(heads, dim, vdim, decay, rot=None):
    assert len(decay) == heads
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    return m


def dense(ff, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, limit=1.1, shared=None):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared[0], "limit": shared[1]} if shared else None}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, streams=3, eps=1e-5, scale=0.7):
    return {"architecture": "Fovosun", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": scale}, "layers": layers}


# every kind of layer, the retention layer without a feed-forward
FO_A = config(64, 300, [
    layer("attention_2", attention(4, 2, 12, 16, 0.4, diff=0.3, window=9, rot=(100.0, 8)), moe(5, 2, 24, 1.3, (40, 0.6))),
    layer("retention", retention(3, 16, 8, [0.5, 0.9, 0.995], rot=(50.0, 16))),
    layer("attention", attention(6, 3, 8, 20, 0.5, diff=0.6, conv=4, temp=(0.7, 5)), dense(72, 0.9))], streams=2, eps=1e-6, scale=1.7)

# retention twice in a row with unlike heads; whole maps turned; one expert; as many key heads as heads; four streams
FO_B = config(96, 257, [
    layer("retention", retention(2, 8, 24, [1.0, 0.7], rot=(1000.0, 4)), dense(100)),
    layer("retention", retention(5, 24, 8, [0.99, 0.0, 0.8, 0.999, 0.3]), moe(3, 3, 36, 0.8)),
    layer("attention", attention(3, 3, 16, 32, 0.3, diff=0.2, conv=2, temp=(0.3, 1)), moe(4, 1, 20, 1.5, (28, 1.1))),
    layer("attention_2", attention(6, 1, 16, 16, 0.35, diff=0.7, window=33, rot=(10000.0, 16)))], streams=4, eps=1e-5, scale=0.4)

# rows that are no multiple of 16 bytes (width 100); odd sizes; a window of one token; no window; no rotation; one stream
FO_C = config(100, 333, [
    layer("attention", attention(5, 1, 6, 10, 0.6, diff=0.5, conv=1, temp=(1.2, 40)), dense(50, 2.0)),
    layer("attention_2", attention(4, 2, 10, 7, 0.4, diff=0.35, window=1, rot=(30.0, 6)), moe(1, 1, 30, 1.0, (12, 2.0))),
    layer("retention", retention(4, 10, 14, [0.95, 0.6, 0.97, 0.2], rot=(20.0, 2)), moe(9, 4, 18, 0.7, (30, 1.0))),
    layer("attention_2", attention(6, 3, 9, 24, 0.5, diff=0.45), dense(44)),
    layer("attention", attention(2, 2, 14, 26, 0.45, diff=0.1, conv=6, temp=(0.5, 13), window=50), dense(31))], streams=1, eps=1e-4)

# the smallest of everything, rows of 60 bytes in bfloat16: one head, sixteen streams
FO_D = config(30, 101, [
    layer("retention", retention(1, 4, 6, [0.9], rot=(10.0, 4)), dense(18)),
    layer("attention", attention(1, 1, 2, 3, 1.0, diff=0.5, conv=3, temp=(0.5, 2)), moe(2, 1, 9, 1.0)),
    layer("attention_2", attention(1, 1, 6, 6, 0.6, diff=0.8, window=3, rot=(10.0, 2)))], streams=16, scale=2.5)

# sizes at which the tensor-core kernels run: rows of 512, stored heads of 32 to 256, pages of 64; windows below and above
# a page; groups of more than 16 query rows per key head; a stored head above the largest the tensor cores take
FO_E = config(512, 3000, [
    layer("attention", attention(8, 2, 32, 64, 0.18, diff=0.5, conv=4, temp=(0.5, 50)), dense(640, 3.0)),
    layer("retention", retention(4, 128, 64, [0.97, 0.999, 0.8, 0.5], rot=(5000.0, 128)), moe(8, 2, 192, 2.0, (192, 1.0))),
    layer("attention_2", attention(4, 4, 64, 128, 0.12, diff=0.3, window=70, rot=(10000.0, 32)), moe(16, 3, 128, 1.0, (64, 2.5))),
    layer("retention", retention(2, 40, 96, [0.9, 0.9995], rot=(100.0, 24))),
    layer("attention_2", attention(18, 1, 16, 16, 0.25, diff=0.2, window=129, rot=(500.0, 16)), dense(256)),
    layer("attention", attention(2, 1, 104, 72, 0.1, diff=0.6, conv=3, temp=(0.4, 100)), dense(320)),
    layer("retention", retention(2, 256, 32, [0.95, 0.99], rot=(3000.0, 64)), dense(448)),
    layer("attention_2", attention(2, 2, 136, 40, 0.08, diff=0.4, window=260, rot=(2000.0, 136)), dense(128))], streams=3, eps=1e-6)

CASES = {"A": (FO_A, [5, 17, 23, 40, 11, 30], 4), "B": (FO_B, [1, 31, 40, 70, 9, 50], 8), "C": (FO_C, [3, 50, 64, 29, 77, 2], 16),
         "D": (FO_D, [4, 19, 1, 33, 8, 12], 4)}


def draw_tensors(cfg_dict: dict, seed: int, sharp: float = 1.0) -> dict:
    """Random weights by tensor name (bfloat16), drawn here with torch's generator.  Norm weights lie around one; the
    queries' projections are `sharp` times as large, which spreads the scores; filters reach every tap; the streams are
    read and mixed unlike one another, near a sum of weight one, so that they neither vanish nor grow; lambda's vectors
    move it away from its constant; router biases are of the logits' size."""
    from kungfu_b200.api import load_config
    from kungfu_b200 import registry
    cfg = load_config(json.loads(json.dumps(cfg_dict)))
    g = torch.Generator().manual_seed(seed)
    n = cfg.streams
    out = {}
    for spec in registry.find(cfg.architecture).tensor_specs(cfg):
        name = spec.name
        x = torch.randn(tuple(spec.shape), generator=g)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            x = 1.0 + 0.2 * x
        elif name.endswith(".in"):
            x = (1.0 + 0.5 * x) / n
        elif name.endswith(".out"):
            x = 0.6 + 0.4 * x
        elif name.endswith(".mix"):
            x = 0.7 * torch.eye(n) + (0.3 + 0.2 * x) / n
        elif name.endswith(".conv"):
            x = 0.5 * x
        elif name.endswith(("lq1", "lk1", "lq2", "lk2")):
            x = 0.6 * x / spec.shape[0] ** 0.25
        elif name.endswith("router.b"):
            x = 0.7 * x
        elif name.endswith(".b"):
            x = 0.3 * x
        elif name == "embed":
            x = 0.8 * x
        else:
            x = x / (spec.shape[-1] ** 0.5)                  # projections keep the spread of their input
            if name.endswith("mix.q"):
                x = sharp * x
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
