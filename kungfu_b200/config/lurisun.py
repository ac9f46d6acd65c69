"""Lurisun hyperparameters, read from the model's own config.json.

A Lurisun file lists its layers one by one; nothing is implied by a layer's index and no size is fixed by the design.

  architecture             "Lurisun"
  width, vocab             residual width, vocabulary
  norm.eps                 epsilon of every RMS norm
  logit_scale              factor of the output logits
  canon.taps               taps of the convolution in front of every mixer
  embedding.bigram         mul_prev, mul_cur, buckets: the row of the second embedding table a pair of tokens reads
  layers[i].type           latent_attention | lightning | attention
  layers[i].mixer          latent_attention: heads, dim (query/key size), vdim (value size), kv_rank, q_rank, scale,
                                             mask {size} (absent: every earlier token is seen)
                           lightning:        heads, dim, vdim, decay (one number per head)
                           attention:        heads, kv_heads, dim, vdim (equal to dim: the keys are the values), scale,
                                             mask {size} (absent: every earlier token is seen), rot {base, dims} | null
  layers[i].mlp            null | {kind: dense, ff}
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field

from .base import ConfigError, KeyReader

LATENT, LIGHTNING, ATTENTION = "latent_attention", "lightning", "attention"


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int | None = None


@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None = None
    rot_base: float = 10000.0
    rot_dims: int = 0                        # 0: no rotation


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    ff: int = 0                              # 0: no feed-forward


@dataclass(frozen=True)
class PairSpec:
    mul_prev: int
    mul_cur: int
    buckets: int


def _sub(k: KeyReader, key: str, required: bool = True) -> KeyReader | None:
    raw = k.raw.get(key)
    k.read.add(key)
    if raw is None:
        if required:
            raise ConfigError(f"{k.where}: required key '{key}' is missing")
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"{k.where}: key '{key}' must be an object, found {raw!r}")
    return KeyReader(raw, f"{k.where}: {key}")


def _mask_size(mk: KeyReader) -> int | None:
    m = _sub(mk, "mask", required=False)
    return m.int("size", None, min=1) if m is not None else None


def _mixer(kind: str, mk: KeyReader):
    heads, dim = mk.int("heads", min=1), mk.int("dim", min=1)
    if kind == LATENT:
        return LatentSpec(heads, dim, mk.int("vdim", dim, min=1), mk.int("kv_rank", min=1), mk.int("q_rank", min=1),
                          mk.float("scale"), _mask_size(mk))
    if kind == LIGHTNING:
        decay = mk.list("decay")
        if not all(isinstance(a, (int, float)) and not isinstance(a, bool) for a in decay):
            raise ConfigError(f"{mk.where}: key 'decay' must be a list of numbers, found {decay!r}")
        return LightningSpec(heads, dim, mk.int("vdim", dim, min=1), tuple(float(a) for a in decay))
    rk = _sub(mk, "rot", required=False)
    base, dims = (rk.float("base"), rk.int("dims", dim, min=0)) if rk is not None else (10000.0, 0)
    return AttentionSpec(heads, mk.int("kv_heads", heads, min=1), dim, mk.int("vdim", dim, min=1), mk.float("scale"),
                         _mask_size(mk), base, dims)


def _ff(k: KeyReader | None) -> int:
    if k is None:
        return 0
    k.str("kind", "dense", choices=("dense",))
    return k.int("ff", min=1)


@dataclass(frozen=True)
class LurisunConfig:
    architecture: str
    width: int
    vocab: int
    norm_eps: float
    logit_scale: float
    taps: int
    pair: PairSpec
    layers: tuple = field(default_factory=tuple)         # LayerSpec per layer

    # what the engine and the command line ask of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "LurisunConfig":
        k = KeyReader(raw, where)
        arch = k.str("architecture")
        width, vocab = k.int("width", min=1), k.int("vocab", min=1)
        b = _sub(_sub(k, "embedding"), "bigram")
        pair = PairSpec(b.int("mul_prev"), b.int("mul_cur"), b.int("buckets", min=1))
        layers = []
        for i, e in enumerate(k.list("layers")):
            ek = KeyReader(e, f"{where}: layers[{i}]")
            kind = ek.str("type", choices=(LATENT, LIGHTNING, ATTENTION))
            layers.append(LayerSpec(kind, _mixer(kind, _sub(ek, "mixer")), _ff(_sub(ek, "mlp", required=False))))
        cfg = cls(arch, width, vocab, _sub(k, "norm").float("eps"), k.float("logit_scale", 1.0),
                  _sub(k, "canon").int("taps", min=1), pair, tuple(layers))
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config") -> None:
        if not self.layers:
            raise ConfigError(f"{where}: 'layers' is empty")
        if not self.norm_eps > 0:
            raise ConfigError(f"{where}: norm.eps must be positive, found {self.norm_eps}")
        if self.taps > 8:
            raise ConfigError(f"{where}: canon.taps above 8 is not supported, found {self.taps}")
        for i, l in enumerate(self.layers):
            at, m = f"{where}: layers[{i}]", l.mixer
            if l.type == LATENT:
                if m.kv_rank > 512:
                    raise ConfigError(f"{at}: kv_rank above 512 is not supported, found {m.kv_rank}")
            elif l.type == LIGHTNING:
                if len(m.decay) != m.heads:
                    raise ConfigError(f"{at}: 'decay' lists {len(m.decay)} numbers for {m.heads} heads")
                if not all(0.0 <= a <= 1.0 for a in m.decay):
                    raise ConfigError(f"{at}: 'decay' must lie between 0 and 1, found {list(m.decay)}")
                if m.dim > 256:
                    raise ConfigError(f"{at}: key size {m.dim} is above 256")
            else:
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: heads {m.heads} is not a multiple of kv_heads {m.kv_heads}")
                if m.vdim != m.dim:
                    raise ConfigError(f"{at}: vdim {m.vdim} must equal dim {m.dim}: the keys are the values")
                if m.dim > 256:
                    raise ConfigError(f"{at}: head sizes above 256 are not supported, found {m.dim}")
                if m.rot_dims % 2 or m.rot_dims > m.dim:
                    raise ConfigError(f"{at}: rot.dims {m.rot_dims} must be even and at most dim {m.dim}")

    def to_dict(self) -> dict:
        """A config.json dictionary that `from_dict` reads back to this configuration."""
        layers = []
        for l in self.layers:
            m = l.mixer
            if l.type == LATENT:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale}
                size = m.window
            elif l.type == LIGHTNING:
                mixer, size = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}, None
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                         "rot": {"base": m.rot_base, "dims": m.rot_dims} if m.rot_dims else None}
                size = m.chunk
            if size is not None:
                mixer["mask"] = {"size": size}
            layers.append({"type": l.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "canon": {"taps": self.taps},
                "embedding": {"bigram": dataclasses.asdict(self.pair)}, "layers": layers}

    def replace(self, **kw) -> "LurisunConfig":
        cfg = dataclasses.replace(self, **kw)
        cfg.validate()
        return cfg

    def state_summary(self, element_size: int = 2) -> list:
        """Per layer, what it keeps per request: bytes per token of its pages, the window that bounds them, fixed bytes (the
        last inputs of the convolution, and a lightning layer's memory)."""
        from ..ops import attention_head_size
        from ..parts.latent import latent_head_size
        tail = 4 * (self.taps - 1) * self.width
        out = []
        for i, l in enumerate(self.layers):
            m = l.mixer
            row = {"layer": i, "fixed_bytes": tail, "window": None, "bytes_per_token": 0}
            if l.type == LATENT:
                row.update(kind="latent_pages", window=m.window, bytes_per_token=2 * latent_head_size(m.kv_rank) * element_size)
            elif l.type == LIGHTNING:
                row.update(kind="memory", fixed_bytes=tail + 4 * m.heads * m.dim * m.vdim)
            else:
                row.update(kind="kv_pages", window=m.chunk, bytes_per_token=2 * m.kv_heads * attention_head_size(m.dim) * element_size)
            out.append(row)
        return out
