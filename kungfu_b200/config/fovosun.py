"""Fovosun hyperparameters, read from the model's own config.json.

A Fovosun file lists its layers one by one; nothing is implied by a layer's index and no size is fixed by the design.

  architecture             "Fovosun"
  width, vocab             residual width, vocabulary
  streams                  copies of the residual stream
  norm.eps                 epsilon of every RMS norm
  embedding.scale          factor of the embedded rows (default 1)
  layers[i].type           attention | attention_2 | retention
  layers[i].mixer          attention, attention_2 (differential attention): heads, kv_heads, dim (query/key size of one map),
                             vdim (value size), scale, diff, and, where present: conv (taps of the convolutions over q, k
                             and v), q_temp {coef, every}, rot {base, dims}, mask {size} (sliding window).  attention has a
                             gate per head, attention_2 biases on q, k and v
                           retention: heads, dim, vdim, decay (one number per head), rot {base, dims}
  layers[i].mlp            null | {kind: dense, ff, limit} | {kind: moe, expert {ff, limit}, router {experts, top},
                             shared {ff, limit} | null}
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field

from .base import ConfigError, KeyReader

ATTENTION, BIASED_ATTENTION, RETENTION = "attention", "attention_2", "retention"


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    taps: int = 0                            # 0: no convolution
    temperature: tuple | None = None         # (coef, every)
    window: int | None = None
    rot_base: float = 10000.0
    rot_dims: int = 0                        # 0: no rotation


@dataclass(frozen=True)
class RetentionSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot_base: float = 10000.0
    rot_dims: int = 0


@dataclass(frozen=True)
class FfnSpec:
    ff: int
    limit: float


@dataclass(frozen=True)
class MlpSpec:
    kind: str                                # dense | moe
    ffn: FfnSpec                             # the feed-forward itself, or one expert
    experts: int = 0
    top: int = 0
    shared: FfnSpec | None = None


@dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: object
    mlp: MlpSpec | None


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


def _rot(mk: KeyReader, dim: int) -> tuple:
    rk = _sub(mk, "rot", required=False)
    return (rk.float("base"), rk.int("dims", dim, min=0)) if rk is not None else (10000.0, 0)


def _mixer(kind: str, mk: KeyReader):
    heads, dim = mk.int("heads", min=1), mk.int("dim", min=1)
    vdim = mk.int("vdim", dim, min=1)
    base, dims = _rot(mk, dim)
    if kind == RETENTION:
        decay = mk.list("decay")
        if not all(isinstance(a, (int, float)) and not isinstance(a, bool) for a in decay):
            raise ConfigError(f"{mk.where}: key 'decay' must be a list of numbers, found {decay!r}")
        return RetentionSpec(heads, dim, vdim, tuple(float(a) for a in decay), base, dims)
    tk, wk = _sub(mk, "q_temp", required=False), _sub(mk, "mask", required=False)
    return AttentionSpec(heads, mk.int("kv_heads", heads, min=1), dim, vdim, mk.float("scale"), mk.float("diff"),
                         mk.int("conv", 0, min=0), (tk.float("coef"), tk.int("every", min=1)) if tk is not None else None,
                         wk.int("size", None, min=1) if wk is not None else None, base, dims)


def _ffn(k: KeyReader) -> FfnSpec:
    return FfnSpec(k.int("ff", min=1), k.float("limit"))


def _mlp(k: KeyReader | None) -> MlpSpec | None:
    if k is None:
        return None
    if k.str("kind", "dense", choices=("dense", "moe")) == "dense":
        return MlpSpec("dense", _ffn(k))
    r, s = _sub(k, "router"), _sub(k, "shared", required=False)
    return MlpSpec("moe", _ffn(_sub(k, "expert")), r.int("experts", min=1), r.int("top", min=1), _ffn(s) if s is not None else None)


@dataclass(frozen=True)
class FovosunConfig:
    architecture: str
    width: int
    vocab: int
    streams: int
    norm_eps: float
    embedding_scale: float
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
    def from_dict(cls, raw: dict, where: str = "config.json") -> "FovosunConfig":
        k = KeyReader(raw, where)
        arch = k.str("architecture")
        ek = _sub(k, "embedding", required=False)
        layers = []
        for i, e in enumerate(k.list("layers")):
            lk = KeyReader(e, f"{where}: layers[{i}]")
            kind = lk.str("type", choices=(ATTENTION, BIASED_ATTENTION, RETENTION))
            layers.append(LayerSpec(kind, _mixer(kind, _sub(lk, "mixer")), _mlp(_sub(lk, "mlp", required=False))))
        cfg = cls(arch, k.int("width", min=1), k.int("vocab", min=1), k.int("streams", min=1), _sub(k, "norm").float("eps"),
                  ek.float("scale", 1.0) if ek is not None else 1.0, tuple(layers))
        cfg.validate(where)
        return cfg

    def validate(self, where: str = "config") -> None:
        from ..ops import MAX_GENERIC_HEAD_DIM, MAX_STREAMS
        if not self.layers:
            raise ConfigError(f"{where}: 'layers' is empty")
        if not self.norm_eps > 0:
            raise ConfigError(f"{where}: norm.eps must be positive, found {self.norm_eps}")
        if self.streams > MAX_STREAMS:
            raise ConfigError(f"{where}: more than {MAX_STREAMS} streams are not supported, found {self.streams}")
        for i, l in enumerate(self.layers):
            at, m, f = f"{where}: layers[{i}]", l.mixer, l.mlp
            if m.rot_dims % 2 or m.rot_dims > m.dim:
                raise ConfigError(f"{at}: rot.dims {m.rot_dims} must be even and at most dim {m.dim}")
            if l.type == RETENTION:
                if len(m.decay) != m.heads:
                    raise ConfigError(f"{at}: 'decay' lists {len(m.decay)} numbers for {m.heads} heads")
                if not all(0.0 <= a <= 1.0 for a in m.decay):
                    raise ConfigError(f"{at}: 'decay' must lie between 0 and 1, found {list(m.decay)}")
                if m.dim > 256:
                    raise ConfigError(f"{at}: key size {m.dim} is above 256")
            else:
                if m.heads % m.kv_heads:
                    raise ConfigError(f"{at}: heads {m.heads} is not a multiple of kv_heads {m.kv_heads}")
                if max(2 * m.dim, m.vdim) > MAX_GENERIC_HEAD_DIM:
                    raise ConfigError(f"{at}: dim above {MAX_GENERIC_HEAD_DIM // 2} or vdim above {MAX_GENERIC_HEAD_DIM} is not "
                                      f"supported, found {m.dim} and {m.vdim}")
                if m.taps > 8:
                    raise ConfigError(f"{at}: conv above 8 taps is not supported, found {m.taps}")
            if f is not None and f.kind == "moe":
                if f.top > f.experts:
                    raise ConfigError(f"{at}: mlp: top {f.top} of {f.experts} experts")
                if f.experts > 1024:
                    raise ConfigError(f"{at}: mlp: more than 1024 experts are not supported")

    def to_dict(self) -> dict:
        """A config.json dictionary that `from_dict` reads back to this configuration."""
        def ffn(s: FfnSpec) -> dict:
            return {"ff": s.ff, "limit": s.limit}

        layers = []
        for l in self.layers:
            m, f = l.mixer, l.mlp
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
            if m.rot_dims:
                mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
            if l.type == RETENTION:
                mixer["decay"] = list(m.decay)
            else:
                mixer.update(kv_heads=m.kv_heads, scale=m.scale, diff=m.diff)
                if m.taps:
                    mixer["conv"] = m.taps
                if m.temperature is not None:
                    mixer["q_temp"] = {"coef": m.temperature[0], "every": m.temperature[1]}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window}
            mlp = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", **ffn(f.ffn)}
            elif f is not None:
                mlp = {"kind": "moe", "expert": ffn(f.ffn), "router": {"experts": f.experts, "top": f.top},
                       "shared": ffn(f.shared) if f.shared is not None else None}
            layers.append({"type": l.type, "mixer": mixer, "mlp": mlp})
        return {"architecture": self.architecture, "width": self.width, "vocab": self.vocab, "streams": self.streams,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "layers": layers}

    def replace(self, **kw) -> "FovosunConfig":
        cfg = dataclasses.replace(self, **kw)
        cfg.validate()
        return cfg

    def state_summary(self, element_size: int = 2) -> list:
        """Per layer, what it keeps per request: bytes per token of its pages, the window that bounds them, fixed bytes (the
        last inputs of the convolutions, or a retention layer's memory)."""
        from ..parts.latent import latent_head_size
        out = []
        for i, l in enumerate(self.layers):
            m = l.mixer
            row = {"layer": i, "fixed_bytes": 0, "window": None, "bytes_per_token": 0}
            if l.type == RETENTION:
                row.update(kind="memory", fixed_bytes=4 * m.heads * m.dim * m.vdim)
            else:
                channels = 2 * (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim
                row.update(kind="kv_pages", window=m.window, fixed_bytes=4 * max(m.taps - 1, 0) * channels,
                           bytes_per_token=2 * m.kv_heads * latent_head_size(max(2 * m.dim, m.vdim)) * element_size)
            out.append(row)
        return out
