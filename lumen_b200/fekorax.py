"""Fekorax: a decoder given as a list of layers (matrix-memory layers; grouped-query attention over chunks with sinks, head gates and
shared keys and values; gated feed-forwards; a norm before and after every sublayer).  The reader of its config.json and the
host side of `lumen_decoder_new`.

`LayerConfig` and `FekoraxConfig` carry every size and constant; nothing here or in the library rests on a particular
model's values.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from . import _lib
from ._lib import BF16, F32, DecoderConfigC, DecoderLayerC
from .model import DecoderModel


@dataclass
class RotConfig:
    """Rotation of the first `dims` numbers of a head; `factor` 0: frequencies as they are."""

    dims: int
    base: float
    factor: float = 0.0
    low: float = 0.0
    high: float = 0.0
    original: float = 0.0

    @classmethod
    def from_dict(cls, d: dict | None) -> "RotConfig":
        if not d:
            return cls(0, 1.0)
        s = d.get("scaling") or {}
        return cls(int(d["dims"]), float(d["base"]), float(s.get("factor", 0.0)), float(s.get("low", 0.0)), float(s.get("high", 0.0)),
                   float(s.get("original", 0.0)))


@dataclass
class LayerConfig:
    """One layer: a mixer ("mlstm" or "attention"), then a feed-forward (`ff` 0: none)."""

    type: str
    heads: int
    dim: int
    vdim: int
    gate_cap: float = 0.0                 # mlstm
    kv_heads: int = 0                     # attention
    kv_from: int | None = None
    scale: float = 1.0
    chunk: int = 0                        # 0: every earlier position is seen
    rot: RotConfig = field(default_factory=lambda: RotConfig(0, 1.0))
    ff: int = 0

    @classmethod
    def from_dict(cls, d: dict) -> "LayerConfig":
        m, mlp = d["mixer"], d.get("mlp")
        layer = cls(d["type"], int(m["heads"]), int(m["dim"]), int(m["vdim"]))
        if layer.type == "mlstm":
            layer.gate_cap = float(m["gate_cap"])
        elif layer.type == "attention":
            layer.kv_heads = int(m["kv_heads"])
            layer.kv_from = None if m.get("kv_from") is None else int(m["kv_from"])
            layer.scale = float(m["scale"])
            layer.chunk = int((m.get("mask") or {}).get("size", 0))
            layer.rot = RotConfig.from_dict(m.get("rot"))
        else:
            raise ValueError(f"unknown mixer {layer.type!r}")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
            layer.ff = int(mlp["ff"])
        return layer

    def to_c(self) -> DecoderLayerC:
        r = self.rot
        return DecoderLayerC(
            heads=self.heads, dim=self.dim, vdim=self.vdim, rot_dims=r.dims, rot_base=r.base, scale=self.scale,
            mlp_kind=_lib.MLP_GATED_GELU if self.ff else _lib.MLP_NONE, ff=self.ff,
            mixer=_lib.MIXER_MLSTM if self.type == "mlstm" else _lib.MIXER_ATTENTION, kv_heads=self.kv_heads,
            kv_from=-1 if self.kv_from is None else self.kv_from, chunk=self.chunk, rot_factor=r.factor, rot_low=r.low, rot_high=r.high,
            rot_original=r.original, gate_cap=self.gate_cap)


@dataclass
class FekoraxConfig:
    vocab_size: int
    width: int
    layers: list = field(default_factory=list)
    norm_eps: float = 1e-5
    max_seq_len: int = 2048
    embed_scale: float = 1.0
    weight_dtype: str = "f32"

    @classmethod
    def from_dict(cls, d: dict, max_seq_len: int, weight_dtype: str) -> "FekoraxConfig":
        return cls(int(d["vocab"]), int(d["width"]), [LayerConfig.from_dict(x) for x in d["layers"]], float(d["norm"]["eps"]), max_seq_len,
                   float((d.get("embedding") or {}).get("scale", 1.0)), weight_dtype)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def to_c(self) -> DecoderConfigC:
        arr = (DecoderLayerC * max(len(self.layers), 1))(*[x.to_c() for x in self.layers])
        return DecoderConfigC(vocab_size=self.vocab_size, width=self.width, num_layers=len(self.layers), layers=arr, norm_eps=self.norm_eps,
                              max_seq_len=self.max_seq_len, weight_dtype=BF16 if self.weight_dtype == "bf16" else F32,
                              embed_scale=self.embed_scale, tied_head=1, norms=_lib.NORM_BOTH)

    def param_shapes(self) -> dict:
        w = self.width
        shapes = {"embed": (self.vocab_size, w), "final.norm": (w,)}
        for i, k in enumerate(self.layers):
            p, h = f"l{i}.", k.heads
            shapes.update({p + "norm1": (w,), p + "norm1b": (w,), p + "mix.q": (h * k.dim, w), p + "mix.o": (w, h * k.vdim)})
            if k.type == "mlstm":
                shapes.update({p + "mix.k": (h * k.dim, w), p + "mix.v": (h * k.vdim, w), p + "mix.g": (h * k.vdim, w),
                               p + "mix.norm": (h * k.vdim,), p + "mix.i": (h, w), p + "mix.i.b": (h,), p + "mix.f": (h, w), p + "mix.f.b": (h,)})
            else:
                shapes.update({p + "mix.q.norm": (k.dim,), p + "mix.sink": (h,), p + "mix.g": (h, w)})
                if k.kv_from is None:
                    shapes.update({p + "mix.k": (k.kv_heads * k.dim, w), p + "mix.v": (k.kv_heads * k.vdim, w), p + "mix.k.norm": (k.dim,)})
            if k.ff:
                shapes.update({p + "norm2": (w,), p + "norm2b": (w,), p + "mlp.gate": (k.ff, w), p + "mlp.up": (k.ff, w), p + "mlp.down": (w, k.ff)})
        return shapes


class FekoraxModel(DecoderModel):
    def _cache_shape(self, layer: int, batch: int) -> tuple:
        k = self.config.layers[layer]
        return (batch, k.heads, k.dim, k.vdim) if k.type == "mlstm" else (batch, k.kv_heads, self.config.max_seq_len, k.dim)
