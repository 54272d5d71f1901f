"""Fegetar: a decoder given as a list of layers (latent attention; dense or routed feed-forwards; bigram and per-layer token
inputs).  The reader of its config.json and the host side of `lumen_decoder_new`.

`LayerConfig` and `FegetarConfig` carry every size and constant; nothing here or in the library rests on a
particular model's values.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from . import _lib
from ._lib import BF16, F32, DecoderConfigC, DecoderLayerC
from .model import DecoderModel


@dataclass
class ExpertConfig:
    ff: int
    limit: float


@dataclass
class LayerConfig:
    """One layer: latent attention, then a feed-forward: none (`ff` and `experts` 0), dense (`ff`), or routed (`experts`)."""

    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    rot_dims: int
    rot_base: float
    scale: float
    ff: int = 0
    experts: int = 0
    top: int = 0
    expert: ExpertConfig | None = None
    shared: ExpertConfig | None = None

    @classmethod
    def from_dict(cls, d: dict) -> "LayerConfig":
        if d["type"] != "latent_attention":
            raise ValueError(f"unknown mixer {d['type']!r}")
        m, rot, mlp = d["mixer"], d["mixer"]["rot"], d.get("mlp")
        layer = cls(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), int(rot["dims"]),
                    float(rot["base"]), float(m["scale"]))
        if mlp is None:
            return layer
        if mlp["kind"] == "dense":
            layer.ff = int(mlp["ff"])
        elif mlp["kind"] == "moe":
            layer.experts, layer.top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
            layer.expert = ExpertConfig(int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"]))
            if mlp.get("shared"):
                layer.shared = ExpertConfig(int(mlp["shared"]["ff"]), float(mlp["shared"]["limit"]))
        else:
            raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
        return layer

    def to_c(self) -> DecoderLayerC:
        kind = _lib.MLP_MOE if self.experts else _lib.MLP_DENSE if self.ff else _lib.MLP_NONE
        e, s = self.expert or ExpertConfig(0, 0.0), self.shared or ExpertConfig(0, 0.0)
        return DecoderLayerC(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.rot_dims, self.rot_base, self.scale, kind,
                             self.ff, self.experts, self.top, e.ff, e.limit, s.ff, s.limit, _lib.MIXER_LATENT, 0, -1)


@dataclass
class FegetarConfig:
    vocab_size: int
    width: int
    layers: list = field(default_factory=list)
    norm_eps: float = 1e-5
    max_seq_len: int = 2048
    bigram_buckets: int = 0
    bigram_mul_prev: int = 0
    bigram_mul_cur: int = 0
    side_dim: int = 0
    weight_dtype: str = "f32"

    @classmethod
    def from_dict(cls, d: dict, max_seq_len: int, weight_dtype: str) -> "FegetarConfig":
        big = (d.get("embedding") or {}).get("bigram") or {}
        side = d.get("token_side") or {}
        return cls(int(d["vocab"]), int(d["width"]), [LayerConfig.from_dict(x) for x in d["layers"]], float(d["norm"]["eps"]), max_seq_len,
                   int(big.get("buckets", 0)), int(big.get("mul_prev", 0)), int(big.get("mul_cur", 0)), int(side.get("dim", 0)), weight_dtype)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def to_c(self) -> DecoderConfigC:
        arr = (DecoderLayerC * max(len(self.layers), 1))(*[x.to_c() for x in self.layers])
        return DecoderConfigC(self.vocab_size, self.width, len(self.layers), arr, self.norm_eps, self.max_seq_len, self.bigram_buckets,
                              self.bigram_mul_prev, self.bigram_mul_cur, self.side_dim, BF16 if self.weight_dtype == "bf16" else F32, 1.0, 0, _lib.NORM_OUTPUT)

    def param_shapes(self) -> dict:
        w, v = self.width, self.vocab_size
        shapes = {"embed": (v, w), "final.norm": (w,), "head": (v, w)}
        if self.bigram_buckets:
            shapes["bigram"] = (self.bigram_buckets + 1, w)
        if self.side_dim:
            shapes["side.embed"] = (v, len(self.layers) * self.side_dim)
        for i, k in enumerate(self.layers):
            p = f"l{i}."
            shapes.update({
                p + "norm1": (w,), p + "mix.q": (k.heads * (k.dim + k.rot_dim), w), p + "mix.dkv": (k.kv_rank + k.rot_dim, w),
                p + "mix.dkv.norm": (k.kv_rank,), p + "mix.uk": (k.heads * k.dim, k.kv_rank), p + "mix.uv": (k.heads * k.vdim, k.kv_rank),
                p + "mix.g": (k.heads, w), p + "mix.o": (w, k.heads * k.vdim),
            })
            if k.ff or k.experts:
                shapes[p + "norm2"] = (w,)
            if k.experts:
                shapes[p + "mlp.router"] = (k.experts, w)
                parts = [(f"mlp.e{e}", k.expert.ff) for e in range(k.experts)] + ([("mlp.shared", k.shared.ff)] if k.shared else [])
                for name, ff in parts:
                    shapes.update({f"{p}{name}.gate": (ff, w), f"{p}{name}.up": (ff, w), f"{p}{name}.down": (w, ff)})
            elif k.ff:
                shapes.update({p + "mlp.up": (k.ff, w), p + "mlp.down": (w, k.ff)})
            if self.side_dim:
                shapes.update({p + "side.gate": (self.side_dim, w), p + "side.proj": (w, self.side_dim), p + "side.norm": (w,)})
        return shapes


class FegetarModel(DecoderModel):
    def _cache_shape(self, layer: int, batch: int) -> tuple:
        k = self.config.layers[layer]
        return batch, 1, self.config.max_seq_len, -(-(k.kv_rank + k.rot_dim) // 16) * 16
