"""LlamaConfig / LlamaModel — host-side mirror of src/models/llama.rs (inference methods)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import numpy as np

from ._lib import BF16, F32, LlamaConfigC
from .model import LanguageModel


@dataclass
class LlamaConfig:
    """src/models/llama.rs:11-37 (TinyLlama defaults) plus what the reference lacks: `head_dim`
    (0 = hidden/heads), `qk_norm` (Qwen3 per-head q/k RMSNorm) and `weight_dtype` ("f32"/"bf16")."""

    vocab_size: int = 32000
    hidden_size: int = 2048
    intermediate_size: int = 5632
    num_hidden_layers: int = 22
    num_attention_heads: int = 32
    num_key_value_heads: int = 4
    rms_norm_eps: float = 1e-5
    max_seq_len: int = 2048
    rope_theta: float = 10000.0
    head_dim: int = 0
    qk_norm: bool = False
    weight_dtype: str = "f32"

    def to_c(self) -> LlamaConfigC:
        return LlamaConfigC(self.vocab_size, self.hidden_size, self.intermediate_size, self.num_hidden_layers,
                            self.num_attention_heads, self.num_key_value_heads, self.rms_norm_eps, self.max_seq_len,
                            self.rope_theta, self.head_dim, int(self.qk_norm), BF16 if self.weight_dtype == "bf16" else F32)

    @property
    def resolved_head_dim(self) -> int:
        return self.head_dim or self.hidden_size // self.num_attention_heads

    def param_shapes(self) -> dict:
        """Names and full shapes of `LlamaModel::named_parameters` (llama.rs:218-279)."""
        from .synth import param_shapes
        return param_shapes(self)


def tp_param_slice(config: "LlamaConfig", tp_rank: int, tp_size: int, name: str) -> dict:
    """The part of parameter `name` that rank `tp_rank` of `tp_size` keeps (`lumen_tp_param_slice`; host
    arithmetic, needs no GPU).  Returns full shape and the kept row / column ranges."""
    from ._lib import check, load
    out = (C.c_size_t * 6)()
    cfg_c = config.to_c()
    check(load().lumen_tp_param_slice(C.byref(cfg_c), tp_rank, tp_size, name.encode(), out))
    rows, cols, r0, nr, c0, nc = (int(v) for v in out)
    return {"shape": (rows,) if cols == 0 else (rows, cols), "rows": (r0, r0 + nr), "cols": (c0, c0 + nc)}


class LlamaModel(LanguageModel):
    """src/models/llama.rs:129-216.  Parameters start unset; fill them with `set_param` /
    `load_state` (the reference's random Kaiming init is not reproduced)."""

    _api = "lumen_llama_"

    def _new(self) -> None:
        cfg_c = self.config.to_c()
        self.ctx.check(self.ctx._lib.lumen_llama_new(self.ctx.h, C.byref(cfg_c), C.byref(self.h)))

    def _cache_shape(self, layer: int, batch: int) -> tuple:
        tp, hkv = self.ctx.tp_size, self.config.num_key_value_heads
        return batch, hkv // tp if hkv % tp == 0 else 1, self.config.max_seq_len, self.config.resolved_head_dim

    def _pos(self, pos: int) -> tuple:
        return (pos,)

    def decode_trace(self) -> np.ndarray:
        """Device trace of the last persistent decode step (needs LUMEN_DECODE_TRACE=1 when the model is
        created).  With nph = 5 * layers + 1 phases (qkv, attention, o, gate/up, down per layer, then lm_head):
        `stamps` [nph, 3] ns at phase start / after its prologue / after its last tile, `end` ns,
        `producer` [nph] ns of the phase's first copy, `input_ready` [nph] ns, `wait_cycles` and
        `busy_cycles` [nph] of consumer warp 0 on weight tiles, `tile_issue` and `tile_release` [512] ns;
        `cta_input` and `cta_done` [nph, 160] ns per CTA (0 where a CTA has no part in the phase)."""
        nph = 5 * self.config.num_hidden_layers + 1
        base = 7 * nph + 1 + 1024
        n = base + 2 * nph * 160
        buf = (C.c_uint64 * n)()
        got = C.c_size_t()
        self.ctx.check(self.ctx._lib.lumen_llama_decode_trace(self.h, buf, n, C.byref(got)))
        a = np.frombuffer(buf, dtype=np.uint64, count=got.value).astype(np.int64)
        return {"stamps": a[:3 * nph].reshape(nph, 3), "end": int(a[3 * nph]),
                "producer": a[3 * nph + 1:4 * nph + 1], "input_ready": a[4 * nph + 1:5 * nph + 1],
                "wait_cycles": a[5 * nph + 1:6 * nph + 1], "busy_cycles": a[6 * nph + 1:7 * nph + 1],
                "tile_issue": a[7 * nph + 1:7 * nph + 513], "tile_release": a[7 * nph + 513:base],
                "cta_input": a[base:base + nph * 160].reshape(nph, 160),
                "cta_done": a[base + nph * 160:base + 2 * nph * 160].reshape(nph, 160)}
