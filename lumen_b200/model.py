"""What the host side of every language model shares: parameters by name, caches, forward, sampling."""
from __future__ import annotations

import ctypes as C
import weakref

import numpy as np

from . import _lib
from ._lib import BF16, F32
from .layers import KVCacheInner
from .tensor import Context, default_context, require_no_grad


class _ParamRef:
    """What `named_parameters()` hands to a loader: `set_raw_data` uploads into the model's slab."""

    def __init__(self, model: "LanguageModel", name: str, shape: tuple):
        self.model, self.name, self.shape = model, name, shape

    def set_raw_data(self, shape, raw_data) -> None:
        self.model.set_param(self.name, np.asarray(raw_data, dtype=np.float32).reshape(shape))


class LanguageModel:
    """A model behind the C ABI.  Subclasses create the handle (`_new`), name its entry points (`_api` + operation) and give
    the caches' geometry.  `config` has `vocab_size`, `num_hidden_layers`, `max_seq_len` and `param_shapes()`."""

    _api = "lumen_model_"

    def __init__(self, config, ctx: Context | None = None):
        self.ctx = ctx or default_context()
        self.config = config
        self.h = C.c_void_p()
        self._new()
        self._finalizer = weakref.finalize(self, self._fn("free"), C.c_void_p(self.h.value))
        self._shapes = config.param_shapes()

    def _new(self) -> None:
        raise NotImplementedError

    def _cache_shape(self, layer: int, batch: int) -> tuple:
        raise NotImplementedError

    def _fn(self, op: str):
        return getattr(self.ctx._lib, self._api + op)

    def _pos(self, pos: int) -> tuple:
        """Further arguments of the forward entry points between the caches and the logits."""
        return ()

    # ---- parameters ---------------------------------------------------------------------------------
    def named_parameters(self) -> dict:
        return {n: _ParamRef(self, n, s) for n, s in self._shapes.items()}

    def set_param(self, name: str, value: np.ndarray, as_bf16_bits: bool = False) -> None:
        """Upload one full (unsharded) tensor by its checkpoint name.  `value` is f32, or uint16
        bf16 bit patterns when `as_bf16_bits`."""
        if as_bf16_bits:
            a = np.ascontiguousarray(value, dtype=np.uint16)
            dt = BF16
        else:
            a = np.ascontiguousarray(value, dtype=np.float32)
            dt = F32
        shape = (C.c_size_t * a.ndim)(*a.shape)
        self.ctx.check(self._fn("set_param")(self.h, name.encode(), a.ctypes.data, shape, a.ndim, dt))

    def load_state(self, params: dict) -> None:
        for name, value in params.items():
            self.set_param(name, value)

    @property
    def weight_bytes_per_step(self) -> int:
        return int(self._fn("weight_bytes")(self.h))

    # ---- caches (llama.rs:161-176) ----------------------------------------------------------------------
    def init_kv_caches(self, batch_size: int) -> list:
        n = self.config.num_hidden_layers
        arr = (C.c_void_p * max(n, 1))()
        self.ctx.check(self._fn("init_kv_caches")(self.h, batch_size, arr))
        return [KVCacheInner(*self._cache_shape(i, batch_size), self.ctx, _handle=C.c_void_p(arr[i])) for i in range(n)]

    def reset_kv_caches(self, caches: list) -> None:
        for c in caches:
            c.reset()

    def _cache_array(self, caches):
        return (C.c_void_p * max(len(caches), 1))(*[c.h for c in caches])

    # ---- forward (llama.rs:181-206) -----------------------------------------------------------------------
    def forward(self, input_ids, caches: list, _pos: int = 0, last_only: bool = False) -> np.ndarray:
        """input_ids[B,S] (token ids, passed as f32 like the reference) -> logits [B,S,V] on the host.
        `last_only` returns [B,V] for the final position only."""
        require_no_grad(f"{type(self).__name__}::forward")
        ids = np.ascontiguousarray(input_ids, dtype=np.float32)
        if ids.ndim != 2:
            raise _lib.LumenError(_lib.ERR_SHAPE, "input_ids must be [B,S]")
        b, s = ids.shape
        v = self.config.vocab_size
        logits = np.empty((b, v) if last_only else (b, s, v), dtype=np.float32)
        fn = self._fn("forward_last" if last_only else "forward")
        self.ctx.check(fn(self.h, ids.ctypes.data, b, s, self._cache_array(caches), len(caches), *self._pos(_pos), logits.ctypes.data))
        return logits

    def forward_sample(self, input_ids, caches: list, temperature: float, top_p: float, repetition_penalty: float,
                       recent_tokens, uniform: float) -> int:
        """`forward` on ids [1,S] followed by `sample_top_p` (src/main.rs:74-137) on the device; returns the
        sampled token id.  `uniform` is the draw in [0,1) the reference takes from its RNG."""
        require_no_grad(f"{type(self).__name__}::forward")
        from ._lib import SampleParamsC
        ids = np.ascontiguousarray(input_ids, dtype=np.float32).reshape(-1)
        rec = np.ascontiguousarray(recent_tokens, dtype=np.int32)
        sp = SampleParamsC(temperature, top_p, repetition_penalty, rec.ctypes.data_as(C.POINTER(C.c_int32)), rec.size, uniform)
        tok = C.c_int32()
        self.ctx.check(self._fn("forward_sample")(self.h, ids.ctypes.data, ids.size, self._cache_array(caches),
                                                                len(caches), C.byref(sp), C.byref(tok)))
        return int(tok.value)

    def forward_device(self, ids_ptr: int, b: int, s: int, caches: list, logits_ptr: int) -> None:
        """Same step with device-resident ids and logits, asynchronous on the context's stream."""
        require_no_grad(f"{type(self).__name__}::forward")
        self.ctx.check(self._fn("forward_device")(self.h, ids_ptr, b, s, self._cache_array(caches),
                                                                len(caches), logits_ptr))


class DecoderModel(LanguageModel):
    """A model given as a list of layers (`config.to_c()` is a `lumen_decoder_config`).  Parameters start unset; fill them with
    `set_param` / `load_state` / the loader, under their checkpoint names."""

    def _new(self) -> None:
        cfg_c = self.config.to_c()
        self.ctx.check(self.ctx._lib.lumen_decoder_new(self.ctx.h, C.byref(cfg_c), C.byref(self.h)))
