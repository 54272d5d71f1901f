"""Model registry: config.json -> configuration and model class, and a loaded model from a checkpoint folder.

An entry maps the name a config.json carries (`architecture`, or the first of Hugging Face's `architectures`) to a
function (config dict, max_seq_len, weight_dtype) -> configuration, and to the model class.
"""
from __future__ import annotations

import json
from pathlib import Path

from .fegetar import FegetarConfig, FegetarModel
from .fekorax import FekoraxConfig, FekoraxModel
from .llama import LlamaConfig, LlamaModel
from .loader import load_weights


def _llama_config(d: dict, max_seq_len: int | None, weight_dtype: str, qk_norm: bool = False) -> LlamaConfig:
    heads = int(d["num_attention_heads"])
    return LlamaConfig(
        vocab_size=int(d["vocab_size"]), hidden_size=int(d["hidden_size"]), intermediate_size=int(d["intermediate_size"]),
        num_hidden_layers=int(d["num_hidden_layers"]), num_attention_heads=heads,
        num_key_value_heads=int(d.get("num_key_value_heads") or heads), rms_norm_eps=float(d.get("rms_norm_eps", 1e-5)),
        max_seq_len=int(max_seq_len or d.get("max_position_embeddings", 2048)), rope_theta=float(d.get("rope_theta", 10000.0)),
        head_dim=int(d.get("head_dim") or 0), qk_norm=qk_norm, weight_dtype=weight_dtype)


MODELS = {
    "LlamaForCausalLM": (_llama_config, LlamaModel),
    "Qwen3ForCausalLM": (lambda d, n, dt: _llama_config(d, n, dt, qk_norm=True), LlamaModel),
    "Fegetar": (lambda d, n, dt: FegetarConfig.from_dict(d, int(n or 2048), dt), FegetarModel),
    "Fekorax": (lambda d, n, dt: FekoraxConfig.from_dict(d, int(n or 2048), dt), FekoraxModel),
}


def architecture_of(config: dict) -> str:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in MODELS:
        raise ValueError(f"no model for architecture {name!r} (known: {', '.join(sorted(MODELS))})")
    return name


def model_config(config: dict, max_seq_len: int | None = None, weight_dtype: str = "bf16"):
    """(configuration, model class) for a parsed config.json."""
    make, cls = MODELS[architecture_of(config)]
    return make(config, max_seq_len, weight_dtype), cls


def load_model(folder, max_seq_len: int | None = None, weight_dtype: str = "bf16", ctx=None):
    """The model of a folder with config.json and model.safetensors."""
    folder = Path(folder)
    cfg, cls = model_config(json.loads((folder / "config.json").read_text()), max_seq_len, weight_dtype)
    model = cls(cfg, ctx)
    missing = load_weights(folder / "model.safetensors", model)
    if missing:
        raise ValueError(f"{folder}: {len(missing)} parameters are missing, the first is {missing[0]}")
    return model
