"""Fekorax without a GPU: configuration reader, registry, parameter names, and the plain implementation's own consistency."""
import json
from pathlib import Path

import numpy as np
import pytest

import fekorax_cases as K
import fekorax_plain as plain


def _cfg(**kw):
    return K.config([(K.matrix(), None), (K.attn(), 88), (K.attn(chunk=30, scale=0.4), None), (K.matrix(heads=2, dim=16, vdim=8, gate_cap=4.0), 40),
                     (K.attn(chunk=17, scale=0.3, kv_from=1), 56)], **kw)


def test_config_reader_takes_every_size(L):
    cfg = L.FekoraxConfig.from_dict(_cfg(), 77, "bf16")
    c = cfg.to_c()
    assert (c.vocab_size, c.width, c.num_layers, c.max_seq_len, c.weight_dtype, c.tied_head, c.norms) == (101, 64, 5, 77, L.BF16, 1, L._lib.NORM_BOTH)
    assert c.embed_scale == 3.0 and c.norm_eps == pytest.approx(1e-4)
    a, b, n, s = c.layers[0], c.layers[1], c.layers[3], c.layers[4]
    assert (a.mixer, a.heads, a.dim, a.vdim, a.mlp_kind) == (L._lib.MIXER_MLSTM, 3, 24, 40, L._lib.MLP_NONE) and a.gate_cap == 9.0
    assert (b.mixer, b.heads, b.kv_heads, b.dim, b.vdim, b.chunk, b.rot_dims, b.kv_from, b.mlp_kind, b.ff) == (L._lib.MIXER_ATTENTION, 4, 2, 32, 24, 48, 20, -1, L._lib.MLP_GATED_GELU, 88)
    assert (b.rot_base, b.rot_factor, b.rot_low, b.rot_high, b.rot_original) == (700.0, 3.0, 1.5, 5.0, 300.0) and b.scale == pytest.approx(0.21)
    assert (n.gate_cap, n.ff, n.mlp_kind) == (4.0, 40, L._lib.MLP_GATED_GELU)
    assert (s.kv_from, s.chunk) == (1, 17)
    bare = L.FekoraxConfig.from_dict(K.config([(K.attn(scaling=None), None)]), 8, "f32").to_c().layers[0]
    assert bare.rot_factor == 0.0


def test_parameter_names_and_shapes(L):
    s = L.FekoraxConfig.from_dict(_cfg(), 8, "f32").param_shapes()
    assert s["l0.mix.q"] == (72, 64) and s["l0.mix.g"] == (120, 64) and s["l0.mix.norm"] == (120,) and s["l0.mix.f.b"] == (3,)
    assert s["l1.mix.k"] == (64, 64) and s["l1.mix.v"] == (48, 64) and s["l1.mix.k.norm"] == (32,) and s["l1.mix.sink"] == (4,)
    assert "l4.mix.k" not in s and "l4.mix.v" not in s and "l4.mix.k.norm" not in s and s["l4.mix.q.norm"] == (32,)
    assert "l0.norm2" not in s and s["l1.norm2b"] == (64,) and s["l1.mlp.down"] == (64, 88) and "head" not in s


def test_registry_picks_the_model_by_config(L):
    cfg, cls = L.model_config(_cfg(), 32, "f32")
    assert cls is L.FekoraxModel and cfg.max_seq_len == 32
    for change in (dict(type="something_else"), dict(mlp=dict(kind="routed"))):
        bad = _cfg()
        bad["layers"][0].update(change)
        with pytest.raises(ValueError):
            L.model_config(bad)


MISTAKES = ("gate bias", "gate cap", "log of the forget gate", "query scale", "decay", "normaliser", "floor", "head norm", "output gate",
            "frequency scaling", "rotate half", "position", "chunks", "key norm", "query norm", "score scale", "grouping", "sink", "sink as it is",
            "head gate", "whose keys", "which is gated", "embedding scale", "norm before", "norm after", "one key more", "one key less")


def test_plain_implementation_sees_every_planted_mistake(L):
    """The tests compare with the plain implementation; each of these mistakes moves its logits.  (A head's norm takes out the
    size of the matrix memory's output, so its denominator shows against a large eps only.)"""
    cfg = _cfg(eps=0.1)
    p = K.weights(L, cfg, 3)
    for name in p:
        if name.endswith((".i", ".f")):
            p[name] = p[name] * 4
    ids = np.random.default_rng(4).integers(0, 101, 80)
    want = plain.forward(ids, cfg, p)
    for mistake in MISTAKES:
        assert K.row_err(plain.forward(ids, cfg, p, without=mistake), want).max() > 0.1, mistake
    assert K.row_err(plain.forward(ids, cfg, p, forget_at=20), want)[20:].max() > 0.1


def test_plain_implementation_is_causal(L):
    cfg = _cfg()
    p = K.weights(L, cfg, 5)
    ids = np.random.default_rng(6).integers(0, 101, 60)
    assert np.allclose(plain.forward(ids, cfg, p)[:35], plain.forward(ids[:35], cfg, p))


def test_chunked_form_of_the_matrix_memory():
    """The sums that the tensor-core kernels form per chunk (a, M, the weights, S and n at chunk starts) equal the recurrence."""
    rng = np.random.default_rng(7)
    T, C, d, v = 75, 16, 6, 5
    q, k, val = rng.standard_normal((T, d)), rng.standard_normal((T, d)), rng.standard_normal((T, v))
    i, f = 3 * rng.standard_normal(T), -np.logaddexp(0, -3 * rng.standard_normal(T))
    S, n, m, want = np.zeros((d, v)), np.zeros(d), 0.0, []
    for t in range(T):
        new = max(f[t] + m, i[t])
        S, n, m = np.exp(f[t] + m - new) * S + np.exp(i[t] - new) * np.outer(k[t], val[t]), np.exp(f[t] + m - new) * n + np.exp(i[t] - new) * k[t], new
        want.append(np.concatenate([S.T @ q[t], [n @ q[t], m]]))
    S0, n0, m0, got = np.zeros((d, v)), np.zeros(d), 0.0, []
    for c in range(0, T, C):
        s = slice(c, min(c + C, T))
        F = np.cumsum(f[s])
        a = i[s] - F
        M = np.maximum(m0, np.maximum.accumulate(a))
        w = np.tril(np.exp(np.minimum(a[None] - M[:, None], 0))) * (q[s] @ k[s].T)
        g = np.exp(m0 - M)[:, None]
        got.append(np.concatenate([w @ val[s] + g * (q[s] @ S0), (w.sum(1) + g[:, 0] * (q[s] @ n0))[:, None], (F + M)[:, None]], axis=1))
        end = np.exp(a - M[-1])
        S0, n0, m0 = np.exp(m0 - M[-1]) * S0 + (end[:, None] * k[s]).T @ val[s], np.exp(m0 - M[-1]) * n0 + end @ k[s], F[-1] + M[-1]
    assert np.allclose(np.concatenate(got), np.array(want))


def test_header_constants_match_the_host_side(L):
    text = (Path(L.__file__).parents[1] / "include" / "lumen_b200.h").read_text()
    lib = L._lib
    for name, v in (("MIXER_LATENT", lib.MIXER_LATENT), ("MIXER_ATTENTION", lib.MIXER_ATTENTION), ("MIXER_MLSTM", lib.MIXER_MLSTM),
                    ("NORM_OUTPUT", lib.NORM_OUTPUT), ("NORM_BOTH", lib.NORM_BOTH), ("MLP_GATED_GELU", lib.MLP_GATED_GELU)):
        assert f"#define LUMEN_{name} {v}\n" in text


def test_loader_takes_a_checkpoint_folder_layout(L, tmp_path):
    """config.json and the safetensors names agree (the upload itself needs a GPU)."""
    from lumen_b200.loader import SafeTensorsFile, save_safetensors
    from lumen_b200.synth import f32_to_bf16_bits
    cfg = _cfg()
    p = K.weights(L, cfg, 1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tmp_path / "model.safetensors", {k: f32_to_bf16_bits(v).reshape(v.shape) for k, v in p.items()})
    got, _ = L.model_config(json.loads((tmp_path / "config.json").read_text()), 16)
    with SafeTensorsFile(tmp_path / "model.safetensors") as f:
        shapes = got.param_shapes()
        assert set(f.names()) == set(shapes)
        assert all(f.tensor(n)[1] == tuple(s) for n, s in shapes.items())
