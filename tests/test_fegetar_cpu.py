"""Fegetar without a GPU: configuration reader, registry, parameter names, trace replay's bookkeeping, and the plain
implementation's own consistency."""
import json

import numpy as np
import pytest

import fegetar_cases as F
import fegetar_plain as plain


def _cfg():
    return F.config([(F.mixer(), F.dense()), (F.mixer(heads=2, rot_dims=4), F.moe()), (F.mixer(kv_rank=40), None)])


def test_config_reader_takes_every_size(L):
    cfg = L.FegetarConfig.from_dict(_cfg(), 77, "bf16")
    c = cfg.to_c()
    assert (c.vocab_size, c.width, c.num_layers, c.max_seq_len, c.side_dim, c.weight_dtype) == (101, 64, 3, 77, 16, L.BF16)
    assert (c.bigram_buckets, c.bigram_mul_prev, c.bigram_mul_cur) == (37, 5, 3)
    a, b, n = c.layers[0], c.layers[1], c.layers[2]
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.rot_dims, a.rot_base, a.mlp_kind, a.ff) == (3, 24, 8, 40, 48, 8, 500.0, 1, 88)
    assert a.scale == pytest.approx(0.1)
    assert (b.heads, b.rot_dims, b.mlp_kind, b.experts, b.top, b.expert_ff, b.shared_ff) == (2, 4, 2, 6, 2, 40, 56)
    assert (b.expert_limit, b.shared_limit) == (1.5, pytest.approx(0.8))
    assert n.mlp_kind == 0 and n.kv_rank == 40


def test_parameter_names_and_shapes(L):
    s = L.FegetarConfig.from_dict(_cfg(), 8, "f32").param_shapes()
    assert s["l0.mix.q"] == (3 * 32, 64) and s["l0.mix.dkv"] == (56, 64) and s["l0.mix.o"] == (64, 120)
    assert s["bigram"] == (38, 64) and s["side.embed"] == (101, 48) and s["l1.mlp.e5.down"] == (64, 40)
    assert s["l1.mlp.shared.gate"] == (56, 64) and "l2.norm2" not in s and "l2.side.proj" in s
    bare = L.FegetarConfig.from_dict(F.config([(F.mixer(), F.moe(shared=None))], bigram=None, side=None), 8, "f32").param_shapes()
    assert not [k for k in bare if "shared" in k or "side" in k or k == "bigram"]


def test_registry_picks_the_model_by_config(L):
    cfg, cls = L.model_config(_cfg(), 32, "f32")
    assert cls is L.FegetarModel and cfg.max_seq_len == 32
    hf = dict(architectures=["Qwen3ForCausalLM"], vocab_size=50, hidden_size=32, intermediate_size=48, num_hidden_layers=2,
              num_attention_heads=4, num_key_value_heads=2, head_dim=16, rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=64)
    cfg, cls = L.model_config(hf)
    assert cls is L.LlamaModel and cfg.qk_norm and cfg.head_dim == 16 and cfg.max_seq_len == 64 and cfg.weight_dtype == "bf16"
    with pytest.raises(ValueError):
        L.model_config(dict(architecture="Nobody"))
    with pytest.raises(ValueError):
        bad = _cfg()
        bad["layers"][0]["type"] = "something_else"
        L.model_config(bad)


def test_plain_implementation_sees_every_planted_mistake(L):
    """The tests compare with the plain implementation; each of these mistakes moves its logits far beyond their tolerances."""
    cfg = _cfg()
    p = F.weights(L, cfg, 3)
    ids = np.random.default_rng(4).integers(0, 101, 12)
    want = plain.forward(ids, cfg, p)
    for mistake in ("bigram", "first row", "interleaving", "position", "latent norm", "gate", "weighted input", "shared", "side", "gain around one"):
        assert F.row_err(plain.forward(ids, cfg, p, without=mistake), want).max() > 0.1, mistake


def test_plain_implementation_is_causal(L):
    cfg = _cfg()
    p = F.weights(L, cfg, 5)
    ids = np.random.default_rng(6).integers(0, 101, 9)
    assert np.allclose(plain.forward(ids, cfg, p)[:5], plain.forward(ids[:5], cfg, p))


class _FakeModel:
    """Records the calls of the replay; logits of a token are its value."""

    def __init__(self):
        self.made = self.resets = 0

    def init_kv_caches(self, b):
        self.made += 1
        return [self.made]

    def reset_kv_caches(self, caches):
        self.resets += 1

    def forward(self, ids, caches, last_only=False):
        lg = np.repeat(ids[..., None], 3, axis=-1).astype(np.float32)
        return lg[:, -1] if last_only else lg


def test_trace_replay_keeps_and_reuses_caches():
    from lumen_b200.replay import TraceReplay
    m = _FakeModel()
    r = TraceReplay(m)
    assert r.entry("a", [5, 6, 7], [0, 2]).tolist() == [[5] * 3, [7] * 3]
    assert r.entry("a", [8], []).shape == (0, 3)
    assert r.entry("b", [9, 4], [1]).tolist() == [[4] * 3]
    assert m.made == 2
    r.end("a")
    r.end("unknown")
    r.entry("c", [1], [0])
    assert m.made == 2 and m.resets == 1 and r.live["c"] == [1]


def test_header_constants_match_the_host_side(L):
    from pathlib import Path
    text = (Path(L.__file__).parents[1] / "include" / "lumen_b200.h").read_text()
    for name, v in (("NONE", L._lib.MLP_NONE), ("DENSE", L._lib.MLP_DENSE), ("MOE", L._lib.MLP_MOE)):
        assert f"#define LUMEN_MLP_{name} {v}\n" in text


def test_loader_takes_a_checkpoint_folder_layout(L, tmp_path):
    """config.json and the safetensors names agree (the upload itself needs a GPU)."""
    from lumen_b200.loader import SafeTensorsFile, save_safetensors
    from lumen_b200.synth import f32_to_bf16_bits
    cfg = _cfg()
    p = F.weights(L, cfg, 1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tmp_path / "model.safetensors", {k: f32_to_bf16_bits(v).reshape(v.shape) for k, v in p.items()})
    got, cls = L.model_config(json.loads((tmp_path / "config.json").read_text()), 16)
    with SafeTensorsFile(tmp_path / "model.safetensors") as f:
        shapes = got.param_shapes()
        assert set(f.names()) == set(shapes)
        assert all(f.tensor(n)[1] == tuple(s) for n, s in shapes.items())
