"""Fegetar on the GPU against the plain implementation (fegetar_plain.py): each mechanism alone, portions of a prompt, decoding,
caches that are used again, far keys and tile borders, and the framework's own entry points.

A mechanism is isolated by weights: an output projection of zeros silences a sublayer (the norm of zeros is zero)."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import fegetar_cases as F
import fegetar_plain as plain

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
# Tolerances (F.tolerance) are three times the error that rounding alone causes at the worst position; these are their bounds.
CAP = {"f32": 1e-4, "bf16": 8e-2}
DTYPES = ("f32", "bf16")


def _ids(n, seed=0, vocab=101):
    return np.random.default_rng(seed).integers(0, vocab, n)


def _silence(p, *parts):
    return {k: np.zeros_like(v) if k.endswith(parts) else v for k, v in p.items()}


def _check(L, cfg, p, ids, cuts_list, dtype, rows=None, max_seq=None, mistakes=()):
    want = plain.forward(ids, cfg, p)
    model = F.build(L, cfg, p, dtype, max_seq or max(len(ids), 16))
    rows = np.ones(len(ids), bool) if rows is None else rows
    tol = F.tolerance(ids, cfg, p, dtype, want, rows)
    assert tol < CAP[dtype], tol
    for cuts in cuts_list:
        err = F.row_err(F.run(L, model, ids, cuts), want)[rows]
        assert err.max() < tol, (cuts, int(err.argmax()), float(err.max()), tol)
    for m in mistakes:  # the mistake would have shown
        assert F.row_err(plain.forward(ids, cfg, p, without=m), want)[rows].max() > 1.5 * tol, m
    return model


def _close(ids, got, cfg, p, dtype):
    """got: logits of the whole sequence."""
    want = plain.forward(ids, cfg, p)
    tol = F.tolerance(ids, cfg, p, dtype, want)
    err = F.row_err(got, want)
    assert tol < CAP[dtype] and err.max() < tol, (int(err.argmax()), float(err.max()), tol)


# ---- one mechanism at a time ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bigram", [(37, 5, 3), (1, 1, 1), (509, 1000003, 999983), None])
def test_embedding_and_bigram(L, dtype, bigram):
    cfg = F.config([(F.mixer(), None)], bigram=bigram, side=None)
    p = _silence(F.weights(L, cfg, 1), "mix.o")
    _check(L, cfg, p, _ids(23), ([23], [1], [2], [5, 1, 1, 3]), dtype,
           mistakes=("bigram", "first row") if bigram and bigram[0] > 1 else ())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [
    F.mixer(), F.mixer(heads=1, dim=16, rot_dim=4, vdim=16, kv_rank=16), F.mixer(heads=5, dim=20, rot_dim=12, vdim=36, kv_rank=100),
    F.mixer(heads=2, dim=64, rot_dim=64, vdim=64, kv_rank=64), F.mixer(heads=4, dim=72, rot_dim=16, vdim=128, kv_rank=192),
    F.mixer(heads=17, dim=16, rot_dim=8, vdim=16, kv_rank=256), F.mixer(heads=2, dim=32, rot_dim=32, vdim=24, kv_rank=512),
    F.mixer(heads=2, dim=96, rot_dim=16, vdim=136, kv_rank=520), F.mixer(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=56, rot_dims=6, base=20.0),
    F.mixer(heads=2, dim=128, rot_dim=80, vdim=72, kv_rank=120), F.mixer(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=9),
])
def test_latent_attention_alone(L, dtype, m):
    """Sizes for every kernel: tensor-core prefill (with 2 and 3 key blocks, 64 and 128 values), tensor-core decode of every
    width, and the general one."""
    cfg = F.config([(m, None)], bigram=None, side=None)
    _check(L, cfg, F.weights(L, cfg, 2), _ids(140, 2), ([140], [100, 1], [75, 65], [70, 2, 30, 3]), dtype,
           mistakes=("interleaving", "position", "latent norm", "gate"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 88), (64, 1), (72, 300), (36, 50), (328, 96)])
def test_dense_alone(L, dtype, width, ff):
    cfg = F.config([(F.mixer(), F.dense(ff))], width=width, bigram=None, side=None)
    p = _silence(F.weights(L, cfg, 3), "mix.o")
    _check(L, cfg, p, _ids(150, 3), ([150], [1], [9], [131, 2]), dtype, mistakes=("gain around one",))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,mlp", [
    (64, F.moe()), (64, F.moe(top=1)), (64, F.moe(experts=3, top=3, shared=None)), (64, F.moe(experts=40, top=6, ff=72, limit=0.3, shared=(136, 2.5))),
    (64, F.moe(experts=1, top=1, ff=8)), (72, F.moe(experts=5, top=2, ff=20, limit=7.0, shared=(12, 0.5))), (36, F.moe(experts=9, top=4, ff=33)),
    (136, F.moe(experts=70, top=8, ff=64, shared=(64, 1.0))),
])
def test_experts_alone(L, dtype, width, mlp):
    cfg = F.config([(F.mixer(), mlp)], width=width, bigram=None, side=None)
    p = _silence(F.weights(L, cfg, 4), "mix.o")
    ids = _ids(150, 4)
    # rows whose choice hangs on a rounding of the scores are left out
    x = p["embed"][ids].astype(np.float64)
    sc = -np.sort(-plain.router_scores(x, {k: v.astype(np.float64) for k, v in p.items() if "router" in k}, "l0.mlp."), axis=1)
    top = mlp["router"]["top"]
    rows = np.ones(len(ids), bool) if top == sc.shape[1] else sc[:, top - 1] - sc[:, top] > 1e-3
    assert rows.mean() > 0.8
    _check(L, cfg, p, ids, ([150], [1], [7], [131, 2]), dtype, rows=rows,
           mistakes=("weighted input",) + (("shared",) if mlp.get("shared") else ()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", [1, 16, 20, 264])
def test_side_input_alone(L, dtype, side):
    cfg = F.config([(F.mixer(), None)] * 3, bigram=None, side=side)
    p = _silence(F.weights(L, cfg, 5), "mix.o")
    _check(L, cfg, p, _ids(140, 5), ([140], [1], [3], [133, 2]), dtype, mistakes=("side",))


# ---- the whole model -------------------------------------------------------------------------------------
def _mixed(top=2, **kw):
    return F.config([(F.mixer(), F.dense()), (F.mixer(heads=2, dim=40, rot_dim=16, vdim=24, kv_rank=80, base=1e4), F.moe(top=top)),
                     (F.mixer(kv_rank=40, rot_dims=4), None), (F.mixer(), F.moe(experts=top + 1, top=top + 1, shared=None)),
                     (F.mixer(heads=4), F.dense(56))], **kw)


@pytest.mark.parametrize("cuts", [[190], [1], [2], [3, 2], [64], [65, 1], [63, 64, 1], [128, 2, 2, 1], [17, 100, 2], [189, 1]])
def test_portions_f32(L, cuts):
    cfg = _mixed()
    _check(L, cfg, F.weights(L, cfg, 6), _ids(190, 6), (cuts,), "f32")


@pytest.mark.parametrize("cuts", [[190], [1], [2], [64], [65, 1], [63, 64, 1], [128, 2, 2, 1], [17, 100, 2]])
def test_portions_bf16(L, cuts):
    """Every expert is chosen here (a choice on the edge would turn a rounding into another expert)."""
    cfg = F.config([(F.mixer(), F.dense()), (F.mixer(heads=2, dim=40, rot_dim=16, vdim=24, kv_rank=80, base=1e4), F.moe(experts=4, top=4)),
                    (F.mixer(kv_rank=40, rot_dims=4), None)])
    _check(L, cfg, F.weights(L, cfg, 8), _ids(190, 8), (cuts,), "bf16")


def test_long_decoding(L):
    cfg = _mixed()
    p, ids = F.weights(L, cfg, 8), _ids(420, 8)
    _check(L, cfg, p, ids, ([20, 1],), "f32")
    cfg = F.config([(F.mixer(heads=7, kv_rank=112), F.dense())])
    _check(L, cfg, F.weights(L, cfg, 8), ids, ([20, 1],), "bf16")


@pytest.mark.parametrize("dtype", DTYPES)
def test_equal_sequences_in_a_batch_match_each_alone(L, dtype):
    cfg = F.config([(F.mixer(), F.dense()), (F.mixer(heads=2), F.moe(experts=4, top=4))])
    p = F.weights(L, cfg, 9)
    model = F.build(L, cfg, p, dtype, 120)
    ids = _ids(3 * 100, 9).reshape(3, 100)
    caches = model.init_kv_caches(3)
    got = []
    with L.no_grad():
        at = 0
        for n in [70, 2, 1, 1, 1, 20, 1, 4]:
            got.append(model.forward(ids[:, at:at + n].astype(np.float32), caches))
            at += n
    got = np.concatenate(got, axis=1)
    for b in range(3):
        _close(ids[b], got[b], cfg, p, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_caches_reset_and_used_again(L, dtype):
    """A long sequence, then a short one in the same caches: nothing of the first (rows, last token) is seen."""
    cfg = F.config([(F.mixer(), F.dense()), (F.mixer(heads=2), None)])
    p = F.weights(L, cfg, 10)
    model = F.build(L, cfg, p, dtype, 150)
    caches = model.init_kv_caches(1)
    for seed, n, cuts in ((1, 150, [150]), (2, 9, [1]), (3, 80, [70, 1]), (4, 2, [2]), (5, 1, [1])):
        model.reset_kv_caches(caches)
        ids = _ids(n, seed)
        _close(ids, F.run(L, model, ids, cuts, caches), cfg, p, dtype)


def test_interleaved_requests_and_freed_caches(L):
    """Requests take turns, step by step; caches of finished ones serve new ones."""
    from lumen_b200.replay import TraceReplay
    cfg = _mixed()
    p = F.weights(L, cfg, 11)
    replay = TraceReplay(F.build(L, cfg, p, "f32", 100))
    ids = {r: _ids(n, i) for i, (r, n) in enumerate([("a", 90), ("b", 41), ("c", 70), ("d", 5)])}
    at, got = {r: 0 for r in ids}, {r: [] for r in ids}
    rng = np.random.default_rng(12)
    with L.no_grad():
        pending, waiting = ["a", "b"], ["c", "d"]
        while pending:
            r = pending[rng.integers(len(pending))]
            n = min(int(rng.choice([1, 1, 2, 3, 30])), len(ids[r]) - at[r])
            got[r].append(replay.entry(r, ids[r][at[r]:at[r] + n].tolist(), list(range(n))))
            at[r] += n
            if at[r] == len(ids[r]):
                replay.end(r)
                pending.remove(r)
                if waiting:
                    pending.append(waiting.pop(0))
    assert len(replay.free) == 2  # two sets of caches served four requests
    for r in ids:
        _close(ids[r], np.concatenate(got[r]), cfg, p, "f32")


# ---- far keys and tile borders -----------------------------------------------------------------------------
def _standing_out(L, m, seed=13):
    """One attention layer in which token 96 asks for token 95: its first head's unrotated query points at that token's key, so
    that one score stands out among hundreds."""
    cfg = F.config([(m, None)], bigram=None, side=None)
    p = F.weights(L, cfg, seed, round_bf16=False)
    eps, rank, d = cfg["norm"]["eps"], m["kv_rank"], m["dim"]
    p["embed"][95] *= 3
    c = plain.rms_norm((p["l0.mix.dkv"][:rank].astype(np.float64) @ p["embed"][95]), p["l0.mix.dkv.norm"], eps)
    key = p["l0.mix.uk"][:d].astype(np.float64) @ c
    want = key / np.linalg.norm(key) ** 2 * 14.0 / m["scale"]
    want = np.concatenate([want, np.zeros(m["rot_dim"])])  # and its rotated query is nothing
    p["embed"][96] = np.linalg.pinv(p["l0.mix.q"][:d + m["rot_dim"]].astype(np.float64)) @ want
    from lumen_b200.synth import bf16_bits_to_f32, f32_to_bf16_bits
    return cfg, {k: bf16_bits_to_f32(f32_to_bf16_bits(np.asarray(v, np.float32))).reshape(v.shape) for k, v in p.items()}


FAR = [(1, 0), (2, 1), (63, 0), (64, 0), (64, 63), (65, 63), (65, 64), (127, 63), (128, 0), (128, 64), (129, 127), (200, 65), (200, 128),
       (299, 0), (299, 1), (299, 191), (299, 192), (299, 298)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m", [F.mixer(heads=2, dim=32, rot_dim=24, vdim=40, kv_rank=72), F.mixer(heads=2, dim=28, rot_dim=8, vdim=40, kv_rank=60),
                               F.mixer(heads=1, dim=36, rot_dim=10, vdim=40, kv_rank=68)])
def test_far_keys_and_borders(L, dtype, m):
    cfg, p = _standing_out(L, m)
    model = F.build(L, cfg, p, dtype, 304)
    caches = model.init_kv_caches(1)
    for i, j in FAR:
        ids = _ids(i + 1, 100 + i + j, 90)
        ids[j], ids[i] = 95, 96
        want = plain.forward(ids, cfg, p)
        lost = plain.forward(ids, cfg, p, hidden_key=j)
        tol = F.tolerance(ids, cfg, p, dtype, want)
        assert tol < CAP[dtype], tol
        assert F.row_err(lost, want)[i] > 0.3, (i, j)  # without that key the last position would say something else
        for cuts in ([i + 1], [i, 1], [i - 1, 2] if i > 1 else [1], [37]):
            model.reset_kv_caches(caches)
            err = F.row_err(F.run(L, model, ids, cuts, caches), want)
            assert err.max() < tol, (i, j, cuts, int(err.argmax()), float(err.max()), tol)


# ---- errors, entry points ----------------------------------------------------------------------------------
def test_errors_come_back_as_status_codes(L):
    cfg = F.config([(F.mixer(), F.dense())])
    model = L.FegetarModel(L.FegetarConfig.from_dict(cfg, 16, "f32"))
    caches = model.init_kv_caches(1)
    with L.no_grad():
        with pytest.raises(L.LumenError) as e:
            model.forward(np.zeros((1, 1)), caches)
        assert e.value.code == L._lib.ERR_MISSING_PARAM
        p = F.weights(L, cfg, 1)
        model.load_state(p)
        for bad, code in ((dict(ids=np.full((1, 1), 101.0)), L._lib.ERR_EMBED_RANGE), (dict(ids=np.zeros((1, 17))), L._lib.ERR_KV_OVERFLOW),
                          (dict(ids=np.zeros((2, 1))), L._lib.ERR_SHAPE)):
            with pytest.raises(L.LumenError) as e:
                model.forward(bad["ids"], caches)
            assert e.value.code == code
        with pytest.raises(L.LumenError) as e:
            model.set_param("nobody", np.zeros(3))
        assert e.value.code == L._lib.ERR_PARAM_NAME
        with pytest.raises(L.LumenError) as e:
            model.set_param("l0.mix.q", np.zeros((3, 3)))
        assert e.value.code == L._lib.ERR_SHAPE
        two = model.init_kv_caches(1)
        llama = L.LlamaModel(L.LlamaConfig(vocab_size=11, hidden_size=64, intermediate_size=8, num_hidden_layers=1, num_attention_heads=1,
                                           num_key_value_heads=1, head_dim=64, max_seq_len=16))
        llama.load_state({n: np.zeros(s, np.float32) for n, s in llama.config.param_shapes().items()})
        with pytest.raises(L.LumenError):
            llama.forward(np.zeros((1, 1)), two)  # a latent cache is not a cache of keys and values
        ids = _ids(5)
        _close(ids, F.run(L, model, ids, [5], two), cfg, p, "f32")


def test_greedy_generation_through_the_chat_session(L):
    cfg = _mixed()
    p = F.weights(L, cfg, 15)
    prompt, n = _ids(21, 15).tolist(), 24
    seq = list(prompt)
    for _ in range(n):
        lg = plain.forward(seq, cfg, p)[-1]
        top = np.sort(lg)[-2:]
        assert top[1] - top[0] > 1e-3  # no close call
        seq.append(int(lg.argmax()))
    from lumen_b200.chat import ChatSession
    s = ChatSession(F.build(L, cfg, p, "f32", 160), lambda t: t, lambda t: t, temperature=0.0, top_p=1.0, repetition_penalty=1.0, max_gen=n)
    assert s.turn(prompt) == seq[len(prompt):]
    # a second turn continues in the kept caches
    more = _ids(6, 15).tolist()
    full = seq + more
    want = int(plain.forward(full, cfg, p)[-1].argmax())
    s.max_gen = 1
    assert s.turn(more) == [want]


def _checkpoint(L, tmp_path, cfg, p):
    from lumen_b200.loader import save_safetensors
    from lumen_b200.synth import f32_to_bf16_bits
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tmp_path / "model.safetensors", {k: f32_to_bf16_bits(v).reshape(v.shape) for k, v in p.items()})


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_and_command_line(L, tmp_path, dtype):
    cfg = F.config([(F.mixer(), F.dense()), (F.mixer(heads=2), F.moe(experts=4, top=4))])
    p = F.weights(L, cfg, 16)
    kind = "f32" if dtype == "float32" else "bf16"
    _checkpoint(L, tmp_path, cfg, p)
    ids = {"x": _ids(80, 1), "y": _ids(7, 2)}
    steps = [("x", 0, 70, [0, 69]), ("x", 70, 72, [1]), ("x", 72, 80, []), ("y", 0, 6, [2, 5]), ("y", 6, 7, [0])]
    lines = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": ids[r][a:b].tolist(), "want": w}],
                                "end": [r] if b == len(ids[r]) else []}) + "\n" for i, (r, a, b, w) in enumerate(steps))
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                       input=lines, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    assert not (out / "2.f32").exists()
    for i, (rid, a, b, w) in enumerate(steps):
        if w:
            got = np.fromfile(out / f"{i}.f32", "<f4").reshape(len(w), 101)
            want = plain.forward(ids[rid], cfg, p)
            full = want.copy()
            full[[a + k for k in w]] = got
            assert F.row_err(full, want).max() < F.tolerance(ids[rid], cfg, p, kind, want), i
    if dtype == "float32":
        seq = ids["y"].tolist()
        for _ in range(3):
            seq.append(int(plain.forward(seq, cfg, p)[-1].argmax()))
        env = dict(os.environ, PYTHONPATH=str(ROOT))
        r = subprocess.run([sys.executable, "-m", "lumen_b200", "generate", "--model", str(tmp_path), "--dtype", dtype, "--max-new", "3", "--ids",
                            " ".join(map(str, ids["y"]))], capture_output=True, text=True, timeout=600, env=env)
        assert r.returncode == 0 and [int(t) for t in r.stdout.split()] == seq[7:], r.stderr[-2000:]
