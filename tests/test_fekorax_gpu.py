"""Fekorax on the GPU against the plain implementation (fekorax_plain.py): each mechanism alone, portions of a prompt, decoding,
caches and states that are used again, far keys and chunk borders, and the framework's own entry points.

A mechanism is isolated by weights: an output projection of zeros silences a sublayer (the norm of zeros is zero)."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import fekorax_cases as K
import fekorax_plain as plain

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
# Tolerances (K.tolerance) are three times the error that rounding alone causes at the worst position; these are their bounds.
CAP = {"f32": 5e-4, "bf16": 2e-1}
DTYPES = ("f32", "bf16")


def _ids(n, seed=0, vocab=101):
    return np.random.default_rng(seed).integers(0, vocab, n)


def _silence(p, *parts):
    return {k: np.zeros_like(v) if k.endswith(parts) else v for k, v in p.items()}


def _check(L, cfg, p, ids, cuts_list, dtype, max_seq=None, mistakes=(), rows=None):
    want = plain.forward(ids, cfg, p)
    model = K.build(L, cfg, p, dtype, max_seq or max(len(ids), 16))
    rows = np.ones(len(ids), bool) if rows is None else rows
    tol, typical = K.tolerance(ids, cfg, p, dtype, want, rows), K.tolerance(ids, cfg, p, dtype, want, rows, np.median)
    assert tol < CAP[dtype], tol
    for cuts in cuts_list:
        err = K.row_err(K.run(L, model, ids, cuts), want)[rows]
        assert err.max() < tol, (cuts, int(err.argmax()), float(err.max()), tol)
        assert np.median(err) < typical, (cuts, float(np.median(err)), typical)
    for m in mistakes:  # the mistake would have shown (in 16 bits: the loss of a state)
        if dtype != "f32" and not isinstance(m, dict):
            continue
        wrong = plain.forward(ids, cfg, p, **(m if isinstance(m, dict) else dict(without=m)))
        assert K.row_err(wrong, want)[rows].max() > 1.5 * tol, m
    return model


def _close(ids, got, cfg, p, dtype):
    """got: logits of the whole sequence."""
    want = plain.forward(ids, cfg, p)
    tol = K.tolerance(ids, cfg, p, dtype, want)
    err = K.row_err(got, want)
    assert tol < CAP[dtype] and err.max() < tol, (int(err.argmax()), float(err.max()), tol)


# ---- one mechanism at a time ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,scale", [(64, 3.0), (36, 0.3), (72, 1.0)])
def test_embedding_and_norms(L, dtype, width, scale):
    cfg = K.config([(K.matrix(), None)], width=width, scale=scale, eps=0.05)
    p = _silence(K.weights(L, cfg, 1), "mix.o")
    _check(L, cfg, p, _ids(140), ([140], [1], [2], [70, 1, 1, 3]), dtype, mistakes=("embedding scale",) if scale != 1.0 else ())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,cap", [
    (3, 24, 40, 9.0), (1, 8, 8, 2.0), (2, 64, 72, 15.0), (5, 7, 9, 6.0), (2, 256, 136, 4.0), (2, 72, 264, 12.0), (1, 192, 300, 9.0), (2, 264, 48, 9.0),
    (1, 16, 520, 3.0), (4, 128, 24, 8.0), (7, 1, 3, 9.0),
])
def test_matrix_memory_alone(L, dtype, heads, dim, vdim, cap):
    """Sizes for every kernel: chunks on the tensor cores with 1 to 4 key blocks and 1 to 5 value tiles, and token by token with
    one to eight slices of the columns, four or one at a time."""
    cfg = K.config([(K.matrix(heads, dim, vdim, cap), None)], eps=0.01)
    _check(L, cfg, K.weights(L, cfg, 2), _ids(290, 2), ([290], [150, 1], [130, 65, 64], [70, 2, 30, 3]), dtype,
           mistakes=("gate bias", "gate cap", "log of the forget gate", "decay", "head norm", "output gate", dict(forget_at=70)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_denominator_of_the_matrix_memory(L, dtype):
    """A head's norm takes out the size of what it norms, unless eps is as large."""
    cfg = K.config([(K.matrix(3, 16, 24, 6.0), None)], eps=0.5)
    p = K.weights(L, cfg, 3)
    _check(L, cfg, p, _ids(200, 3), ([200], [1], [130, 3]), dtype, mistakes=("normaliser", "floor", "query scale"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("forget,gain", [(7.0, 1.0), (-6.0, 1.0), (2.0, 12.0)])
def test_gates_far_from_their_middle(L, dtype, forget, gain):
    """Memories that keep everything, that keep nothing, and gates that jump between the two."""
    cfg = K.config([(K.matrix(2, 32, 24, 14.0), None)], eps=0.1)
    p = K.weights(L, cfg, 4, forget=forget)
    for n in ("l0.mix.i", "l0.mix.f"):
        p[n] = K.bf16_exact(p[n] * gain)
    _check(L, cfg, p, _ids(400, 4), ([400], [129, 1], [257, 5]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("a", [
    dict(), dict(heads=6, kv_heads=2, dim=64, vdim=64, chunk=64, rot_dims=64), dict(heads=4, kv_heads=1, dim=128, vdim=128, chunk=100, rot_dims=32, scaling=None),
    dict(heads=5, kv_heads=5, dim=72, vdim=40, chunk=7, rot_dims=2), dict(heads=2, kv_heads=1, dim=192, vdim=120, chunk=1000, rot_dims=48),
    dict(heads=3, kv_heads=1, dim=200, vdim=64, chunk=33, rot_dims=200), dict(heads=8, kv_heads=2, dim=40, vdim=136, chunk=65, rot_dims=8),
    dict(heads=4, kv_heads=2, dim=7, vdim=5, chunk=50, rot_dims=6), dict(heads=2, kv_heads=2, dim=300, vdim=16, chunk=128, rot_dims=10),
    dict(heads=10, kv_heads=1, dim=64, vdim=40, chunk=90, rot_dims=24), dict(heads=18, kv_heads=2, dim=96, vdim=128, chunk=400, rot_dims=96),
    dict(heads=1, kv_heads=1, dim=16, vdim=8, chunk=1, rot_dims=4), dict(heads=3, kv_heads=3, dim=48, vdim=70, chunk=192, rot_dims=0),
])
def test_attention_alone(L, dtype, a):
    """Sizes for every kernel: tensor-core prompts with 1 to 3 key blocks and 64 or 128 values, single rows on the warp-level tensor cores
    (1 to 4 key blocks, one or two value blocks, up to two groups of heads), and the general row kernel of every width."""
    kw = dict(a, scale=0.6 * a.get("dim", 32) ** -0.5)
    cfg = K.config([(K.attn(**kw), None)])
    mistakes = ["query norm", "key norm", "sink", "head gate"]
    if kw["chunk"] > 1 if "chunk" in kw else True:
        mistakes += ["position"] if kw.get("rot_dims", 20) > 4 else []
        mistakes += ["chunks"] if kw.get("chunk", 48) < 200 else []
        mistakes += ["grouping"] if 1 < kw.get("kv_heads", 2) < kw.get("heads", 4) else []
    else:
        mistakes = ["sink", "head gate", "chunks"]
    _check(L, cfg, K.weights(L, cfg, 5), _ids(210, 5), ([210], [140, 1], [75, 65], [70, 2, 30, 3]), dtype, mistakes=mistakes)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scaling", [dict(factor=8.0, low=1.0, high=4.0, original=256), dict(factor=2.0, low=3.0, high=9.0, original=1000), None])
def test_frequency_scaling(L, dtype, scaling):
    """Large queries and keys, so that angles decide; every pair of the three ranges of wavelengths is there."""
    a = K.attn(heads=2, kv_heads=1, dim=32, vdim=32, chunk=500, rot_dims=32, base=3000.0, scaling=scaling, scale=1.0)
    cfg = K.config([(a, None)])
    p = K.weights(L, cfg, 6)
    _check(L, cfg, p, _ids(180, 6), ([180], [170, 1], [90, 2]), dtype, mistakes=("frequency scaling",) if scaling else ())


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_and_values_of_another_layer(L, dtype):
    """Three layers read the first one's rows, through masks and scales of their own; one in between has its own."""
    shared = dict(heads=4, kv_heads=2, dim=32, vdim=24)
    cfg = K.config([(K.attn(**shared, chunk=40, scale=0.2), None), (K.attn(**shared, chunk=90, scale=0.3, kv_from=0), None),
                    (K.attn(**shared, chunk=70, scale=0.25), None), (K.attn(**shared, chunk=1000, scale=0.15, kv_from=0), None),
                    (K.attn(**shared, chunk=25, scale=0.2, kv_from=2), None)])
    _check(L, cfg, K.weights(L, cfg, 7), _ids(200, 7), ([200], [1], [140, 1], [70, 66, 2]), dtype, mistakes=("whose keys", "chunks"))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff", [(64, 88), (64, 1), (72, 300), (36, 50), (328, 96)])
def test_feed_forward_alone(L, dtype, width, ff):
    cfg = K.config([(K.matrix(), ff)], width=width)
    p = _silence(K.weights(L, cfg, 8), "mix.o")
    _check(L, cfg, p, _ids(150, 8), ([150], [1], [9], [131, 2]), dtype, mistakes=("which is gated", "norm before"))


# ---- the whole model -------------------------------------------------------------------------------------
# (Seed 42: no position at which rounding alone moves the logits of this model far; a matrix memory's output may nearly vanish.)
def _mixed(**kw):
    """Both mixers, with and without a feed-forward, in every succession."""
    kw.setdefault("eps", 0.1)
    return K.config([(K.matrix(), None), (K.matrix(2, 16, 24, 5.0), 40), (K.attn(scale=0.15), 88), (K.attn(heads=2, dim=16, vdim=40, chunk=30, rot_dims=12, scale=0.2), None),
                     (K.matrix(4, 8, 16), None), (K.attn(chunk=75, scale=0.12, kv_from=2), 56)], **kw)


@pytest.mark.parametrize("cuts", [[200], [1], [2], [3, 2], [64], [65, 1], [63, 64, 1], [128, 2, 2, 1], [17, 100, 2], [199, 1], [47, 2, 48]])
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions(L, dtype, cuts):
    cfg = _mixed()
    _check(L, cfg, K.weights(L, cfg, 42), _ids(200, 42), (cuts,), dtype)


def test_attention_in_the_first_layer(L):
    cfg = K.config([(K.attn(), None), (K.matrix(), 40)])
    for dtype in DTYPES:
        _check(L, cfg, K.weights(L, cfg, 10), _ids(150, 10), ([150], [1], [70, 3]), dtype)


@pytest.mark.parametrize("width", [40, 36, 68])
def test_widths_beside_the_tensor_cores(L, width):
    """Row lengths that TMA cannot step over take the 32-bit kernels in bf16 models too."""
    cfg = K.config([(K.matrix(), 33), (K.attn(scale=0.15), 50)], width=width)
    _check(L, cfg, K.weights(L, cfg, 11), _ids(140, 11), ([140], [1], [70, 2]), "bf16")


def test_long_decoding(L):
    cfg = _mixed()
    p, ids = K.weights(L, cfg, 42), _ids(420, 42)
    for dtype in DTYPES:
        _check(L, cfg, p, ids, ([20, 1],), dtype)


def _one_token_opens_the_gate(L, token, vocab, width, seed):
    """A memory that forgets nothing and that `token` alone writes strongly (by a number of its embedding that no other has)."""
    cfg = K.config([(K.matrix(1, 16, 16, 12.0), None)], vocab=vocab, width=width, eps=0.02)
    p = K.weights(L, cfg, seed, forget=40.0)
    p["embed"][:, 0] = 0
    p["embed"][token, 0] = 2
    p["l0.norm1"][0] = 1
    p["l0.mix.i"] = np.zeros_like(p["l0.mix.i"])
    p["l0.mix.i"][0, 0] = 8
    p["l0.mix.i.b"] = np.full(1, -6, np.float32)
    p["l0.mix.f"] = np.zeros_like(p["l0.mix.f"])
    return cfg, p


def test_a_portion_of_many_chunks(L):
    """More chunks than the memories of which are kept at a time; what was stored in the first ones is still read in the last."""
    n = 64 * 128 + 300
    cfg, p = _one_token_opens_the_gate(L, 45, 50, 32, 13)
    ids = _ids(n, 13, 40)
    ids[100] = 45
    rows = np.zeros(n, bool)
    rows[-300:] = True
    for dtype in DTYPES:
        _check(L, cfg, p, ids, ([n], [n - 100, 60, 2]), dtype, rows=rows, mistakes=(dict(forget_at=101), dict(forget_at=64 * 128)))


@pytest.mark.parametrize("dtype", DTYPES)
def test_equal_sequences_in_a_batch_match_each_alone(L, dtype):
    cfg = _mixed()
    p = K.weights(L, cfg, 42)
    model = K.build(L, cfg, p, dtype, 240)
    ids = _ids(3 * 215, 42).reshape(3, 215)
    caches = model.init_kv_caches(3)
    got = []
    with L.no_grad():
        at = 0
        for n in [150, 2, 1, 1, 1, 20, 1, 4, 35]:
            got.append(model.forward(ids[:, at:at + n].astype(np.float32), caches))
            at += n
    got = np.concatenate(got, axis=1)
    for b in range(3):
        _close(ids[b], got[b], cfg, p, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_caches_reset_and_used_again(L, dtype):
    """A long sequence, then short ones in the same caches: nothing of the first (rows, memories, maxima) is seen."""
    cfg = _mixed()
    p = K.weights(L, cfg, 42, forget=6.0)
    model = K.build(L, cfg, p, dtype, 170)
    caches = model.init_kv_caches(1)
    for seed, n, cuts in ((1, 170, [170]), (2, 9, [1]), (3, 80, [70, 1]), (4, 2, [2]), (5, 1, [1]), (6, 140, [140]), (7, 12, [3])):
        model.reset_kv_caches(caches)
        ids = _ids(n, seed)
        _close(ids, K.run(L, model, ids, cuts, caches), cfg, p, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_and_freed_caches(L, dtype):
    """Requests take turns, step by step; caches of finished ones serve new ones."""
    from lumen_b200.replay import TraceReplay
    cfg = _mixed()
    p = K.weights(L, cfg, 42)
    replay = TraceReplay(K.build(L, cfg, p, dtype, 160))
    ids = {r: _ids(n, i) for i, (r, n) in enumerate([("a", 150), ("b", 41), ("c", 90), ("d", 5)])}
    at, got = {r: 0 for r in ids}, {r: [] for r in ids}
    rng = np.random.default_rng(17)
    with L.no_grad():
        pending, waiting = ["a", "b"], ["c", "d"]
        while pending:
            r = pending[rng.integers(len(pending))]
            n = min(int(rng.choice([1, 1, 2, 3, 30, 70])), len(ids[r]) - at[r])
            got[r].append(replay.entry(r, ids[r][at[r]:at[r] + n].tolist(), list(range(n))))
            at[r] += n
            if at[r] == len(ids[r]):
                replay.end(r)
                pending.remove(r)
                if waiting:
                    pending.append(waiting.pop(0))
    assert len(replay.free) == 2  # two sets of caches served four requests
    for r in ids:
        _close(ids[r], np.concatenate(got[r]), cfg, p, dtype)


# ---- far keys and chunk borders ----------------------------------------------------------------------------
def _standing_out(L, chunk, dim, vdim, heads=2, seed=18):
    """One attention layer in which token 96 asks for token 95: the keys' and queries' rotated part is silent, and the first head's
    query of that token is its key, so that one score stands out among hundreds."""
    rot = 8
    cfg = K.config([(K.attn(heads=heads, kv_heads=1, dim=dim, vdim=vdim, chunk=chunk, rot_dims=rot, scale=16.0 / (dim - rot)), None)], eps=1e-6)
    p = K.weights(L, cfg, seed)
    for n in ("q.norm", "k.norm"):
        p["l0.mix." + n] = np.concatenate([np.zeros(rot), np.ones(dim - rot)]).astype(np.float32)
    p["l0.norm1"] = np.ones_like(p["l0.norm1"])
    p["l0.mix.sink"] = np.zeros_like(p["l0.mix.sink"])
    key = p["l0.mix.k"].astype(np.float64) @ p["embed"][95]
    row = np.linalg.pinv(p["l0.mix.q"][:dim].astype(np.float64)) @ key
    p["embed"][96] = K.bf16_exact(row / np.sqrt(np.mean(row * row)) * 0.4)
    p["l0.mix.g"] = np.zeros_like(p["l0.mix.g"])
    return cfg, p


def _borders(chunk):
    """(query, key): just inside and just outside the chunk, at tile borders, far away."""
    c = chunk
    out = [(1, 0), (63, 0), (64, 1), (65, 64), (127, 63), (128, 0), (129, 127), (200, 65), (299, 0), (299, 191), (299, 298)]
    for k in (1, 2):
        out += [(k * c, k * c - 1), (k * c + 1, k * c), (k * c + c - 1, k * c), (k * c + c - 1, k * c - 1), (k * c + c // 2, k * c), (k * c + c // 2, k * c - 1)]
    return sorted({(i, j) for i, j in out if 0 <= j < i < 300})


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk,dim,vdim", [(48, 40, 24), (128, 56, 40), (100, 37, 24), (1000, 40, 72), (63, 60, 24), (65, 40, 24), (32, 36, 20)])
def test_far_keys_and_chunk_borders(L, dtype, chunk, dim, vdim):
    cfg, p = _standing_out(L, chunk, dim, vdim)
    model = K.build(L, cfg, p, dtype, 304)
    caches = model.init_kv_caches(1)
    seen = unseen = 0
    for i, j in _borders(chunk):
        ids = _ids(i + 1, 100 + i + j, 90)
        ids[j], ids[i] = 95, 96
        want = plain.forward(ids, cfg, p)
        tol = K.tolerance(ids, cfg, p, dtype, want)
        assert tol < CAP[dtype], tol
        if i // chunk == j // chunk:  # without that key the last position would say something else
            seen += 1
            assert K.row_err(plain.forward(ids, cfg, p, hidden_key=j), want)[i] > 0.2, (i, j)
        else:  # and with it, too
            unseen += 1
            if j == i // chunk * chunk - 1:
                assert K.row_err(plain.forward(ids, cfg, p, without="one key more"), want)[i] > 0.2, (i, j)
        for cuts in ([i + 1], [i, 1], [i - 1, 2] if i > 1 else [1], [37], [max(1, i - 70), 71]):
            model.reset_kv_caches(caches)
            err = K.row_err(K.run(L, model, ids, cuts, caches), want)
            assert err.max() < tol, (i, j, cuts, int(err.argmax()), float(err.max()), tol)
    assert seen > 3 and (unseen > 3 or chunk >= 300)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_memory_of_a_far_token(L, dtype):
    """Token 95 opens the input gate of a memory that forgets nothing: it is read hundreds of tokens later, wherever the sequence
    was cut between."""
    cfg, p = _one_token_opens_the_gate(L, 95, 101, 64, 19)
    ids = _ids(430, 20, 90)
    ids[5] = 95
    rows = np.arange(430) > 300
    _check(L, cfg, p, ids, ([430], [1], [129, 2, 128, 1], [64], [6, 3, 300, 1]), dtype, rows=rows, mistakes=(dict(forget_at=6), dict(forget_at=300)))


# ---- errors, entry points ----------------------------------------------------------------------------------
def test_errors_come_back_as_status_codes(L):
    cfg = _mixed()
    model = K.build(L, cfg, K.weights(L, cfg, 1), "f32", 16)
    caches = model.init_kv_caches(1)
    with L.no_grad():
        for ids, code in ((np.full((1, 1), 101.0), L._lib.ERR_EMBED_RANGE), (np.zeros((1, 17)), L._lib.ERR_KV_OVERFLOW), (np.zeros((2, 1)), L._lib.ERR_SHAPE)):
            with pytest.raises(L.LumenError) as e:
                model.forward(ids, caches)
            assert e.value.code == code
        for c in caches[:3]:
            with pytest.raises(L.LumenError):
                c.read()  # a state, or rows of two sizes
    for layers in ([(K.attn(kv_from=0), None)], [(K.matrix(), None), (K.attn(kv_from=0), None)], [(K.attn(), None), (K.attn(kv_from=0), None), (K.attn(kv_from=1), None)],
                   [(K.attn(), None), (K.attn(dim=16, rot_dims=8, kv_from=0), None)], [(K.attn(heads=3, kv_heads=2), None)], [(K.attn(rot_dims=40), None)]):
        with pytest.raises(L.LumenError):
            L.FekoraxModel(L.FekoraxConfig.from_dict(K.config(layers), 16, "f32"))


def test_greedy_generation_through_the_chat_session(L):
    cfg = _mixed()
    p = K.weights(L, cfg, 21)
    prompt, n = _ids(21, 21).tolist(), 40
    seq = list(prompt)
    for _ in range(n):
        lg = plain.forward(seq, cfg, p)[-1]
        top = np.sort(lg)[-2:]
        assert top[1] - top[0] > 1e-3  # no close call
        seq.append(int(lg.argmax()))
    from lumen_b200.chat import ChatSession
    s = ChatSession(K.build(L, cfg, p, "f32", 160), lambda t: t, lambda t: t, temperature=0.0, top_p=1.0, repetition_penalty=1.0, max_gen=n)
    assert s.turn(prompt) == seq[len(prompt):]
    # a second turn continues in the kept caches
    more = _ids(6, 22).tolist()
    want = int(plain.forward(seq + more, cfg, p)[-1].argmax())
    s.max_gen = 1
    assert s.turn(more) == [want]
    s.reset()  # and a new conversation starts from nothing
    s.max_gen = 5
    assert s.turn(prompt) == seq[len(prompt):len(prompt) + 5]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_program_and_command_line(L, tmp_path, dtype):
    from lumen_b200.loader import save_safetensors
    from lumen_b200.synth import f32_to_bf16_bits
    cfg = _mixed()
    p = K.weights(L, cfg, 42)
    kind = "f32" if dtype == "float32" else "bf16"
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(tmp_path / "model.safetensors", {k: f32_to_bf16_bits(v).reshape(v.shape) for k, v in p.items()})
    ids = {"x": _ids(140, 1), "y": _ids(7, 2)}
    steps = [("x", 0, 70, [0, 69]), ("x", 70, 72, [1]), ("x", 72, 139, []), ("x", 139, 140, [0]), ("y", 0, 6, [2, 5]), ("y", 6, 7, [0])]
    lines = "".join(json.dumps({"step": i, "entries": [{"id": r, "tokens": ids[r][a:b].tolist(), "want": w}],
                                "end": [r] if b == len(ids[r]) else []}) + "\n" for i, (r, a, b, w) in enumerate(steps))
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "140"],
                       input=lines, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(6)]
    assert not (out / "2.f32").exists()
    for i, (rid, a, b, w) in enumerate(steps):
        if w:
            got = np.fromfile(out / f"{i}.f32", "<f4").reshape(len(w), 101)
            want = plain.forward(ids[rid], cfg, p)
            full = want.copy()
            full[[a + k for k in w]] = got
            assert K.row_err(full, want).max() < K.tolerance(ids[rid], cfg, p, kind, want), i
    if dtype == "float32":
        seq = ids["y"].tolist()
        for _ in range(3):
            seq.append(int(plain.forward(seq, cfg, p)[-1].argmax()))
        env = dict(os.environ, PYTHONPATH=str(ROOT))
        r = subprocess.run([sys.executable, "-m", "lumen_b200", "generate", "--model", str(tmp_path), "--dtype", dtype, "--max-new", "3", "--ids",
                            " ".join(map(str, ids["y"]))], capture_output=True, text=True, timeout=600, env=env)
        assert r.returncode == 0 and [int(t) for t in r.stdout.split()] == seq[7:], r.stderr[-2000:]
