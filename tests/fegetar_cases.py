"""Small Fegetar configurations and random weights for the tests."""
from __future__ import annotations

import numpy as np


def mixer(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=48, rot_dims=None, base=500.0, scale=0.1):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                rot=dict(base=base, dims=rot_dim if rot_dims is None else rot_dims))


def dense(ff=88):
    return dict(kind="dense", ff=ff)


def moe(experts=6, top=2, ff=40, limit=1.5, shared=(56, 0.8)):
    d = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))
    if shared:
        d["shared"] = dict(ff=shared[0], limit=shared[1])
    return d


def config(layers, vocab=101, width=64, eps=1e-4, bigram=(37, 5, 3), side=16):
    """layers: [(mixer, mlp or None)]"""
    c = dict(architecture="Fegetar", vocab=vocab, width=width, norm=dict(eps=eps),
             layers=[dict(type="latent_attention", mixer=m, mlp=f) for m, f in layers])
    if bigram:
        c["embedding"] = dict(bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2]))
    if side:
        c["token_side"] = dict(dim=side)
    return c


def weights(L, cfg, seed=0, round_bf16=True):
    """Random weights under their checkpoint names; matrices keep a row's size, gains are away from their neutral value.
    Values are exact in bf16, so that both storage types hold the same model."""
    from lumen_b200.synth import bf16_bits_to_f32, f32_to_bf16_bits
    shapes = L.FegetarConfig.from_dict(cfg, 8, "f32").param_shapes()
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in sorted(shapes.items()):
        w = rng.standard_normal(shape).astype(np.float32)
        if len(shape) == 1:
            w = w * np.float32(0.3) + np.float32(1.0 if name.endswith(("dkv.norm", "side.norm")) else 0.0)
        elif name in ("embed", "bigram", "side.embed"):
            pass
        elif name.endswith("router"):
            w = w * np.float32(2.0 * shape[1] ** -0.5)
        else:
            w = w * np.float32(1.2 * shape[1] ** -0.5)
        out[name] = bf16_bits_to_f32(f32_to_bf16_bits(w)).reshape(shape) if round_bf16 else w
    return out


def build(L, cfg, p, dtype="f32", max_seq=160):
    model = L.FegetarModel(L.FegetarConfig.from_dict(cfg, max_seq, dtype))
    model.load_state(p)
    return model


def run(L, model, tokens, cuts, caches=None):
    """Logits [T, vocab] with the tokens fed in portions of the given sizes (the last one repeats until the end)."""
    own = caches or model.init_kv_caches(1)
    tokens, out, at = np.asarray(tokens, dtype=np.float32), [], 0
    cuts = list(cuts)
    with L.no_grad():
        while at < len(tokens):
            n = min(cuts.pop(0) if len(cuts) > 1 else cuts[0], len(tokens) - at)
            out.append(model.forward(tokens[None, at:at + n], own)[0])
            at += n
    assert all(c.len == len(tokens) for c in own) or caches is not None
    return np.concatenate(out)


def row_err(got, want):
    """Per position: rms of the difference over rms of the logits (means taken off)."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


FLOOR = {"f32": 4e-6, "bf16": 6e-3}


def tolerance(ids, cfg, p, dtype, want, rows=None):
    """Three times what rounding alone does to this model and these tokens (see row_err), and at least a floor."""
    import fegetar_plain as plain
    if dtype == "f32":
        near = plain.forward(ids, cfg, p, dtype=np.float32)
    else:
        near = plain.forward(ids, cfg, p, rounding=plain.to_bf16)
    err = row_err(near, want)
    return max(3 * float((err if rows is None else err[rows]).max()), FLOOR[dtype])
