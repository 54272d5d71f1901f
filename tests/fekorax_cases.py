"""Small Fekorax configurations and random weights for the tests."""
from __future__ import annotations

import numpy as np

from fegetar_cases import row_err, run  # noqa: F401

FLOOR = {"f32": 8e-6, "bf16": 6e-3}


def matrix(heads=3, dim=24, vdim=40, gate_cap=9.0):
    return "mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap)


SCALING = dict(factor=3.0, low=1.5, high=5.0, original=300)


def attn(heads=4, kv_heads=2, dim=32, vdim=24, chunk=48, rot_dims=20, base=700.0, scaling=SCALING, scale=0.21, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=chunk), rot=dict(base=base, dims=rot_dims))
    if scaling:
        m["rot"]["scaling"] = scaling
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def config(layers, vocab=101, width=64, eps=1e-4, scale=3.0):
    """layers: [((type, mixer), ff or None)]"""
    return dict(architecture="Fekorax", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                layers=[dict(type=t, mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None) for (t, m), ff in layers])


def weights(L, cfg, seed=0, forget=2.0):
    """Random weights under their checkpoint names; matrices keep a row's size, gains are away from one, `forget`: mean bias of the
    forget gates.  Values are exact in bf16, so that both storage types hold the same model."""
    shapes = L.FekoraxConfig.from_dict(cfg, 8, "f32").param_shapes()
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in sorted(shapes.items()):
        w = rng.standard_normal(shape).astype(np.float32)
        if name.endswith(".f.b"):
            w = w + np.float32(forget)
        elif name.endswith((".i.b", ".sink")):
            pass
        elif len(shape) == 1:
            w = w * np.float32(0.3) + np.float32(1.0)
        elif name == "embed":
            w = w * np.float32(0.4)
        else:
            w = w * np.float32(1.2 * shape[1] ** -0.5)
        out[name] = bf16_exact(w)
    return out


def bf16_exact(w):
    from lumen_b200.synth import bf16_bits_to_f32, f32_to_bf16_bits
    w = np.asarray(w, np.float32)
    return bf16_bits_to_f32(f32_to_bf16_bits(w)).reshape(w.shape)


def build(L, cfg, p, dtype="f32", max_seq=160):
    model = L.FekoraxModel(L.FekoraxConfig.from_dict(cfg, max_seq, dtype))
    model.load_state(p)
    return model


def tolerance(ids, cfg, p, dtype, want, rows=None, of=np.max):
    """Three times what rounding alone does to this model and these tokens (see row_err; `of`: the worst position, or the median one),
    and at least a floor."""
    import fekorax_plain as plain
    near = plain.forward(ids, cfg, p, **(dict(dtype=np.float32) if dtype == "f32" else dict(rounding=plain.to_bf16)))
    err = row_err(near, want)
    return max(3 * float(of(err if rows is None else err[rows])), FLOOR[dtype])
