"""Plain, slow implementation of the Fegetar decoder in float64 numpy: one function per mechanism, no cache, no batching, no
code shared with the product.  Test infrastructure.

`cfg` is a config.json dictionary, `p` the parameters by name.  `without` plants one mistake (its name) so that a test can
show that the mistake would be seen.

`forward` can also run in float32, or with the input of every product rounded to bfloat16: what these two differ from the
float64 result by is the error that rounding alone causes in a model, and the measure of the tests' tolerances.
"""
from __future__ import annotations

import numpy as np

_ROUND = None  # applied to the inputs of products (None: exact)


def product(x, w):
    return (x if _ROUND is None else _ROUND(x)) @ w.T


def to_bf16(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = (u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) & np.uint32(0xFFFF0000)
    return u.view(np.float32).reshape(np.shape(x)).astype(np.asarray(x).dtype)


def rms_norm(x, gain, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * gain


def gelu_tanh(z):
    return 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def embed_tokens(tokens, cfg, p, without=None):
    x = p["embed"][tokens].copy()
    big = cfg.get("embedding", {}).get("bigram")
    if big and without != "bigram":
        n = big["buckets"]
        for t, tok in enumerate(tokens):
            row = n if t == 0 and without != "first row" else (int(tokens[max(t - 1, 0)]) * big["mul_prev"] + int(tok) * big["mul_cur"]) % n
            x[t] += p["bigram"][row]
    return x


def rotate(v, positions, rot, without=None):
    """v [T, ..., n]; the first rot['dims'] numbers turn in pairs (2i, 2i + 1)."""
    n = rot["dims"]
    out = v.copy()
    for i in range(n // 2):
        angle = (positions + (1 if without == "position" else 0)) * rot["base"] ** (-2.0 * i / n)
        angle = angle.reshape((-1,) + (1,) * (v.ndim - 2))
        a, b = (i, i + n // 2) if without == "interleaving" else (2 * i, 2 * i + 1)
        out[..., a] = v[..., a] * np.cos(angle) - v[..., b] * np.sin(angle)
        out[..., b] = v[..., b] * np.cos(angle) + v[..., a] * np.sin(angle)
    return out


def latent_attention(h, m, p, pre, eps, without=None, hidden_key=None):
    """`hidden_key`: a position that nobody but itself sees (a planted mistake)."""
    T, H, d, r, vd, rank = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (product(h, p[pre + "q"])).reshape(T, H, d + r)
    down = product(h, p[pre + "dkv"])
    c = down[:, :rank] if without == "latent norm" else rms_norm(down[:, :rank], p[pre + "dkv.norm"], eps)
    k_rot = rotate(down[:, rank:], pos, m["rot"], without)
    q_rot = rotate(q[..., d:], pos, m["rot"], None if without == "position" else without)
    k = product(c, p[pre + "uk"]).reshape(T, H, d)
    v = product(c, p[pre + "uv"]).reshape(T, H, vd)
    gate = sigmoid(product(h, p[pre + "g"]))
    out = np.zeros((T, H, vd), h.dtype)
    for i in range(T):
        s = (np.einsum("hd,jhd->hj", q[i, :, :d], k[:i + 1]) + np.einsum("hr,jr->hj", q_rot[i], k_rot[:i + 1])) * m["scale"]
        if hidden_key is not None and hidden_key < i:
            s[:, hidden_key] = -np.inf
        w = np.exp(s - s.max(axis=1, keepdims=True))
        w /= w.sum(axis=1, keepdims=True)
        out[i] = np.einsum("hj,jhv->hv", w, v[:i + 1])
        if without != "gate":
            out[i] *= gate[i][:, None]
    return product(out.reshape(T, H * vd), p[pre + "o"])


def dense(h, p, pre):
    return product(gelu_tanh(product(h, p[pre + "up"])), p[pre + "down"])


def expert(h, p, pre, limit):
    g = np.minimum(product(h, p[pre + ".gate"]), limit)
    u = np.clip(product(h, p[pre + ".up"]), -limit, limit)
    return product(g * sigmoid(1.702 * g) * (u + 1), p[pre + ".down"])


def router_scores(h, p, pre):
    return sigmoid(h @ p[pre + "router"].T)


def moe(h, mlp, p, pre, without=None):
    scores = router_scores(h, p, pre)
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e in np.argsort(-scores[t], kind="stable")[:mlp["router"]["top"]]:
            w = scores[t, e]
            if without == "weighted input":
                out[t] += w * expert(h[t], p, f"{pre}e{e}", mlp["expert"]["limit"])
            else:
                out[t] += expert(w * h[t], p, f"{pre}e{e}", mlp["expert"]["limit"])
    if mlp.get("shared") and without != "shared":
        out += expert(h, p, pre + "shared", mlp["shared"]["limit"])
    return out


def side_input(x, tokens, layer, dim, p, pre, eps):
    e = p["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    y = product(gelu_tanh(product(x, p[pre + "gate"])) * e, p[pre + "proj"])
    return rms_norm(y, p[pre + "norm"], eps)


def forward(tokens, cfg, p, without=None, hidden_key=None, dtype=np.float64, rounding=None):
    """Logits [T, vocab] of one sequence."""
    global _ROUND
    tokens = np.asarray(tokens, dtype=np.int64)
    p = {k: np.asarray(v, dtype=dtype) for k, v in p.items()}
    _ROUND = rounding
    try:
        return _forward(tokens, cfg, p, without, hidden_key)
    finally:
        _ROUND = None


def _forward(tokens, cfg, p, without, hidden_key):
    eps = cfg["norm"]["eps"]
    x = embed_tokens(tokens, cfg, p, without)
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        one = 0.0 if without == "gain around one" else 1.0
        y = latent_attention(x, layer["mixer"], p, pre + "mix.", eps, without, hidden_key)
        x = x + rms_norm(y, one + p[pre + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = dense(x, p, pre + "mlp.") if mlp["kind"] == "dense" else moe(x, mlp, p, pre + "mlp.", without)
            x = x + rms_norm(y, one + p[pre + "norm2"], eps)
        if cfg.get("token_side") and without != "side":
            x = x + side_input(x, tokens, i, cfg["token_side"]["dim"], p, pre + "side.", eps)
    return rms_norm(x, 1.0 + p["final.norm"], eps) @ p["head"].T
