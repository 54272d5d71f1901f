"""Plain, slow implementation of the Fegetar decoder in float64 numpy: one function per mechanism, no cache, no batching, no
code shared with the product.  Test infrastructure.

`cfg` is a config.json dictionary, `p` the parameters by name.  `without` plants one mistake (its name) so that a test can
show that the mistake would be seen.
"""
from __future__ import annotations

import numpy as np


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
    q = (h @ p[pre + "q"].T).reshape(T, H, d + r)
    down = h @ p[pre + "dkv"].T
    c = down[:, :rank] if without == "latent norm" else rms_norm(down[:, :rank], p[pre + "dkv.norm"], eps)
    k_rot = rotate(down[:, rank:], pos, m["rot"], without)
    q_rot = rotate(q[..., d:], pos, m["rot"], None if without == "position" else without)
    k = (c @ p[pre + "uk"].T).reshape(T, H, d)
    v = (c @ p[pre + "uv"].T).reshape(T, H, vd)
    gate = sigmoid(h @ p[pre + "g"].T)
    out = np.zeros((T, H, vd))
    for i in range(T):
        s = (np.einsum("hd,jhd->hj", q[i, :, :d], k[:i + 1]) + np.einsum("hr,jr->hj", q_rot[i], k_rot[:i + 1])) * m["scale"]
        if hidden_key is not None and hidden_key < i:
            s[:, hidden_key] = -np.inf
        w = np.exp(s - s.max(axis=1, keepdims=True))
        w /= w.sum(axis=1, keepdims=True)
        out[i] = np.einsum("hj,jhv->hv", w, v[:i + 1])
        if without != "gate":
            out[i] *= gate[i][:, None]
    return out.reshape(T, H * vd) @ p[pre + "o"].T


def dense(h, p, pre):
    return gelu_tanh(h @ p[pre + "up"].T) @ p[pre + "down"].T


def expert(h, p, pre, limit):
    g = np.minimum(h @ p[pre + ".gate"].T, limit)
    u = np.clip(h @ p[pre + ".up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ p[pre + ".down"].T


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
    y = (gelu_tanh(x @ p[pre + "gate"].T) * e) @ p[pre + "proj"].T
    return rms_norm(y, p[pre + "norm"], eps)


def forward(tokens, cfg, p, without=None, hidden_key=None, streams=None):
    """Logits [T, vocab] of one sequence.  `streams`: a list that receives the residual after every layer."""
    tokens = np.asarray(tokens, dtype=np.int64)
    p = {k: np.asarray(v, dtype=np.float64) for k, v in p.items()}
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
        if streams is not None:
            streams.append(x)
    return rms_norm(x, 1.0 + p["final.norm"], eps) @ p["head"].T
