"""Plain, slow implementation of the Fekorax decoder in float64 numpy: one function per mechanism, no cache, no portions, no code
shared with the product.  Test infrastructure (small helpers come from fegetar_plain.py).

`cfg` is a config.json dictionary, `p` the parameters by name.  `without` plants one mistake (its name) so that a test can
show that the mistake would be seen.  `forward` can also run in float32, or with the input of every product rounded to
bfloat16: what these two differ from the float64 result by is the error that rounding alone causes.
"""
from __future__ import annotations

import numpy as np

import fegetar_plain as base
from fegetar_plain import gelu_tanh, product, rms_norm, sigmoid, to_bf16  # noqa: F401


def short(x):
    """A projection that a 16-bit model may keep in 16 bits."""
    return x if base._ROUND is None else base._ROUND(x)


def log_gates(h, m, p, pre, without=None):
    """Log input and forget gates [T, heads], in full precision."""
    cap = m["gate_cap"]
    zi, zf = h @ p[pre + "i"].T, h @ p[pre + "f"].T
    if without != "gate bias":
        zi, zf = zi + p[pre + "i.b"], zf + p[pre + "f.b"]
    if without != "gate cap":
        zi, zf = cap * np.tanh(zi / cap), cap * np.tanh(zf / cap)
    return zi, zf if without == "log of the forget gate" else -np.logaddexp(0, -zf)


def mlstm(h, m, p, pre, eps, without=None, forget_at=None):
    """Token by token.  `forget_at`: the state is lost before this token (a planted mistake)."""
    T, H, d, v = len(h), m["heads"], m["dim"], m["vdim"]
    q = short(product(h, p[pre + "q"])).reshape(T, H, d) * (1.0 if without == "query scale" else d ** -0.5)
    k = short(product(h, p[pre + "k"])).reshape(T, H, d)
    val = short(product(h, p[pre + "v"])).reshape(T, H, v)
    i, f = log_gates(h, m, p, pre, without)
    S, n, mx = np.zeros((H, d, v), h.dtype), np.zeros((H, d), h.dtype), np.zeros(H, h.dtype)
    out = np.zeros((T, H, v), h.dtype)
    for t in range(T):
        if t == forget_at:
            S, n, mx = S * 0, n * 0, mx * 0
        new = np.maximum(f[t] + mx, i[t])
        keep, put = np.exp(f[t] + mx - new), np.exp(i[t] - new)
        if without == "decay":
            keep = keep * 0 + 1
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * val[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        mx = new
        den = np.exp(-mx) if without == "normaliser" else np.maximum(np.abs((n * q[t]).sum(1)), 0 if without == "floor" else np.exp(-mx))
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / (den + 1e-6)[:, None]
    if without != "head norm":
        out = rms_norm(out, 1.0, eps)
    y = out.reshape(T, H * v) * p[pre + "norm"]
    if without != "output gate":
        y = y * sigmoid(short(product(h, p[pre + "g"])))
    return product(y, p[pre + "o"])


def frequencies(rot, without=None):
    n = rot["dims"]
    f = rot["base"] ** (-2.0 * np.arange(n // 2) / max(n, 1))
    s = rot.get("scaling")
    if not s or without == "frequency scaling":
        return f
    out = []
    for x in f:
        length = 2 * np.pi / x
        if length < s["original"] / s["high"]:
            out.append(x)
        elif length > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            w = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
            out.append((1 - w) * x / s["factor"] + w * x)
    return np.array(out)


def rotate(x, rot, without=None, shift=0):
    """x [T, heads, n]: the pairs (i, i + dims / 2) turn."""
    half, out = rot["dims"] // 2, x.copy()
    for i, f in enumerate(frequencies(rot, without)):
        a, b = (2 * i, 2 * i + 1) if without == "rotate half" else (i, i + half)
        angle = ((np.arange(len(x)) + shift) * f)[:, None]
        c, s = np.cos(angle).astype(x.dtype), np.sin(angle).astype(x.dtype)
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def first_key(i, m, without=None):
    """The first position that position i sees."""
    size = (m.get("mask") or {}).get("size")
    if not size or without == "chunks":
        return 0
    lo = i // size * size
    return {"one key more": max(lo - 1, 0), "one key less": min(lo + 1, i)}.get(without, lo)


def keys_values(h, m, p, pre, eps, without=None):
    T, G = len(h), m["kv_heads"]
    k = product(h, p[pre + "k"]).reshape(T, G, m["dim"])
    if without != "key norm":
        k = rms_norm(k, p[pre + "k.norm"], eps)
    return short(rotate(k, m["rot"], without)), short(product(h, p[pre + "v"]).reshape(T, G, m["vdim"]))


def attention(h, m, p, pre, eps, kv, without=None, hidden_key=None):
    """`hidden_key`: a position that nobody but itself sees (a planted mistake)."""
    T, H, G = len(h), m["heads"], m["kv_heads"]
    k, v = kv
    q = product(h, p[pre + "q"]).reshape(T, H, m["dim"])
    if without != "query norm":
        q = rms_norm(q, p[pre + "q.norm"], eps)
    q = rotate(q, m["rot"], without, 1 if without == "position" else 0)
    out = np.zeros((T, H, m["vdim"]), h.dtype)
    for i in range(T):
        lo = first_key(i, m, without)
        for hd in range(H):
            g = hd % G if without == "grouping" else hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * (1.0 if without == "score scale" else m["scale"])
            if hidden_key is not None and lo <= hidden_key < i:
                s[hidden_key - lo] = -np.inf
            sink = p[pre + "sink"][hd] * (m["scale"] if without == "sink as it is" else 1)
            top = max(s.max(), sink)
            w = np.exp(s - top)
            out[i, hd] = w @ v[lo:i + 1, g] / (w.sum() + (0 if without == "sink" else np.exp(sink - top)))
    if without != "head gate":
        out = out * sigmoid(product(h, p[pre + "g"]))[:, :, None]
    return product(out.reshape(T, H * m["vdim"]), p[pre + "o"])


def feed_forward(h, p, pre, without=None):
    g, u = product(h, p[pre + "gate"]), product(h, p[pre + "up"])
    return product(g * gelu_tanh(u) if without == "which is gated" else gelu_tanh(g) * u, p[pre + "down"])


def forward(tokens, cfg, p, without=None, hidden_key=None, forget_at=None, dtype=np.float64, rounding=None):
    """Logits [T, vocab] of one sequence."""
    tokens = np.asarray(tokens, dtype=np.int64)
    p = {k: np.asarray(v, dtype=dtype) for k, v in p.items()}
    base._ROUND = rounding
    try:
        return _forward(tokens, cfg, p, without, hidden_key, forget_at)
    finally:
        base._ROUND = None


def _forward(tokens, cfg, p, without, hidden_key, forget_at):
    eps = cfg["norm"]["eps"]
    x = p["embed"][tokens] * (1.0 if without == "embedding scale" else cfg["embedding"]["scale"])

    def sublayer(x, pre, which, f):
        h = x if without == "norm before" else rms_norm(x, p[f"{pre}norm{which}"], eps)
        y = f(h)
        return x + (y if without == "norm after" else rms_norm(y, p[f"{pre}norm{which}b"], eps))

    kvs = {}
    for i, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{i}."

        def mix(h):
            if layer["type"] == "mlstm":
                return mlstm(h, m, p, pre + "mix.", eps, without, forget_at)
            if m.get("kv_from") is None:
                kvs[i] = keys_values(h, m, p, pre + "mix.", eps, without)
            source = i if m.get("kv_from") is None else max(kvs) if without == "whose keys" else m["kv_from"]
            return attention(h, m, p, pre + "mix.", eps, kvs[source], without, hidden_key)

        x = sublayer(x, pre, 1, mix)
        if layer.get("mlp"):
            x = sublayer(x, pre, 2, lambda h: feed_forward(h, p, pre + "mlp.", without))
    return rms_norm(x, p["final.norm"], eps) @ p["embed"].T
