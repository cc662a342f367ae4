"""Petelix, written out plainly: float64 numpy over a whole sequence, one function per mechanism.

Shares no code with the package.  A model is a dict `cfg` (the nested form of its config.json) and a dict of
float64 arrays by tensor name; `run(cfg, tensors, tokens)` returns the logits of every position, `streams(...)` the
residual stream behind every layer.

Notation: T positions, d width, H query heads, G key/value heads, dk key size, dv value size, eps the norms' epsilon.
  R(x, w)          x / sqrt(mean(x^2) + eps) * w
  layer            x <- x + attention(R_1(x));  x <- x + experts(R_2(x))
  attention        q = R(W_q h, w_q) and k = R(W_k h, w_k) over the whole rows, then split into heads and rotated on their
                   first r elements (2i with 2i + 1); v = W_v h; s = c tanh(scale (q . k) / c) over 0 <= i - j < window;
                   p_j = exp(s_j) / (1 + sum exp s); heads side by side times sigmoid(W_g h); W_o.  A layer may take another
                   layer's k and v instead of its own
  experts          s = softmax(W_r h) over experts and identity experts; chosen by s + b inside the groups whose largest
                   s + b is among the `keep` largest; sum of s_e W_down (silu(W_gate h) * (W_up h)), of s_e h for an identity
"""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def rotary_frequencies(dims, base):
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)


def rotate(x, positions, freqs):
    """x [T, heads, size]: of each head the first 2 len(freqs) elements, element 2i with 2i + 1.  The angle is a float32
    product (positions and angles are 32-bit in the design); the rest is float64."""
    n = len(freqs)
    a = (np.asarray(positions, dtype=np.float32)[:, None] * np.asarray(freqs, dtype=np.float32)[None, :]).astype(np.float64)
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    out = x.copy()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def softmax_with_one_more(s):
    """s [..., keys] (minus infinity: not visible) -> exp(s) / (1 + sum exp(s))."""
    m = np.maximum(s.max(-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(-m))


def visible(T, window):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i - j < (T if window is None else window))


def attend(q, k, v, scale, cap, window):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], positions 0..T-1 -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    see = visible(T, window)
    out = np.empty((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap:
            s = soft_cap(s, cap)
        out[:, h] = softmax_with_one_more(np.where(see, s, -np.inf)) @ v[:, g]
    return out


def keys_and_values(h, w, p, m, eps):
    T = h.shape[0]
    k = norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).reshape(T, m["kv_heads"], m["dim"])
    if m.get("rot"):
        k = rotate(k, np.arange(T), rotary_frequencies(m["rot"]["dims"], m["rot"]["base"]))
    return k, (h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"])


def queries(h, w, p, m, eps):
    T = h.shape[0]
    q = norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).reshape(T, m["heads"], m["dim"])
    if m.get("rot"):
        q = rotate(q, np.arange(T), rotary_frequencies(m["rot"]["dims"], m["rot"]["base"]))
    return q


def attention(h, w, p, m, eps, kv):
    q = queries(h, w, p, m, eps)
    window = m["mask"]["size"] if m.get("mask") else None
    a = attend(q, kv[0], kv[1], m["scale"], m.get("softcap"), window).reshape(h.shape[0], -1)
    return (a * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def choose(s, b, top, count, keep):
    """s [E] scores, b [E] correction -> the chosen experts, the largest s + b first."""
    c = s + b
    per = len(s) // count
    best = c.reshape(count, per).max(-1)
    kept = sorted(range(count), key=lambda g: (-best[g], g))[:keep]
    allowed = [e for e in range(len(s)) if e // per in kept]
    return sorted(allowed, key=lambda e: (-c[e], e))[:top]


def expert(x, gate, up, down):
    return down @ (silu(gate @ x) * (up @ x))


def experts(h, w, p, f):
    r = f["router"]
    E, ident = r["experts"], r.get("identity", 0)
    groups = r.get("groups") or dict(count=1, keep=1)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        z = w[p + "router"] @ h[t]
        s = np.exp(z - z.max())
        s = s / s.sum()
        assert len(s) == E + ident
        for e in choose(s, w[p + "correction"], r["top"], groups["count"], groups["keep"]):
            y = h[t] if e >= E else expert(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"])
            out[t] += s[e] * y
    return out


def streams(cfg, w, tokens):
    """The residual stream [T, d] behind every layer, in order."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)].astype(np.float64) * (cfg.get("embedding") or {}).get("scale", 1.0)
    kept, out = {}, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if m.get("kv_from") is None:
            kept[i] = keys_and_values(h, w, p + "mix.", m, eps)
        x = x + attention(h, w, p + "mix.", m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        if L.get("mlp") is not None:
            x = x + experts(norm(x, w[p + "norm2"], eps), w, p + "mlp.", L["mlp"])
        out.append(x)
    return out


def run(cfg, w, tokens):
    return norm(streams(cfg, w, tokens)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
