"""Vofezen, written out plainly: float64 numpy over a whole sequence, one function per mechanism.

Shares no code with the package.  A model is a dict `cfg` (the nested form of its config.json) and a dict of
float64 arrays by tensor name; `run(cfg, tensors, tokens)` returns the logits of every position, `streams(...)` the
residual stream behind every layer.

Notation: T positions, d width, H query heads, G key/value heads, dk key size, dv value size, eps the norm's epsilon.
  N(x, w)          x / sqrt(mean(x^2) + eps) * (1 + w)
  layer            x <- x + N_1b(mixer(N_1(x)));  x <- x + N_2b(ff(N_2(x)))
  attention        q, k = W h, rotated on their first r elements (i with i + r/2); v = W_v h, in every mixing layer but the
                   first (1 - l) v + l v_first; softmax((q . k) scale) over j <= i with exp(sink_h) once more in the
                   denominator; heads side by side; W_o
  latent attention cq = R(W_dq h) w_q; q_h = W_uq,h cq = [plain | rotated]; [c' | kr] = W_dkv h; c = R(c') w_c; k_h =
                   W_uk,h c, v_h = W_uv,h c; scale (q_plain . k + rot(q_rotated) . rot(kr)); softmax over j <= i; W_o
  feed-forward     W_down max(W_up h + b, 0)^2 + b'
"""
import math

import numpy as np


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def rotary_frequencies(dims, base, scaling=None):
    """(f_i for i < dims/2, magnitude of cos and sin); scaling {factor, original, fast, slow}."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, freqs, mag=1.0):
    """x [T, heads, size]: the first 2 len(freqs) elements of each head, element i with i + len(freqs).  The angle is a
    float32 product (positions and angles are 32-bit in the design); the rest is float64."""
    n = len(freqs)
    if n == 0:
        return x
    a = (np.asarray(positions, dtype=np.float32)[:, None] * np.asarray(freqs, dtype=np.float32)[None, :]).astype(np.float64)
    c, s = (mag * np.cos(a))[:, None, :], (mag * np.sin(a))[:, None, :]
    out = x.copy()
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def softmax_with_sink(s, sink=None):
    """s [..., keys] (minus infinity: not visible); sink: a number that joins the denominator as exp(sink)."""
    m = s.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    total = e.sum(-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - m)
    return e / total


def attend(q, k, v, scale, sinks=None):
    """q [T, H, dk], k [T, G, dk], v [T, G, dv], positions 0..T-1 -> [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    hidden = np.triu(np.ones((T, T), dtype=bool), 1)
    out = np.empty((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s[hidden] = -np.inf
        out[:, h] = softmax_with_sink(s, None if sinks is None else sinks[h]) @ v[:, g]
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, p, m, v_first):
    """h [T, d] -> (result, this layer's own values before mixing).  v_first None: nothing to mix with."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dk)
    k = (h @ w[p + "k"].T).reshape(T, G, dk)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        f, mag = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate(q, np.arange(T), f, mag), rotate(k, np.arange(T), f, mag)
    own = v
    if m.get("v_mix") and v_first is not None:
        v = mix_values(v, v_first.reshape(v.shape), float(w[p + "vmix"]))
    o = attend(q, k, v, m["scale"], w[p + "sink"])
    return o.reshape(T, H * dv) @ w[p + "o"].T, own


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = unit_rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, dn + dr)
    z = h @ w[p + "dkv"].T
    c = unit_rms(z[:, :rk], eps) * w[p + "dkv.norm"]
    qn, qr, kr = q[..., :dn], q[..., dn:], z[:, rk:].reshape(T, 1, dr)
    rot = m.get("rot")
    if rot and rot["dims"]:
        f, mag = rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        qr, kr = rotate(qr, np.arange(T), f, mag), rotate(kr, np.arange(T), f, mag)
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, dn), np.repeat(kr, H, 1)], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    o = attend(np.concatenate([qn, qr], -1), k, v, m["scale"])
    return o.reshape(T, H * dv) @ w[p + "o"].T


def feed_forward(h, w, p):
    return np.maximum(h @ w[p + "up"].T + w[p + "up.b"], 0.0) ** 2 @ w[p + "down"].T + w[p + "down.b"]


def streams(cfg, w, tokens):
    """The residual stream [T, d] behind every layer, in order."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)].astype(np.float64)
    v_first, out = None, []
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if L["type"] == "attention":
            y, own = attention(h, w, p + "mix.", m, v_first)
            if m.get("v_mix") and v_first is None:
                v_first = own
        else:
            y = latent_attention(h, w, p + "mix.", m, eps)
        x = x + norm(y, w[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
        out.append(x)
    return out


def run(cfg, w, tokens):
    x = streams(cfg, w, tokens)[-1]
    return norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
