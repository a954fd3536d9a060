"""A plain, slow evaluation of the Tokovik design in numpy, one function per mechanism, for the tests to compare the
engine with.  Everything runs over a whole sequence at once in float64; there is no cache, no state carried between calls
and no code shared with the package.

``params`` maps tensor names to arrays, ``cfg`` is the parsed config.json.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps) * w


def linear(w, x):
    return x @ w.T


def yarn_frequencies(rot):
    """(frequency of every pair, factor of cosine and sine)."""
    n, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not s:
        return f, 1.0
    place = lambda turns: n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))  # noqa: E731
    lo, hi = max(math.floor(place(s["fast"])), 0), min(math.ceil(place(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotated_halves(x, positions, rot):
    """x[tokens, ..., n]: dimension i turns together with dimension i + dims / 2, i < dims / 2; the rest passes."""
    half = rot["dims"] // 2
    f, m = yarn_frequencies(rot)
    a = np.asarray(positions, np.float64)[:, None] * np.array(f)[None, :]
    a = a.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (half,))
    c, s = m * np.cos(a), m * np.sin(a)
    out = np.array(x, np.float64)
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


def window_attention(q, k, v, scale, window):
    """q[T, H, n], k[T, G, n], v[T, G, m] -> [T, H, m]; query head h reads key head h // (H / G); query i sees the keys
    i - window + 1 .. i."""
    t, heads = q.shape[:2]
    per = heads // k.shape[1]
    i, j = np.arange(t)[:, None], np.arange(t)[None, :]
    seen = (j <= i) & (i - j < window)
    out = np.zeros((t, heads, v.shape[2]))
    for h in range(heads):
        s = np.where(seen, q[:, h] @ k[:, h // per].T * scale, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = p / p.sum(-1, keepdims=True) @ v[:, h // per]
    return out


def attention_branch(h, w, m, eps):
    """h[T, width], w: the branch's tensors by short name, m: its sizes."""
    t, heads, kv, dim, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (linear(w["q"], h) + w["q.b"]).reshape(t, heads, dim)
    k = (linear(w["k"], h) + w["k.b"]).reshape(t, kv, dim)
    v = (linear(w["v"], h) + w["v.b"]).reshape(t, kv, vd)
    pos = np.arange(t)
    q = rotated_halves(rms_norm(q, w["q.norm"], eps), pos, m["rot"])
    k = rotated_halves(rms_norm(k, w["k.norm"], eps), pos, m["rot"])
    return linear(w["o"], window_attention(q, k, v, m["scale"], m["mask"]["size"]).reshape(t, heads * vd))


def channel_decays(h, w, tau):
    return sigmoid(linear(w["a2"], linear(w["a1"], h)) + w["a2.b"]) ** (1.0 / tau)


def gated_recurrence(q, k, v, decay):
    """q, k, decay [T, H, n], v [T, H, m]: S = diag(decay) S + k v^T, o = S^T q, token after token from S = 0."""
    t, heads, n = q.shape
    s = np.zeros((heads, n, v.shape[2]))
    o = np.zeros((t, heads, v.shape[2]))
    for i in range(t):
        s = decay[i][:, :, None] * s + k[i][:, :, None] * v[i][:, None, :]
        o[i] = np.einsum("hnm,hn->hm", s, q[i])
    return o


def gated_branch(h, w, m, eps):
    t, heads, dim, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(w["q"], h).reshape(t, heads, dim) * dim ** -0.5
    k = linear(w["k"], h).reshape(t, heads, dim)
    v = linear(w["v"], h).reshape(t, heads, vd)
    o = gated_recurrence(q, k, v, channel_decays(h, w, m["tau"]).reshape(t, heads, dim))
    o = rms_norm(o, w["norm"], eps).reshape(t, heads * vd)
    return linear(w["o"], o * silu(linear(w["g"], h)))


def under(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def parallel(h, w, m, eps):
    left = attention_branch(h, under(w, "left."), m["left"], eps)
    right = gated_branch(h, under(w, "right."), m["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def swiglu_mlp(h, w):
    return linear(w["down"], silu(linear(w["gate"], h)) * linear(w["up"], h))


def forward(params, cfg, tokens):
    """(logits[T, vocab], residual stream after every layer [layers, T, width])."""
    eps = cfg["norm"]["eps"]
    p = {k: np.asarray(v, np.float64) for k, v in params.items()}
    norm = lambda name, x: rms_norm(x, 1.0 + p[name], eps)  # noqa: E731
    x = p["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    taps = []
    for i, layer in enumerate(cfg["layers"]):
        x = x + norm(f"l{i}.norm1", parallel(x, under(p, f"l{i}.mix."), layer["mixer"], eps))
        if layer["mlp"] is not None:
            x = x + norm(f"l{i}.norm2", swiglu_mlp(x, under(p, f"l{i}.mlp.")))
        taps.append(x)
    return linear(p["head"], norm("final.norm", x)) * cfg["logit_scale"], np.stack(taps)
