"""A plain, slow evaluation of the Losarax design in numpy, one function per mechanism, for the tests to compare the
engine with.  Everything runs over a whole sequence at once in float64; there is no cache, no state carried between calls
and no code shared with the package.

``params`` maps tensor names to arrays, ``cfg`` is the parsed config.json.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, -1, keepdims=True) + eps) * w


def layer_norm(x, w, b, eps):
    d = x - np.mean(x, -1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, -1, keepdims=True) + eps) * w + b


def linear(w, x):
    return x @ w.T


def rotate_interleaved(x, positions, dims, base):
    """x[tokens, ..., n]: pairs (2i, 2i+1) of the first `dims` values turn by position * base^(-2i/dims)."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    a = np.asarray(positions, np.float64)[:, None] * f[None, :]
    a = a.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (dims // 2,))
    out = np.array(x, np.float64)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_softmax_attention(q, k, v, scale):
    """q[T, H, n], k[T, H, n], v[T, H, m] -> [T, H, m]; query i sees keys 0..i."""
    s = np.einsum("ihn,jhn->hij", q, k) * scale
    t = q.shape[0]
    s = np.where(np.tril(np.ones((t, t), bool))[None], s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    p /= p.sum(-1, keepdims=True)
    return np.einsum("hij,jhm->ihm", p, v)


def latent_attention(h, w, m, eps):
    """h[T, width], w: the mixer's tensors by short name, m: the mixer's sizes."""
    t, heads, dim, rd, vd, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(t)
    q = linear(w["uq"], rms_norm(linear(w["dq"], h), w["dq.norm"], eps)).reshape(t, heads, dim + rd)
    low = linear(w["dkv"], h)
    c = rms_norm(low[:, :rank], w["dkv.norm"], eps)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    k_rot = rotate_interleaved(low[:, rank:], pos, dims, base)
    q_rot = rotate_interleaved(q[..., dim:], pos, dims, base)
    k_nope = linear(w["uk"], c).reshape(t, heads, dim)
    v = linear(w["uv"], c).reshape(t, heads, vd)
    qq = np.concatenate([q[..., :dim], q_rot], -1)
    kk = np.concatenate([k_nope, np.repeat(k_rot[:, None, :], heads, 1)], -1)
    o = causal_softmax_attention(qq, kk, v, m["scale"]).reshape(t, heads * vd)
    return linear(w["o"], o * sigmoid(linear(w["g"], h)))


def decayed_outer_product_recurrence(q, k, v, decay):
    """q, k [T, H, n], v [T, H, m], decay [H]: S = decay S + k v^T, o = S^T q, token after token from S = 0."""
    t, heads, n = q.shape
    s = np.zeros((heads, n, v.shape[2]))
    o = np.zeros((t, heads, v.shape[2]))
    for i in range(t):
        s = np.asarray(decay, np.float64)[:, None, None] * s + k[i][:, :, None] * v[i][:, None, :]
        o[i] = np.einsum("hnm,hn->hm", s, q[i])
    return o


def lightning(h, w, m, eps):
    t, heads, dim, vd = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(linear(w["q"], h)).reshape(t, heads, dim)
    k = silu(linear(w["k"], h)).reshape(t, heads, dim)
    v = silu(linear(w["v"], h)).reshape(t, heads, vd)
    o = decayed_outer_product_recurrence(q, k, v, m["decay"]).reshape(t, heads * vd)
    return linear(w["o"], rms_norm(o, w["norm"], eps) * sigmoid(linear(w["g"], h)))


def squared_relu_mlp(h, w):
    return linear(w["down"], np.maximum(linear(w["up"], h), 0.0) ** 2)


def hyper_connection(xs, w, norm, sublayer):
    """xs[s, T, width]; w: `in` [s], `mix` [from, to], `out` [s]."""
    y = sublayer(norm(np.einsum("s,stw->tw", w["in"], xs)))
    return np.einsum("st,snw->tnw", w["mix"], xs) + w["out"][:, None, None] * y[None]


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(params, cfg, tokens):
    """(logits[T, vocab], residual stream after every layer run [runs, T, width])."""
    eps, streams = cfg["norm"]["eps"], cfg["streams"]
    p = {k: np.asarray(v, np.float64) for k, v in params.items()}
    under = lambda prefix: {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}  # noqa: E731
    norm_of = lambda name: (lambda x: layer_norm(x, p[name], p[name + ".b"], eps))  # noqa: E731
    x = norm_of("embed.norm")(p["embed"][np.asarray(tokens)])
    xs = np.repeat(x[None], streams, 0)
    mixers = {"lightning": lightning, "latent_attention": latent_attention}
    taps = []
    for i in layer_order(cfg):
        layer = cfg["layers"][i]
        mix = under(f"l{i}.mix.")
        xs = hyper_connection(xs, under(f"l{i}.hc1."), norm_of(f"l{i}.norm1"),
                              lambda h: mixers[layer["type"]](h, mix, layer["mixer"], eps))
        if layer["mlp"] is not None:
            xs = hyper_connection(xs, under(f"l{i}.hc2."), norm_of(f"l{i}.norm2"),
                                  lambda h: squared_relu_mlp(h, under(f"l{i}.mlp.")))
        taps.append(xs.sum(0))
    return linear(p["head"], norm_of("final.norm")(xs.sum(0))), np.stack(taps)
