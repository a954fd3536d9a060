"""What the GPU tests of layered designs share: feeding portions, cutting prompts, comparing rows."""
from __future__ import annotations

import json

import numpy as np

from camelid_b200.safetensors import to_bf16, write_safetensors

DTYPES = ["float32", "bfloat16"]
# largest row error allowed, relative to the reference's rms
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


def feed(eng, seq, tokens, parts, taps=0):
    """The tokens in portions of the given sizes; logits of every token (and the residual after every layer run)."""
    at, logits, stream = 0, [], []
    for k in parts:
        r = eng.extend(seq, tokens[at:at + k], at, list(range(k)), taps=taps)
        logits.append(r[1])
        if taps:
            stream.append(r[2])
        at += k
    assert at == len(tokens)
    return (np.concatenate(logits), np.concatenate(stream, 1)) if taps else np.concatenate(logits)


def cut(n, sizes):
    """n cut into portions of the sizes, over and over."""
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out


def rel_rms(got, ref):
    """Per row: rms of the difference over the rms of the whole reference."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def check(got, ref, dtype, what, factor=1.0):
    e = rel_rms(got, ref)
    assert np.isfinite(got).all() and e.max() <= factor * LIMIT[dtype], (what, float(e.max()), int(np.unravel_index(e.argmax(), e.shape)[-1]))


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def write_folder(path, cfg, params):
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", {k: to_bf16(v).reshape(v.shape) for k, v in params.items()})
    return path


def greedy_follows(plain, params, cfg, prompt, out, dtype):
    """Every generated token is the plain evaluation's best one, or as good within the tolerance."""
    toks = list(prompt)
    for t in out:
        ref = plain(params, cfg, toks)[0][-1]
        assert ref[t] >= ref.max() - 4 * LIMIT[dtype] * np.sqrt((ref ** 2).mean()), (len(toks), t)
        toks.append(int(t))
