"""Small random Tokovik models for the tests: configurations, weights rounded to bfloat16, engines."""
from __future__ import annotations

import numpy as np

from camelid_b200.safetensors import from_bf16, to_bf16

import plain_tokovik as pt

YARN = {"factor": 4.0, "original": 96, "fast": 6.0, "slow": 0.5}


def left(heads=6, kv_heads=2, dim=24, vdim=16, window=9, dims=8, base=1000.0, scaling=YARN, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
            "rot": {"base": base, "dims": dims, "scaling": scaling}, "scale": scale or 1.5 * dim ** -0.5}


def right(heads=3, dim=24, vdim=16, tau=16.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def layer(l=None, r=None, ff=50):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right()}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=203, eps=1e-5, embed=3.7, logit=0.8, rank=11):
    """rank: of the decays; a number, or one per layer.  Not part of the checkpoint's configuration."""
    return {"architecture": "Tokovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed}, "logit_scale": logit,
            "layers": layers, "ranks": rank if isinstance(rank, list) else [rank] * len(layers)}


# name -> configuration; together they leave no size equal to another, cross every limit of the kernels' fast forms, and mix
# sizes, windows and feed-forwards within a model
CASES = {
    "one_layer": config([layer()]),
    "unequal_layers": config([layer(left(heads=5, kv_heads=1, dim=40, vdim=56, window=37, dims=16), right(heads=2, dim=40, vdim=72), 90),
                              layer(left(heads=4, kv_heads=4, window=1, dims=24, scaling=None), right(heads=5, dim=16, vdim=8, tau=3.0), 0),
                              layer(left(heads=8, kv_heads=2, dim=16, vdim=24, window=64, dims=4, base=50000.0), right(heads=1, dim=56, vdim=40), 33)],
                             rank=[11, 3, 24]),
    "odd_sizes": config([layer(left(heads=3, kv_heads=1, dim=21, vdim=13, window=33, dims=6), right(heads=3, dim=19, vdim=11, tau=1.0), 45),
                         layer(left(heads=2, kv_heads=2, dim=27, vdim=9, window=2, dims=26, base=31.0), right(heads=2, dim=33, vdim=35), 0)],
                        width=91, vocab=157, eps=1e-3, rank=5),
    "many_heads_per_key": config([layer(left(heads=34, kv_heads=2, dim=32, vdim=8, window=70))], width=64, embed=1.0, logit=1.0),
    "wide": config([layer(left(heads=4, kv_heads=2, dim=136, vdim=72, window=1000, dims=32), right(heads=2, dim=136, vdim=72), 200)], width=264, vocab=301),
    "beyond_the_fast_forms": config([layer(left(heads=2, kv_heads=1, dim=40, vdim=264, window=21), right(heads=1, dim=300, vdim=40), 0)], width=120),
}


def tensor_shapes(cfg) -> dict:
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w)}
    for i, e in enumerate(cfg["layers"]):
        p, l, r = f"l{i}.", e["mixer"]["left"], e["mixer"]["right"]
        out[p + "norm1"] = (w,)
        for name, rows in (("q", l["heads"] * l["dim"]), ("k", l["kv_heads"] * l["dim"]), ("v", l["kv_heads"] * l["vdim"])):
            out[p + "mix.left." + name] = (rows, w)
            out[p + "mix.left." + name + ".b"] = (rows,)
        out.update({p + "mix.left.q.norm": (l["dim"],), p + "mix.left.k.norm": (l["dim"],), p + "mix.left.o": (w, l["heads"] * l["vdim"])})
        gk, gv, rank = r["heads"] * r["dim"], r["heads"] * r["vdim"], cfg["ranks"][i]
        for name, rows in (("q", gk), ("k", gk), ("v", gv), ("g", gv), ("a1", rank)):
            out[p + "mix.right." + name] = (rows, w)
        out.update({p + "mix.right.a2": (gk, rank), p + "mix.right.a2.b": (gk,), p + "mix.right.norm": (r["vdim"],), p + "mix.right.o": (w, gv),
                    p + "mix.left.out": (w,), p + "mix.right.out": (w,)})
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            out.update({p + "norm2": (w,), p + "mlp.gate": (ff, w), p + "mlp.up": (ff, w), p + "mlp.down": (w, ff)})
    out.update({"final.norm": (w,), "head": (cfg["vocab"], w)})
    return out


def random_params(cfg, seed: int) -> dict:
    """f32 arrays whose values are bfloat16 numbers.  The decays of a layer reach from a fraction of a token to hundreds."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        if name.endswith("a2.b"):
            z = 2.0 + 3.0 * z
        elif name.endswith(".b"):
            z *= 0.4
        elif name.endswith(("norm1", "norm2", "final.norm")):
            z *= 0.3  # stored around zero
        elif len(shape) == 1:
            z = 1.0 + 0.3 * z
        elif name != "embed":
            z /= np.sqrt(shape[1])
        out[name] = z
    return rounded(out)


def rounded(params) -> dict:
    return {k: from_bf16(to_bf16(v)).reshape(v.shape) for k, v in params.items()}


def spec(cfg):
    from camelid_b200 import tokovik

    shapes = tensor_shapes(cfg)
    return tokovik.spec_from_config(cfg, lambda name: shapes[name])


def engine(cfg, params, max_pos, max_seqs=1, dtype="float32", **kw):
    from camelid_b200.layered import LayeredEngine

    eng = LayeredEngine(spec(cfg), max_pos, max_seqs, dtype, **kw)
    for name in eng.tensors():
        eng.set_tensor(name, to_bf16(params[name]))
    return eng


plain = pt.forward
