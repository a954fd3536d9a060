"""Small random Losarax models for the tests: configurations, weights rounded to bfloat16, checkpoint folders."""
from __future__ import annotations

import numpy as np

from camelid_b200.safetensors import from_bf16, to_bf16

import plain_losarax as pl
from layered_helpers import LIMIT, rel_rms, tokens, write_folder  # noqa: F401


def latent(heads=3, dim=24, vdim=16, q_rank=40, kv_rank=56, rot_dim=8, dims=None, base=10000.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot_dim,
                      "rot": {"base": base, "dims": rot_dim if dims is None else dims}, "scale": scale or (dim + rot_dim) ** -0.5},
            "mlp": None}


def lightning(heads=3, dim=24, vdim=16, decay=None):
    return {"type": "lightning",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** -(2 + i) for i in range(heads)]}, "mlp": None}


def with_mlp(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def config(layers, width=72, vocab=203, streams=2, loop=None, eps=1e-5):
    return {"architecture": "Losarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers,
            "loop": loop or {"start": 0, "stop": len(layers), "times": 1}}


# name -> configuration; together they leave no size equal to another, cross every limit of the kernels' fast forms, and
# put the feed-forward, the loop and the mixers in different places
CASES = {
    "latent": config([with_mlp(latent(), 90)]),
    "lightning": config([lightning()]),
    "both_mlp_on_lightning": config([latent(heads=5, vdim=40), with_mlp(lightning(heads=2, dim=40, vdim=24), 50), latent(scale=0.3)], streams=3,
                                    loop={"start": 1, "stop": 3, "times": 3}),
    "one_stream_no_loop": dict(config([with_mlp(lightning(vdim=33), 61), with_mlp(latent(heads=9, dim=8, vdim=8, base=100.0), 130)], streams=1), loop=None),
    "odd_sizes": config([with_mlp(latent(heads=2, dim=21, vdim=13, q_rank=37, kv_rank=51, rot_dim=10, dims=6), 77),
                         with_mlp(lightning(heads=3, dim=19, vdim=11, decay=[0.0, 0.5, 1.0]), 45)], width=91, vocab=157, streams=5, eps=1e-3),
    "wide_latent": config([latent(heads=17, dim=48, vdim=72, q_rank=160, kv_rank=528, rot_dim=32, base=500.0),
                           lightning(heads=2, dim=136, vdim=72)], width=264, vocab=301, streams=4),
    "long_keys": config([lightning(heads=1, dim=300, vdim=40, decay=[0.97]), lightning(heads=4, dim=72, vdim=130)], width=120, streams=2),
}


def tensor_shapes(cfg) -> dict:
    w, s, out = cfg["width"], cfg["streams"], {}

    def norm(name):
        out[name] = out[name + ".b"] = (w,)

    out["embed"] = (cfg["vocab"], w)
    norm("embed.norm")
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        h, d, v = m["heads"], m["dim"], m["vdim"]
        norm(f"l{i}.norm1")
        if layer["type"] == "latent_attention":
            r = m["rot_dim"]
            out.update({p + "dq": (m["q_rank"], w), p + "dq.norm": (m["q_rank"],), p + "uq": (h * (d + r), m["q_rank"]), p + "dkv": (m["kv_rank"] + r, w),
                        p + "dkv.norm": (m["kv_rank"],), p + "uk": (h * d, m["kv_rank"]), p + "uv": (h * v, m["kv_rank"])})
        else:
            out.update({p + "q": (h * d, w), p + "k": (h * d, w), p + "v": (h * v, w), p + "norm": (h * v,)})
        out.update({p + "g": (h * v, w), p + "o": (w, h * v)})
        for q in (1, 2) if layer["mlp"] else (1,):
            out.update({f"l{i}.hc{q}.in": (s,), f"l{i}.hc{q}.out": (s,), f"l{i}.hc{q}.mix": (s, s)})
        if layer["mlp"]:
            norm(f"l{i}.norm2")
            out.update({f"l{i}.mlp.up": (layer["mlp"]["ff"], w), f"l{i}.mlp.down": (w, layer["mlp"]["ff"])})
    norm("final.norm")
    out["head"] = (cfg["vocab"], w)
    return out


def random_params(cfg, seed: int) -> dict:
    """f32 arrays whose values are bfloat16 numbers.  Queries and keys are scaled up so that single keys stand out."""
    rng = np.random.default_rng(seed)
    s, out = cfg["streams"], {}
    for name, shape in tensor_shapes(cfg).items():
        z = rng.standard_normal(shape)
        if name.endswith((".b",)):
            z *= 0.3
        elif name.endswith(".in"):
            z = 1.0 / s + 0.3 * z
        elif name.endswith(".out"):
            z = 1.0 + 0.4 * z
        elif name.endswith(".hc1.mix") or name.endswith(".hc2.mix"):
            z = np.eye(s) * 0.9 + 0.2 * z
        elif "norm" in name.rsplit(".", 1)[-1] or name.endswith(("norm1", "norm2")):
            z = 1.0 + 0.3 * z
        elif name != "embed":
            z /= np.sqrt(shape[1])
            if name.endswith((".uq", ".uk")):
                z *= 1.8
        out[name] = from_bf16(to_bf16(z)).reshape(shape)
    return out


def engine(cfg, params, max_pos, max_seqs=1, dtype="float32", **kw):
    from camelid_b200 import losarax
    from camelid_b200.layered import LayeredEngine

    eng = LayeredEngine(losarax.spec_from_config(cfg), max_pos, max_seqs, dtype, **kw)
    for name in eng.tensors():
        eng.set_tensor(name, to_bf16(params[name]))
    return eng


plain = pl.forward
