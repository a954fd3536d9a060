"""The Tokovik design: config.json of a checkpoint folder to a ``LayeredSpec``, and its loader.

A decoder whose layers run two mixers side by side on the same input, sliding-window attention with grouped heads
(``left``) and gated linear attention (``right``), each normed before they are averaged; norms sit on the sublayers' outputs
only."""
from __future__ import annotations

import json
from pathlib import Path

from .layered import PARALLEL, POST_NORM, SWIGLU, GatedSpec, LayeredEngine, LayeredSpec, LayerSpec, WindowSpec
from .safetensors import SafetensorsFile

ARCHITECTURE = "Tokovik"


def _mlp_width(i: int, mlp) -> int:
    if mlp is None:
        return 0
    if mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not part of the design")
    return int(mlp["ff"])


def _window(i: int, m: dict) -> WindowSpec:
    heads, kv = int(m["heads"]), int(m["kv_heads"])
    if kv < 1 or heads % kv:
        raise ValueError(f"layer {i}: {heads} query heads do not share {kv} key heads evenly")
    size = int(m["mask"]["size"])
    if size < 1:
        raise ValueError(f"layer {i}: a window of {size} tokens")
    rot = m["rot"]
    if int(rot["dims"]) > int(m["dim"]) or int(rot["dims"]) % 2:
        raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions of {m['dim']}")
    s = rot.get("scaling")
    yarn = {} if s is None else {"rot_" + k: float(s[k]) for k in ("factor", "original", "fast", "slow")}
    return WindowSpec(heads, kv, int(m["dim"]), int(m["vdim"]), size, float(m["scale"]), int(rot["dims"]), float(rot["base"]), **yarn)


def _layer(i: int, entry: dict, rank: int) -> LayerSpec:
    if entry["type"] != "parallel":
        raise ValueError(f"layer {i}: mixer {entry['type']!r} is not part of the design")
    r = entry["mixer"]["right"]
    return LayerSpec(PARALLEL, ff=_mlp_width(i, entry.get("mlp")), mlp=SWIGLU, window=_window(i, entry["mixer"]["left"]),
                     gated=GatedSpec(int(r["heads"]), int(r["dim"]), int(r["vdim"]), rank, float(r["tau"])))


def spec_from_config(config: dict, shape) -> LayeredSpec:
    """shape(name): the shape of a tensor of the checkpoint (the rank of the decays is given there only)."""
    layers = [_layer(i, e, int(shape(f"l{i}.mix.right.a1")[0])) for i, e in enumerate(config["layers"])]
    return LayeredSpec(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]), layers=layers, residual=POST_NORM,
                       embed_scale=float(config["embedding"]["scale"]), logit_scale=float(config["logit_scale"]))


def load_engine(path, max_pos: int, max_seqs: int = 1, dtype: str = "bfloat16", **kw) -> LayeredEngine:
    """An engine filled from a folder with config.json and model.safetensors."""
    path = Path(path)
    f = SafetensorsFile(path / "model.safetensors")
    try:
        eng = LayeredEngine(spec_from_config(json.loads((path / "config.json").read_text()), f.shape), max_pos, max_seqs, dtype, **kw)
        eng.load(f)
        return eng
    finally:
        f.close()
