"""The Losarax design: config.json of a checkpoint folder to a ``LayeredSpec``, and its loader.

A decoder whose layers mix latent attention and lightning attention (linear attention with a fixed decay per head) in
the order the configuration lists, on a residual of several streams tied by hyper-connections; a range of layers can be
passed several times with the same weights."""
from __future__ import annotations

import json
from pathlib import Path

from .layered import LATENT, LIGHTNING, LayeredEngine, LayerSpec, LayeredSpec
from .safetensors import SafetensorsFile

ARCHITECTURE = "Losarax"


def _mlp_width(i: int, mlp) -> int:
    if mlp is None:
        return 0
    if mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not part of the design")
    return int(mlp["ff"])


def _layer(i: int, entry: dict) -> LayerSpec:
    m, kind = entry["mixer"], entry["type"]
    ff = _mlp_width(i, entry.get("mlp"))
    if kind == "latent_attention":
        rot = m["rot"]
        if int(rot["dims"]) > int(m["rot_dim"]):
            raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions of {m['rot_dim']}")
        return LayerSpec(LATENT, int(m["heads"]), int(m["dim"]), int(m["vdim"]), ff, q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]),
                         rot_dim=int(m["rot_dim"]), rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), scale=float(m["scale"]))
    if kind == "lightning":
        decay = [float(d) for d in m["decay"]]
        if len(decay) != int(m["heads"]):
            raise ValueError(f"layer {i}: {len(decay)} decays for {m['heads']} heads")
        return LayerSpec(LIGHTNING, int(m["heads"]), int(m["dim"]), int(m["vdim"]), ff, decay=decay)
    raise ValueError(f"layer {i}: mixer {kind!r} is not part of the design")


def spec_from_config(config: dict) -> LayeredSpec:
    layers = [_layer(i, e) for i, e in enumerate(config["layers"])]
    loop = config.get("loop")
    span = (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else (0, 0, 1)
    if not (0 <= span[0] <= span[1] <= len(layers) and span[2] >= 1):
        raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
    return LayeredSpec(vocab=int(config["vocab"]), width=int(config["width"]), eps=float(config["norm"]["eps"]), layers=layers,
                       streams=int(config.get("streams", 1)), loop=span)


def load_engine(path, max_pos: int, max_seqs: int = 1, dtype: str = "bfloat16", **kw) -> LayeredEngine:
    """An engine filled from a folder with config.json and model.safetensors."""
    path = Path(path)
    spec = spec_from_config(json.loads((path / "config.json").read_text()))
    f = SafetensorsFile(path / "model.safetensors")
    try:
        eng = LayeredEngine(spec, max_pos, max_seqs, dtype, **kw)
        eng.load(f)
        return eng
    finally:
        f.close()
