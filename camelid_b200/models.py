"""The models the engine serves, by architecture name, and one loader for all of them.

A path is a GGUF file (architecture in its metadata) or a folder with config.json (key ``architecture``) and
model.safetensors."""
from __future__ import annotations

import json
from pathlib import Path

from . import gguf, losarax, tokovik


def _load_gguf(path, max_pos, max_seqs, dtype, **kw):
    if dtype not in (None, "quantized"):
        raise ValueError(f"a GGUF model computes on its quantised weights; dtype {dtype!r} does not apply")
    return gguf.load_engine(path, max_pos=max_pos, max_seqs=max_seqs, **kw)


def _load_layered(design):
    def load(path, max_pos, max_seqs, dtype, **kw):
        if not max_pos:
            raise ValueError("this design sets no context length of its own: give max_pos")
        return design.load_engine(path, max_pos, max_seqs, dtype or "bfloat16", **kw)

    return load


ARCHITECTURES = {
    "llama": _load_gguf,  # dense llama shapes and Mixtral shapes
    **{design.ARCHITECTURE: _load_layered(design) for design in (losarax, tokovik)},
}


def architecture_of(path) -> str:
    path = Path(path)
    if path.is_dir():
        config = json.loads((path / "config.json").read_text())
        if "architecture" not in config:
            raise ValueError(f"{path / 'config.json'} names no architecture")
        return config["architecture"]
    g = gguf.GgufFile(path)
    try:
        return g.metadata["general.architecture"]
    finally:
        g.close()


def load_model(path, max_pos: int | None = None, max_seqs: int = 1, dtype: str | None = None, **kw):
    """The engine of the model at `path`: a ``TokenEngine``, whatever its architecture."""
    arch = architecture_of(path)
    if arch not in ARCHITECTURES:
        raise ValueError(f"architecture {arch!r} is not one of {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[arch](path, max_pos, max_seqs, dtype, **kw)
