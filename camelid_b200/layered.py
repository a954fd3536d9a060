"""Engines of layered designs: models described layer by layer (``LayeredSpec``), with named bfloat16 tensors."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np

from ._lib import GatedDesc, LayerDesc, LayeredConfig, WindowDesc, check, lib
from .engine import BF16, F32, TokenEngine, _np_ptr

LATENT, LIGHTNING, PARALLEL = 1, 2, 3
RELU2, SWIGLU = 0, 1
STREAMS, POST_NORM = 0, 1
DTYPES = {"bfloat16": BF16, "float32": F32}


@dataclass
class WindowSpec:
    """Attention with grouped heads: a query sees ``window`` tokens, itself included (0: every earlier one); the first
    ``rot_dims`` dimensions turn, with YaRN-scaled frequencies if ``rot_factor`` is given."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 0.0
    rot_factor: float = 0.0
    rot_original: float = 0.0
    rot_fast: float = 0.0
    rot_slow: float = 0.0


@dataclass
class GatedSpec:
    """Linear attention with a decay per key channel, from a projection of rank ``rank``."""
    heads: int
    dim: int
    vdim: int
    rank: int
    tau: float


@dataclass
class LayerSpec:
    """One layer: a mixer and, unless ``ff`` is 0, a feed-forward of that width (``mlp``: its kind).  A parallel layer's
    sizes are in ``window`` and ``gated``."""
    type: int
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    ff: int = 0
    mlp: int = RELU2
    window: WindowSpec | None = None
    gated: GatedSpec | None = None
    # latent attention
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_dims: int = 0
    rot_base: float = 0.0
    scale: float = 1.0
    # lightning attention: one decay per head
    decay: list = field(default_factory=list)


@dataclass
class LayeredSpec:
    vocab: int
    width: int
    eps: float
    layers: list
    streams: int = 1
    loop: tuple = (0, 0, 1)  # layers start .. stop-1 run `times` times in a row
    residual: int = STREAMS
    embed_scale: float = 1.0
    logit_scale: float = 1.0

    @property
    def runs(self) -> list:
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, len(self.layers)))


@dataclass
class LayeredRuntime:
    """What the token-driven calls look up (the fields every engine's cfg has)."""
    vocab: int
    hidden: int
    max_pos: int
    max_seqs: int


class LayeredEngine(TokenEngine):
    """A layered design on the device.  Sequences live in slots 0..max_seqs-1; a slot's caches and states belong together,
    so a call starts a sequence at position 0 or continues it where it ends (``filled``)."""

    def __init__(self, spec: LayeredSpec, max_pos: int, max_seqs: int = 1, dtype: str = "bfloat16", device: int = -1, flags: int = 0,
                 portion: int = 0):
        """portion: most rows of one step of a prompt (0: the library's own number); windowed caches are sized by it."""
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r} is not one of {sorted(DTYPES)}")
        self.spec = spec
        self.cfg = LayeredRuntime(spec.vocab, spec.width, max_pos, max(1, max_seqs))
        arr = (LayerDesc * len(spec.layers))()
        keep = []
        for d, s in zip(arr, spec.layers):
            for name in ("type", "heads", "dim", "vdim", "q_rank", "kv_rank", "rot_dim", "rot_dims", "ff", "mlp", "scale", "rot_base"):
                setattr(d, name, getattr(s, name))
            if s.type == PARALLEL:
                d.window, d.gated = WindowDesc(**vars(s.window)), GatedDesc(**vars(s.gated))
            if s.type == LIGHTNING:
                if len(s.decay) != s.heads:
                    raise ValueError(f"{len(s.decay)} decays for {s.heads} heads")
                dec = np.ascontiguousarray(s.decay, np.float32)
                keep.append(dec)
                d.decay = dec.ctypes.data_as(C.POINTER(C.c_float))
        c = LayeredConfig(n_layers=len(spec.layers), loop_start=spec.loop[0], loop_stop=spec.loop[1], loop_times=spec.loop[2], streams=spec.streams,
                          width=spec.width, vocab=spec.vocab, max_pos=max_pos, max_seqs=self.cfg.max_seqs, dtype=DTYPES[dtype], device=device,
                          flags=flags, residual=spec.residual, portion=portion, eps=spec.eps, embed_scale=spec.embed_scale,
                          logit_scale=spec.logit_scale, layers=arr)
        h = C.c_void_p()
        check(lib().cmld_engine_create_layered(C.byref(c), C.byref(h)))
        self._h = h.value

    def tensors(self) -> dict:
        """name -> shape of every tensor the model needs ((rows, cols) for matrices, (count,) for vectors)."""
        out = {}
        name, rows, cols = C.c_char_p(), C.c_int64(), C.c_int64()
        for i in range(lib().cmld_engine_named_count(self._h)):
            check(lib().cmld_engine_named_info(self._h, i, C.byref(name), C.byref(rows), C.byref(cols)))
            out[name.value.decode()] = (rows.value, cols.value) if rows.value else (cols.value,)
        return out

    def set_tensor(self, name: str, values: np.ndarray):
        """uint16 = bfloat16 patterns; float32 for vectors."""
        a = np.ascontiguousarray(values)
        if a.dtype not in (np.dtype(np.uint16), np.dtype(np.float32)):
            raise ValueError(f"tensor {name}: {a.dtype} is neither bfloat16 patterns (uint16) nor float32")
        check(lib().cmld_engine_set_named(self._h, name.encode(), BF16 if a.dtype == np.uint16 else F32, _np_ptr(a), a.nbytes))

    def synth_tensor(self, name: str, seed: int, stream: int, mean: float, sigma: float):
        check(lib().cmld_engine_synth_named(self._h, name.encode(), seed, stream, mean, sigma))

    def load(self, file):
        """Every tensor from a ``safetensors.SafetensorsFile``; names and shapes must agree."""
        need = self.tensors()
        have = set(file.names())
        missing, extra = sorted(set(need) - have), sorted(have - set(need))
        if missing or extra:
            raise ValueError(f"checkpoint and model differ: missing {missing[:5]}, not used {extra[:5]}")
        for name, shape in need.items():
            got = file.shape(name)
            if (got != shape) if len(shape) == 2 else (int(np.prod(got)) != shape[0]):
                raise ValueError(f"tensor {name} has shape {got}, the configuration asks for {shape}")
            if file.dtype(name) != "BF16":
                raise ValueError(f"tensor {name} is {file.dtype(name)}, expected BF16")
            self.set_tensor(name, file.data(name))

    def filled(self, slot: int = 0) -> int:
        n = C.c_int64(0)
        check(lib().cmld_engine_slot_filled(self._h, slot, C.byref(n)))
        return int(n.value)

    def layer_runs(self) -> int:
        return len(self.spec.runs)
