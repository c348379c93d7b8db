"""Model registry: which configuration class a ``config.json`` belongs to, and how its weights load.

``read_config`` looks the document's ``architecture`` up in ``REGISTRY``; a document without a registered
one is a Llama/Qwen2 configuration (``UnifiedConfig``), whose weights are a palettized ``.cimage``.  A
model described layer by layer (``LayeredConfig``) lists its layers, each with a mixer, the mixer's sizes
and a feed-forward; mixers are looked up in ``MIXERS``, so another design reuses them by listing them.
"""
from __future__ import annotations

import ctypes as C
import glob
import json
import math
import os
from dataclasses import dataclass, field
from typing import List, Optional, Tuple

import numpy as np

from ._lib import LayerConfig, LayeredModelConfig
from .backend import CudaBackend, PrismEngine, model_config
from .graph import UnifiedConfig

DTYPES = {"bfloat16": 0, "float32": 1}
MIXER_LIGHTNING, MIXER_LATENT_ATTENTION = 0, 1


def yarn_frequencies(base: float, dims: int, scaling: Optional[dict]) -> Tuple[np.ndarray, float]:
    """Angle per position of the ``dims / 2`` pairs of a rotate-half rotation, and the factor of cos and sin.

    With ``scaling`` (YaRN) the pairs that turn at least ``fast`` times over the ``original`` context keep their
    frequency, those that turn at most ``slow`` times are slowed down ``factor`` times, the ones between are
    blended linearly by pair index."""
    pairs = np.arange(dims // 2, dtype=np.float64)
    freq = np.power(float(base), -2.0 * pairs / dims)
    if not scaling:
        return freq, 1.0
    factor, log_base = float(scaling["factor"]), math.log(base)
    pair_of = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * log_base)  # noqa: E731
    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    ramp = np.clip((pairs - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq * (1.0 - ramp) + freq / factor * ramp, 0.1 * math.log(factor) + 1.0


@dataclass
class LayerSpec:
    """One layer as the engine takes it (``prism_layer_config``)."""

    mixer: int
    heads: int
    dim: int
    vdim: int
    ff: int = 0
    decay: Optional[np.ndarray] = None
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_freq: Optional[np.ndarray] = None
    rot_mul: float = 1.0
    scale: float = 1.0
    window: int = 0


def _lightning(m: dict) -> dict:
    decay = np.asarray(m["decay"], np.float32).reshape(-1)
    if decay.size != m["heads"]:
        raise ValueError(f"lightning: {decay.size} decays for {m['heads']} heads")
    return dict(mixer=MIXER_LIGHTNING, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=decay)


def _latent_attention(m: dict) -> dict:
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    if rot["dims"] % 2 or rot["dims"] > m["rot_dim"]:
        raise ValueError(f"latent_attention: cannot rotate {rot['dims']} of {m['rot_dim']} dimensions")
    freq, mul = yarn_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
    return dict(mixer=MIXER_LATENT_ATTENTION, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], q_rank=m["q_rank"],
                kv_rank=m["kv_rank"], rot_dim=m["rot_dim"], rot_freq=freq.astype(np.float32), rot_mul=mul, scale=m["scale"],
                window=(m.get("mask") or {}).get("size", 0))


MIXERS = {"lightning": _lightning, "latent_attention": _latent_attention}


@dataclass
class LayeredConfig:
    """A decoder described layer by layer."""

    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    layers: List[LayerSpec] = field(default_factory=list)

    @classmethod
    def from_dict(cls, raw: dict) -> "LayeredConfig":
        layers = []
        for i, ly in enumerate(raw["layers"]):
            if ly["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {ly['type']!r} (known: {', '.join(sorted(MIXERS))})")
            mlp = ly.get("mlp")
            if mlp and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            layers.append(LayerSpec(ff=mlp["ff"] if mlp else 0, **MIXERS[ly["type"]](ly["mixer"])))
        return cls(vocab=raw["vocab"], width=raw["width"], norm_eps=raw["norm"]["eps"], residual_mult=raw["residual_mult"],
                   logit_scale=raw["logit_scale"], layers=layers)

    def to_c(self, dtype: str, max_seq: int, max_batch: int):
        """``(prism_layered_config, prism_layer_config[], arrays to keep alive during the call)``."""
        if dtype not in DTYPES:
            raise ValueError(f"dtype must be one of {', '.join(DTYPES)}")
        keep = []

        def floats(a):
            if a is None or not len(a):
                return None
            buf = (C.c_float * len(a))(*[float(x) for x in a])
            keep.append(buf)
            return C.cast(buf, C.POINTER(C.c_float))

        arr = (LayerConfig * len(self.layers))()
        for c, s in zip(arr, self.layers):
            c.mixer, c.heads, c.dim, c.vdim, c.ff = s.mixer, s.heads, s.dim, s.vdim, s.ff
            c.q_rank, c.kv_rank, c.rot_dim = s.q_rank, s.kv_rank, s.rot_dim
            c.rot_mul, c.scale, c.window = s.rot_mul, s.scale, s.window
            c.decay = floats(s.decay)
            c.rot_pairs = 0 if s.rot_freq is None else len(s.rot_freq)
            c.rot_freq = floats(s.rot_freq)
        mc = LayeredModelConfig(self.vocab, self.width, len(self.layers), self.norm_eps, self.residual_mult, self.logit_scale,
                                DTYPES[dtype], max_seq, max_batch)
        return mc, arr, keep

    def tensor_shapes(self) -> dict:
        """Checkpoint name -> shape of every tensor the model needs."""
        out = {"embed": (self.vocab, self.width)}
        for i, s in enumerate(self.layers):
            p, hv, d = f"l{i}.", s.heads * s.vdim, self.width
            out[p + "norm1"] = (d,)
            if s.mixer == MIXER_LIGHTNING:
                out.update({p + "mix.q": (s.heads * s.dim, d), p + "mix.k": (s.heads * s.dim, d), p + "mix.v": (hv, d),
                            p + "mix.g": (hv, d), p + "mix.norm": (hv,), p + "mix.o": (d, hv)})
            else:
                out.update({p + "mix.dq": (s.q_rank, d), p + "mix.dq.norm": (s.q_rank,),
                            p + "mix.uq": (s.heads * (s.dim + s.rot_dim), s.q_rank), p + "mix.dkv": (s.kv_rank + s.rot_dim, d),
                            p + "mix.dkv.norm": (s.kv_rank,), p + "mix.uk": (s.heads * s.dim, s.kv_rank),
                            p + "mix.uv": (hv, s.kv_rank), p + "mix.g": (hv, d), p + "mix.o": (d, hv)})
            if s.ff:
                out.update({p + "mlp.up": (s.ff, d), p + "mlp.up.b": (s.ff,), p + "mlp.down": (d, s.ff), p + "mlp.down.b": (d,)})
        out["final.norm"] = (self.width,)
        out["head"] = (self.vocab, self.width)
        return out


# architecture named by config.json -> configuration class
REGISTRY = {"Mefipel": LayeredConfig}


def read_config(path: str):
    """Configuration of the model in a folder (or of one ``config.json``)."""
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        raw = json.load(f)
    return REGISTRY.get(raw.get("architecture"), UnifiedConfig).from_dict(raw)


def load_model(backend: CudaBackend, folder: str, dtype: str = "bfloat16", max_seq: int = 4096, max_batch: int = 1) -> PrismEngine:
    """Engine of the model in ``folder``: config.json with ``*.safetensors`` (layered) or one ``.cimage``
    (palettized; its arithmetic is fixed, ``dtype`` must stay "bfloat16")."""
    cfg = read_config(folder)
    if isinstance(cfg, LayeredConfig):
        eng = PrismEngine(backend, cfg, dtype=dtype, max_seq=max_seq, max_batch=max_batch)
        try:
            eng.load_safetensors(os.path.join(folder, "model.safetensors"))
        except Exception:
            eng.close()
            raise
        return eng
    if dtype != "bfloat16":
        raise ValueError("palettized models have no 32-bit form")
    images = sorted(glob.glob(os.path.join(folder, "*.cimage")))
    if len(images) != 1:
        raise FileNotFoundError(f"{folder}: expected one .cimage, found {len(images)}")
    mc = model_config(cfg.num_layers, cfg.hidden_size, cfg.num_heads, cfg.num_kv_heads, cfg.head_dim, cfg.intermediate_size,
                      cfg.vocab_size, cfg.norm_eps, cfg.rope_theta, cfg.tie_word_embeddings, max_seq=max_seq, max_batch=max_batch)
    return PrismEngine.load(backend, images[0], mc, cfg.key_prefix)
