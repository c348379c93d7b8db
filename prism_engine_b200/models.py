"""Model registry: which configuration class a ``config.json`` belongs to, and how its weights load.

``read_config`` looks the document's ``architecture`` up in ``REGISTRY``; a document without a registered
one is a Llama/Qwen2 configuration (``UnifiedConfig``), whose weights are a palettized ``.cimage``.  A
model described layer by layer (``LayeredConfig``) lists its layers, each with a mixer, the mixer's sizes
and a feed-forward; mixers are looked up in ``MIXERS``, feed-forwards in ``FEED_FORWARDS``, so another design
reuses them by listing them.  What is common to the layers of a design -- how sublayers follow one another,
how norm weights are stored, what is done around a sublayer -- are fields of the configuration, filled in by
the design's entry of ``REGISTRY``.
"""
from __future__ import annotations

import ctypes as C
import glob
import json
import math
import os
from dataclasses import dataclass, field, fields
from typing import List, Optional, Tuple

import numpy as np

from ._lib import LayerConfig, LayeredModelConfig
from .backend import CudaBackend, PrismEngine, model_config
from .graph import UnifiedConfig

DTYPES = {"bfloat16": 0, "float32": 1}
MIXER_LIGHTNING, MIXER_LATENT_ATTENTION, MIXER_ATTENTION, MIXER_GATED_DELTA, MIXER_PAIR = range(5)
ARRANGE_PARALLEL, ARRANGE_SEQUENTIAL = range(2)


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
    """One layer as the engine takes it (``prism_layer_config``); also one mixer of a pair."""

    mixer: int
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    decay: Optional[np.ndarray] = None
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    rot_freq: Optional[np.ndarray] = None
    rot_mul: float = 1.0
    scale: float = 1.0
    window: int = 0
    kv_heads: int = 0
    conv: int = 0
    left: Optional["LayerSpec"] = None
    right: Optional["LayerSpec"] = None
    ff: int = 0
    experts: int = 0
    top: int = 0
    expert_groups: int = 0
    groups_keep: int = 0


def _window(m: dict) -> int:
    return (m.get("mask") or {}).get("size") or 0


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
                window=_window(m))


def _shared_heads(kind: str, m: dict) -> dict:
    if m["kv_heads"] < 1 or m["heads"] % m["kv_heads"]:
        raise ValueError(f"{kind}: {m['heads']} heads cannot share {m['kv_heads']}")
    return dict(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"])


def _attention(m: dict) -> dict:
    return dict(mixer=MIXER_ATTENTION, scale=m["scale"], window=_window(m), **_shared_heads("attention", m))


def _gated_delta(m: dict) -> dict:
    return dict(mixer=MIXER_GATED_DELTA, conv=m["conv"], **_shared_heads("gated_delta", m))


def _parallel(m: dict) -> dict:
    return dict(mixer=MIXER_PAIR, left=LayerSpec(**_attention(m["left"])), right=LayerSpec(**_gated_delta(m["right"])))


MIXERS = {"lightning": _lightning, "latent_attention": _latent_attention, "attention": _attention, "gated_delta": _gated_delta,
          "parallel": _parallel}


def _dense(m: dict) -> dict:
    return dict(ff=m["ff"])


def _moe(m: dict) -> dict:
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    if r["experts"] % groups["count"] or not 1 <= groups["keep"] <= groups["count"]:
        raise ValueError(f"moe: {r['experts']} experts do not form {groups['count']} equal groups of which {groups['keep']} are kept")
    if not 1 <= r["top"] <= r["experts"] // groups["count"] * groups["keep"]:
        raise ValueError(f"moe: cannot choose {r['top']} experts")
    return dict(ff=m["expert"]["ff"], experts=r["experts"], top=r["top"], expert_groups=groups["count"], groups_keep=groups["keep"])


FEED_FORWARDS = {"dense": _dense, "moe": _moe}


def _mixer_shapes(p: str, s: LayerSpec, d: int) -> dict:
    hv, hk = s.heads * s.vdim, s.heads * s.dim
    if s.mixer == MIXER_PAIR:
        out = {}
        for side, sub in (("left.", s.left), ("right.", s.right)):
            out.update(_mixer_shapes(p + side, sub, d))
            out[p + side + "out"] = (d,)
        return out
    if s.mixer == MIXER_LIGHTNING:
        out = {"q": (hk, d), "k": (hk, d), "v": (hv, d), "g": (hv, d), "norm": (hv,)}
    elif s.mixer == MIXER_LATENT_ATTENTION:
        out = {"dq": (s.q_rank, d), "dq.norm": (s.q_rank,), "uq": (s.heads * (s.dim + s.rot_dim), s.q_rank),
               "dkv": (s.kv_rank + s.rot_dim, d), "dkv.norm": (s.kv_rank,), "uk": (hk, s.kv_rank), "uv": (hv, s.kv_rank), "g": (hv, d)}
    elif s.mixer == MIXER_ATTENTION:
        out = {"q": (hk, d), "k": (s.kv_heads * s.dim, d), "v": (s.kv_heads * s.vdim, d)}
    else:
        qk = s.kv_heads * s.dim
        out = {"q": (qk, d), "q.conv": (qk, s.conv), "k": (qk, d), "k.conv": (qk, s.conv), "v": (hv, d), "v.conv": (hv, s.conv), "b": (s.heads, d),
               "a": (s.heads, d), "A_log": (s.heads,), "dt_bias": (s.heads,), "norm": (s.vdim,), "g": (hv, d)}
    out["o"] = (d, hv)
    return {p + k: v for k, v in out.items()}


@dataclass
class LayeredConfig:
    """A decoder described layer by layer."""

    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    layers: List[LayerSpec] = field(default_factory=list)
    arrangement: int = ARRANGE_PARALLEL
    norm_offset: float = 0.0        # norm weights are stored minus this
    canon_taps: int = 0             # input convolution of every sublayer
    gated_residual: bool = False
    depth_average: bool = False
    max_positions: int = 0          # learned position table

    @classmethod
    def from_dict(cls, raw: dict) -> "LayeredConfig":
        """Configuration by the document's ``architecture``."""
        return REGISTRY[raw["architecture"]](raw)

    @staticmethod
    def read_layers(raw: dict) -> List[LayerSpec]:
        layers = []
        for i, ly in enumerate(raw["layers"]):
            if ly["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {ly['type']!r} (known: {', '.join(sorted(MIXERS))})")
            mlp = ly.get("mlp")
            if mlp and mlp.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            layers.append(LayerSpec(**MIXERS[ly["type"]](ly["mixer"]), **(FEED_FORWARDS[mlp["kind"]](mlp) if mlp else {})))
        return layers

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

        def fill(c, s):
            for f in fields(s):
                v = getattr(s, f.name)
                if f.name in ("decay", "rot_freq"):
                    setattr(c, f.name, floats(v))
                elif f.name in ("left", "right"):
                    if v is not None:
                        sub = LayerConfig()
                        fill(sub, v)
                        keep.append(sub)
                        setattr(c, f.name, C.addressof(sub))
                else:
                    setattr(c, f.name, v)
            c.rot_pairs = 0 if s.rot_freq is None else len(s.rot_freq)

        arr = (LayerConfig * len(self.layers))()
        for c, s in zip(arr, self.layers):
            fill(c, s)
        mc = LayeredModelConfig(vocab=self.vocab, width=self.width, num_layers=len(self.layers), norm_eps=self.norm_eps,
                                residual_mult=self.residual_mult, logit_scale=self.logit_scale, dtype=DTYPES[dtype], max_seq=max_seq,
                                max_batch=max_batch, arrangement=self.arrangement, norm_offset=self.norm_offset, canon_taps=self.canon_taps,
                                gated_residual=self.gated_residual, depth_average=self.depth_average, max_positions=self.max_positions)
        return mc, arr, keep

    def tensor_shapes(self) -> dict:
        """Checkpoint name -> shape of every tensor the model needs."""
        d, out = self.width, {"embed": (self.vocab, self.width)}
        if self.max_positions:
            out["pos"] = (self.max_positions, d)
        for i, s in enumerate(self.layers):
            p, subs = f"l{i}.", ("1", "2") if s.ff else ("1",)
            out[p + "norm1"] = (d,)
            out.update(_mixer_shapes(p + "mix.", s, d))
            if s.ff and self.arrangement == ARRANGE_SEQUENTIAL:
                out[p + "norm2"] = (d,)
            if s.experts:
                out.update({p + "mlp.router": (s.experts, d), p + "mlp.correction": (s.experts,)})
                for e in range(s.experts):
                    out.update({p + f"mlp.e{e}.up": (s.ff, d), p + f"mlp.e{e}.down": (d, s.ff)})
            elif s.ff:
                out.update({p + "mlp.up": (s.ff, d), p + "mlp.up.b": (s.ff,), p + "mlp.down": (d, s.ff), p + "mlp.down.b": (d,)})
            for n in subs:
                if self.canon_taps:
                    out[p + "canon" + n] = (d, self.canon_taps)
                if self.gated_residual:
                    out.update({p + "rg" + n: (d, d), p + "rg" + n + ".b": (d,)})
            if self.depth_average:
                out[p + "dwa"] = (i + 2,)
        out["final.norm"] = (self.width,)
        out["head"] = (self.vocab, self.width)
        return out


def _mefipel(raw: dict) -> LayeredConfig:
    return LayeredConfig(vocab=raw["vocab"], width=raw["width"], norm_eps=raw["norm"]["eps"], residual_mult=raw["residual_mult"],
                         logit_scale=raw["logit_scale"], layers=LayeredConfig.read_layers(raw))


def _tozarax(raw: dict) -> LayeredConfig:
    return LayeredConfig(vocab=raw["vocab"], width=raw["width"], norm_eps=raw["norm"]["eps"], layers=LayeredConfig.read_layers(raw),
                         arrangement=ARRANGE_SEQUENTIAL, norm_offset=1.0, canon_taps=raw["canon"]["taps"], gated_residual=True,
                         depth_average=True, max_positions=raw["max_positions"])


# architecture named by config.json -> its configuration from the document
REGISTRY = {"Mefipel": _mefipel, "Tozarax": _tozarax}


def read_config(path: str):
    """Configuration of the model in a folder (or of one ``config.json``)."""
    if os.path.isdir(path):
        path = os.path.join(path, "config.json")
    with open(path) as f:
        raw = json.load(f)
    return REGISTRY.get(raw.get("architecture"), UnifiedConfig.from_dict)(raw)


def load_model(backend: CudaBackend, folder: str, dtype: str = "bfloat16", max_seq: int = 4096, max_batch: int = 1) -> PrismEngine:
    """Engine of the model in ``folder``: config.json with ``*.safetensors`` (layered) or one ``.cimage``
    (palettized; its arithmetic is fixed, ``dtype`` must stay "bfloat16")."""
    cfg = read_config(folder)
    if isinstance(cfg, LayeredConfig):
        if cfg.max_positions:  # a sequence cannot be longer than the position table
            max_seq = min(max_seq, cfg.max_positions)
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
