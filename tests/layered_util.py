"""Small random models described layer by layer, for the tests of the layered engine (config dict + bf16 weights)."""
import json
import struct

import numpy as np


def lightning(heads, dim, vdim, decay=None, ff=None):
    decay = [float(d) for d in (decay if decay is not None else np.linspace(0.5, 0.99, heads))]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window=None, scale=None, dims=None, base=1e4, scaling="yarn", ff=None):
    if scaling == "yarn":
        scaling = {"factor": 3.0, "fast": 8.0, "original": 256, "slow": 0.5}
    rot = {"base": base, "dims": rot_dim if dims is None else dims}
    if scaling:
        rot["scaling"] = scaling
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot": rot,
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(layers, width=48, vocab=131, eps=1e-5, residual_mult=0.7, logit_scale=1.5):
    return {"architecture": "Mefipel", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "vocab": vocab, "width": width}


# ---- sequential arrangement --------------------------------------------------------------------------
def attention(heads, kv_heads, dim, vdim, window=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.3 * dim ** -0.5 if scale is None else scale}
    if window:
        m["mask"] = {"size": window}
    return m


def delta(heads, kv_heads, dim, vdim, conv=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def pair(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def tozarax(layers, width=48, vocab=131, eps=1e-5, taps=3, max_positions=600):
    return {"architecture": "Tozarax", "canon": {"taps": taps}, "layers": layers, "max_positions": max_positions, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def sequential(layers, width=48, vocab=131, eps=1e-5, norm_offset=0.0, **options):
    """A design of its own from the same parts: any mixer or feed-forward, any of the options left out."""
    return {"architecture": "SequentialTest", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "norm_offset": norm_offset,
            "options": options}


def _register():
    from prism_engine_b200 import models as m

    m.REGISTRY["SequentialTest"] = lambda raw: m.LayeredConfig(
        vocab=raw["vocab"], width=raw["width"], norm_eps=raw["norm"]["eps"], layers=m.LayeredConfig.read_layers(raw),
        arrangement=m.ARRANGE_SEQUENTIAL, norm_offset=raw["norm_offset"], **raw["options"])


_register()


def sequential_weights(cfg, seed=0, apart=1.0):
    """As weights(); `apart`: how far the experts of a layer (and their corrections) differ.  A little makes a routing
    decided by rounding harmless, 1 makes them independent."""
    import prism_engine_b200 as p

    rng = np.random.default_rng([8, seed])
    c = p.LayeredConfig.from_dict(cfg)
    out, base = {}, {}
    for name, shape in c.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if leaf.startswith("norm") and name.count(".") == 1 or name == "final.norm":
            v = rng.normal(0.0, 0.3, shape) + 1.0 - c.norm_offset
        elif leaf in ("norm", "out"):
            v = rng.normal(1.0, 0.3, shape)
        elif leaf == "dwa":
            v = rng.normal(0.0, 0.2, shape)
            v[-1] += 1.0
        elif leaf == "correction":
            v = rng.normal(0.0, 0.3 * apart, shape)
        elif leaf in ("A_log", "dt_bias"):
            v = rng.normal(-1.0, 0.8, shape)
        elif leaf.startswith("canon") or leaf == "conv":
            v = rng.normal(0.0, 0.5, shape)
        elif leaf == "pos":
            v = rng.normal(0.0, 0.4, shape)
        elif leaf == "b" and len(shape) == 1:
            v = rng.normal(0.0, 0.5, shape)
        elif len(shape) == 1:
            v = rng.normal(0.0, 0.3, shape)
        else:
            v = rng.normal(0.0, 1.0 if name == "embed" else 1.2 / np.sqrt(shape[1]), shape)
        head, _, part = name.partition(".mlp.e")
        if part:
            key = head, leaf
            base.setdefault(key, rng.normal(0.0, 1.2 / np.sqrt(shape[1]), shape))
            v = (1.0 - apart) * base[key] + apart * v
        out[name] = round_bf16(v)[1]
    return out


def keep_bf16(x):
    return round_bf16(x)[1].astype(np.float64).reshape(np.shape(x))


def expected(cfg, w, toks, dtype):
    """The restatement's logits of a sequential model; for bf16 with the activations between linears rounded as a
    16-bit run rounds them, so that norms of small values and choices of experts see the same rounding."""
    from oracle import layered as orc

    return orc.forward(cfg, w, toks, **({"rounding": keep_bf16} if dtype == "bfloat16" else {}))


def round_bf16(x):
    """Nearest bf16 (ties to even) of a float array: (bit patterns, float32 values)."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    b = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)
    return b, (b.astype(np.uint32) << 16).view(np.float32)


def weights(cfg, seed=0):
    """name -> float32 array of bf16 values; matrices keep the variance of their input, norms vary around 1."""
    import prism_engine_b200 as p

    rng = np.random.default_rng([7, seed])
    out = {}
    for name, shape in p.LayeredConfig.from_dict(cfg).tensor_shapes().items():
        if len(shape) == 1:
            v = rng.normal(0.0, 0.3, shape) + (0.0 if name.endswith(".b") else 1.0)
        else:
            v = rng.normal(0.0, 1.0 if name == "embed" else 1.2 / np.sqrt(shape[1]), shape)
        out[name] = round_bf16(v)[1]
    return out


def bits(x):
    return round_bf16(x)[0]


def engine(be, cfg, w, dtype="float32", max_seq=512, max_batch=1, chunk=None):
    import prism_engine_b200 as p

    if chunk is not None:
        be.set_option("layered_chunk", chunk)
    try:
        eng = p.PrismEngine(be, p.LayeredConfig.from_dict(cfg), dtype=dtype, max_seq=max_seq, max_batch=max_batch)
    finally:
        if chunk is not None:
            be.set_option("layered_chunk", 2048)
    for name, a in w.items():
        eng.set_tensor(name, bits(a))
    return eng


def run_portions(eng, tokens, sizes):
    """Logits at every position of one sequence fed in portions of the given sizes (the last one repeats)."""
    seq = eng.open_sequence()
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(eng.extend([(seq, tokens[at:at + n], list(range(n)))]))
        at += n
        i += 1
    eng.close_sequence(seq)
    return np.concatenate(out)


def error(got, want):
    """Worst position: rms over the vocabulary of the difference (mean removed) over the rms spread of the logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    return float(np.sqrt((d * d).mean(axis=-1)).max() / spread)


TOL = {"float32": 2e-5, "bfloat16": 4e-2}


def write_safetensors(path, w, dtype="BF16", pad=0):
    head, blobs, at = {}, [], 0
    for name, a in w.items():
        b = bits(a).tobytes()
        head[name] = {"dtype": dtype, "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    head["__metadata__"] = {"format": "pt"}
    h = json.dumps(head).encode() + b" " * pad
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
