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
