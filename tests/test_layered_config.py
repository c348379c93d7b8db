"""Model registry, configuration, rotation frequencies and the oracle of the layered models (CPU)."""
import json
import subprocess
import sys
import os

import numpy as np
import pytest

import layered_util as U
from oracle import layered as orc

import prism_engine_b200 as p
from prism_engine_b200 import models

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _write(tmp_path, raw):
    (tmp_path / "config.json").write_text(json.dumps(raw))
    return str(tmp_path)


def test_registry_picks_the_class(tmp_path):
    raw = U.model([U.lightning(2, 8, 12, ff=40), U.latent(3, 8, 4, 20, 24, 16, window=9)])
    cfg = p.read_config(_write(tmp_path, raw))
    assert isinstance(cfg, p.LayeredConfig)
    assert [s.mixer for s in cfg.layers] == [models.MIXER_LIGHTNING, models.MIXER_LATENT_ATTENTION]
    assert cfg.layers[0].ff == 40 and cfg.layers[1].ff == 0 and cfg.layers[1].window == 9
    qwen = {"architectures": ["Qwen2ForCausalLM"], "hidden_size": 64, "num_attention_heads": 4, "num_hidden_layers": 2}
    assert isinstance(p.read_config(_write(tmp_path, qwen)), p.UnifiedConfig)


def test_unknown_parts_are_refused():
    bad = U.model([U.lightning(2, 8, 12)])
    bad["layers"][0]["type"] = "mystery"
    with pytest.raises(ValueError, match="unknown mixer"):
        p.LayeredConfig.from_dict(bad)
    bad = U.model([U.lightning(2, 8, 12, ff=16)])
    bad["layers"][0]["mlp"]["kind"] = "sparse"
    with pytest.raises(ValueError, match="feed-forward"):
        p.LayeredConfig.from_dict(bad)
    with pytest.raises(ValueError, match="decays"):
        p.LayeredConfig.from_dict(U.model([U.lightning(2, 8, 12, decay=[0.5])]))
    with pytest.raises(ValueError, match="rotate"):
        p.LayeredConfig.from_dict(U.model([U.latent(2, 8, 4, 8, 8, 8, dims=6)]))


@pytest.mark.parametrize("base,dims,scaling", [
    (1e4, 16, None), (2e5, 64, {"factor": 8.0, "fast": 24.0, "original": 4096, "slow": 1.5}),
    (5e5, 2, {"factor": 2.0, "fast": 4.0, "original": 128, "slow": 1.0}),
    (1e4, 10, {"factor": 1.0, "fast": 1.0, "original": 64, "slow": 1.0}),       # lo == hi or close
    (1e4, 24, {"factor": 40.0, "fast": 1e-3, "original": 64, "slow": 1e-4})])   # hi clamped to dims - 1
def test_rotation_frequencies(base, dims, scaling):
    f, mul = models.yarn_frequencies(base, dims, scaling)
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = scaling
    want, wmul = orc.rotation_frequencies(rot)
    np.testing.assert_allclose(f, want, rtol=1e-12)
    assert mul == pytest.approx(wmul, rel=1e-12)


def test_tensor_shapes_and_c_structs():
    raw = U.model([U.latent(3, 8, 6, 20, 24, 16, window=5, dims=4, ff=24), U.lightning(1, 8, 12)])
    cfg = p.LayeredConfig.from_dict(raw)
    shapes = cfg.tensor_shapes()
    assert shapes["l0.mix.uq"] == (3 * 14, 24) and shapes["l0.mix.dkv"] == (22, 48) and shapes["l1.mix.norm"] == (12,)
    assert "l1.mlp.up" not in shapes and shapes["l0.mlp.down.b"] == (48,)
    mc, arr, keep = cfg.to_c("float32", 100, 3)
    assert (mc.vocab, mc.dtype, mc.max_seq, mc.max_batch, mc.num_layers) == (131, 1, 100, 3, 2)
    assert arr[0].rot_pairs == 2 and arr[0].rot_dim == 6 and not arr[0].decay and arr[1].decay[0] == pytest.approx(0.5)
    with pytest.raises(ValueError):
        cfg.to_c("float16", 1, 1)


def test_command_line(tmp_path):
    raw = U.model([U.lightning(2, 8, 12)])
    folder = _write(tmp_path, raw)
    out = subprocess.run([sys.executable, "-m", "prism_engine_b200", "info", "--model", folder], capture_output=True, text=True, cwd=ROOT, check=True)
    info = json.loads(out.stdout)
    assert info["kind"] == "layered" and info["layers"] == 1 and info["parameters"] > 0
    # a palettized model has no 32-bit form: the trace replay says so before it needs a GPU
    folder = _write(tmp_path, {"hidden_size": 64, "num_attention_heads": 4})
    rc = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", folder, "--max-tokens", "8"],
                        stdin=subprocess.DEVNULL, capture_output=True).returncode
    assert rc == 3


def test_lightning_recurrence_against_closed_form():
    rng = np.random.default_rng(1)
    T, mx = 9, {"heads": 2, "dim": 3, "vdim": 4, "decay": [0.5, 0.9]}
    w = {k: rng.normal(size=s) for k, s in dict(q=(6, 5), k=(6, 5), v=(8, 5), g=(8, 5), o=(5, 8)).items()}
    w["norm"] = rng.normal(size=8)
    h = rng.normal(size=(T, 5))
    q, k, v = (orc.silu(h @ w[n].T).reshape(T, 2, -1) for n in "qkv")
    o = np.zeros((T, 2, 4))
    for t in range(T):
        for j in range(t + 1):
            for n in range(2):
                o[t, n] += (q[t, n] @ k[j, n]) * mx["decay"][n] ** (t - j) * v[j, n]
    want = orc.rms_norm(o.reshape(T, 8), w["norm"], 1e-3) * orc.sigmoid(h @ w["g"].T) @ w["o"].T
    np.testing.assert_allclose(orc.lightning(h, w, mx, 1e-3), want, rtol=1e-9, atol=1e-12)


def test_rotation_is_relative_and_window_counts_itself():
    rot = {"base": 100.0, "dims": 6}
    rng = np.random.default_rng(2)
    a, b = rng.normal(size=(1, 8)), rng.normal(size=(1, 8))
    s = [float((orc.rotate(a, [i], rot) @ orc.rotate(b, [j], rot).T)[0, 0]) for i, j in ((5, 2), (105, 102))]
    assert s[0] == pytest.approx(s[1], rel=1e-9)
    assert np.array_equal(orc.rotate(a, [7], rot)[0, 6:], a[0, 6:])
    assert [orc.window_visible(10, j, 3) for j in (7, 8, 9, 10, 11)] == [False, True, True, True, False]
