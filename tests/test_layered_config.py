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


# ---- sequential layers -----------------------------------------------------------------------------------------

def _tozarax():
    return U.tozarax([U.pair(U.attention(4, 2, 8, 12, window=9), U.delta(3, 1, 16, 20, conv=4), U.moe(8, 3, 24, (4, 2))),
                      U.pair(U.attention(2, 1, 8, 8), U.delta(1, 1, 8, 8))], taps=2, max_positions=70)


def test_sequential_configuration(tmp_path):
    cfg = p.read_config(_write(tmp_path, _tozarax()))
    a, b = cfg.layers
    assert (cfg.arrangement, cfg.norm_offset, cfg.canon_taps, cfg.max_positions) == (models.ARRANGE_SEQUENTIAL, 1.0, 2, 70)
    assert cfg.gated_residual and cfg.depth_average
    assert a.mixer == models.MIXER_PAIR and a.left.window == 9 and b.left.window == 0 and a.right.conv == 4
    assert (a.ff, a.experts, a.top, a.expert_groups, a.groups_keep, b.ff) == (24, 8, 3, 4, 2, 0)
    sh = cfg.tensor_shapes()
    assert sh["l0.mix.left.v"] == (24, 48) and sh["l0.mix.right.v"] == (60, 48) and sh["l0.mix.right.k.conv"] == (16, 4)
    assert sh["l0.dwa"] == (2,) and sh["l1.dwa"] == (3,) and sh["pos"] == (70, 48) and sh["l0.rg2"] == (48, 48) and sh["l0.canon1"] == (48, 2)
    assert "l1.norm2" not in sh and "l1.rg2" not in sh and "l1.canon2" not in sh and "l0.mlp.e8.up" not in sh
    mc, arr, keep = cfg.to_c("bfloat16", 64, 2)
    assert (mc.arrangement, mc.canon_taps, mc.depth_average, mc.max_positions) == (1, 2, 1, 70)
    from prism_engine_b200._lib import LayerConfig
    right = LayerConfig.from_address(arr[0].right)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.conv) == (3, 1, 16, 20, 4) and keep
    bad = _tozarax()
    bad["layers"][0]["mlp"]["router"]["groups"]["keep"] = 1
    with pytest.raises(ValueError, match="choose 3"):
        p.LayeredConfig.from_dict(bad)
    bad = _tozarax()
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 3
    with pytest.raises(ValueError, match="share"):
        p.LayeredConfig.from_dict(bad)


def test_oracle_gated_delta_against_its_triangular_form():
    """The recurrence against the solved system of all updates (one chunk, state from zero)."""
    rng = np.random.default_rng(3)
    T, D, V = 11, 4, 5
    mx = {"heads": 1, "kv_heads": 1, "dim": D, "vdim": V, "conv": 2}
    w = {n: rng.normal(size=s) for n, s in {"q": (D, 6), "k": (D, 6), "v": (V, 6), "b": (1, 6), "a": (1, 6), "g": (V, 6), "o": (6, V), "q.conv": (D, 2),
                                            "k.conv": (D, 2), "v.conv": (V, 2), "A_log": 1, "dt_bias": 1, "norm": V}.items()}
    h = rng.normal(size=(T, 6))
    act = lambda n: orc.silu(orc.causal_conv(h @ w[n].T, w[n + ".conv"]))  # noqa: E731
    q, k, v = orc.unit(act("q")) * D ** -0.5, orc.unit(act("k")), act("v")
    L = np.cumsum(-np.exp(w["A_log"]) * np.log1p(np.exp(h @ w["a"].T + w["dt_bias"])))
    beta = orc.sigmoid(h @ w["b"].T)[:, 0]
    dec = np.exp(L[:, None] - L[None, :])
    u = np.linalg.solve(np.eye(T) + np.tril(beta[:, None] * dec * (k @ k.T), -1), beta[:, None] * v)
    o = np.tril(dec * (q @ k.T)) @ u
    want = orc.rms_norm(o, w["norm"], 1e-3) * orc.silu(h @ w["g"].T) @ w["o"].T
    np.testing.assert_allclose(orc.gated_delta(h, w, mx, 1e-3), want, rtol=1e-8, atol=1e-10)


def test_oracle_routing():
    z = np.log(np.array([0.9, 0.12, 0.6, 0.55, 0.5, 0.45, 0.8, 0.2]) / (1 - np.array([0.9, 0.12, 0.6, 0.55, 0.5, 0.45, 0.8, 0.2])))
    best, weight = orc.route(z, np.zeros(8), 3, None)
    assert best == [0, 6, 2] and weight == pytest.approx([0.9, 0.8, 0.6])
    # groups (0 1)(2 3)(4 5)(6 7) score 1.02, 1.15, 0.95, 1.0: the first two are kept
    assert orc.route(z, np.zeros(8), 3, {"count": 4, "keep": 2})[0] == [0, 2, 3]
    best, weight = orc.route(z, np.array([-2.0, 0, 0, 0, 0, 0, -2.0, -2.0]), 2, {"count": 4, "keep": 3})
    assert best == [2, 3] and weight == pytest.approx([0.6, 0.55])  # the weight is the score without the correction
    assert orc.route(z, np.full(8, -5.0), 2, {"count": 2, "keep": 1})[0] == [0, 2]


def test_oracle_convolution_and_average():
    x, w = np.arange(1.0, 6.0)[:, None], np.array([[100.0, 10.0, 1.0]])
    assert orc.causal_conv(x, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]
    assert orc.depth_average([0.5, 2.0], [np.ones(2), np.full(2, 3.0)]).tolist() == [6.5, 6.5]
