"""The layered engine on the GPU against the plain restatement (oracle/layered.py): mechanisms alone, portions,
decoding, batches, slots, window and chunk edges, generation, loading, command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import layered_util as U
from oracle import layered as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


def tokens(n, vocab, seed=0):
    return np.random.default_rng([11, seed]).integers(0, vocab, n).tolist()


def check(be, cfg, n=70, sizes=(10 ** 9,), dtype="float32", seed=0, **kw):
    w = U.weights(cfg, seed)
    toks = tokens(n, cfg["vocab"], seed)
    want = orc.forward(cfg, w, toks)
    eng = U.engine(be, cfg, w, dtype, max_seq=n, **kw)
    try:
        got = U.run_portions(eng, toks, list(sizes))
    finally:
        eng.close()
    err = U.error(got, want)
    assert err < U.TOL[dtype], err
    return err


LIGHTNING = [
    dict(heads=2, dim=16, vdim=32), dict(heads=1, dim=8, vdim=8, decay=[1.0]), dict(heads=3, dim=20, vdim=36, decay=[0.2, 0.97, 1.0]),
    dict(heads=2, dim=7, vdim=13), dict(heads=1, dim=136, vdim=40), dict(heads=1, dim=256, vdim=64, decay=[0.9985]),
    dict(heads=1, dim=272, vdim=24, decay=[0.9]), dict(heads=2, dim=24, vdim=16, decay=[0.0, 0.5])]
LATENT = [
    dict(heads=2, dim=16, rot_dim=8, vdim=24, q_rank=40, kv_rank=32, window=20),
    dict(heads=1, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=8),
    dict(heads=3, dim=20, rot_dim=6, vdim=28, q_rank=33, kv_rank=37, window=17),            # nothing a multiple of 8
    dict(heads=5, dim=24, rot_dim=16, vdim=40, q_rank=64, kv_rank=72, window=1),
    dict(heads=2, dim=16, rot_dim=16, vdim=136, q_rank=40, kv_rank=100, window=33, dims=8),  # part of rot_dim turns
    dict(heads=18, dim=8, rot_dim=8, vdim=16, q_rank=24, kv_rank=24, scaling=None),          # more than 16 heads
    dict(heads=1, dim=192, rot_dim=64, vdim=256, q_rank=72, kv_rank=264, window=50),
    dict(heads=2, dim=200, rot_dim=64, vdim=48, q_rank=72, kv_rank=64, window=40),           # too wide to expand
    dict(heads=2, dim=16, rot_dim=8, vdim=72, q_rank=16, kv_rank=640, window=3, dims=0),
    dict(heads=1, dim=16, rot_dim=8, vdim=16, q_rank=16, kv_rank=1400, window=30)]           # too wide for the tensor-core rows


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(LIGHTNING)))
def test_lightning_alone(backend, dtype, i):
    check(backend, U.model([U.lightning(**LIGHTNING[i])], width=40 + 8 * i), n=150, dtype=dtype, seed=i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(LATENT)))
def test_latent_attention_alone(backend, dtype, i):
    check(backend, U.model([U.latent(**LATENT[i])], width=40 + 8 * i), n=150, dtype=dtype, seed=i)
    check(backend, U.model([U.latent(**LATENT[i])], width=40 + 8 * i), n=45, sizes=(20, 1), dtype=dtype, seed=i)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_and_constants(backend, dtype):
    cfg = U.model([U.lightning(1, 8, 8, ff=72)], width=56, eps=0.3, residual_mult=1.7, logit_scale=0.4)
    w = U.weights(cfg, 3)
    w["l0.mix.o"] *= 0.0  # the feed-forward alone
    toks = tokens(40, cfg["vocab"], 3)
    want = orc.forward(cfg, w, toks)
    eng = U.engine(backend, cfg, w, dtype)
    got = U.run_portions(eng, toks, [30, 1])
    eng.close()
    assert U.error(got, want) < U.TOL[dtype]
    if dtype == "float32":  # scale and offset too, not only the shape of the logits
        np.testing.assert_allclose(got, want, rtol=1e-4, atol=1e-4)
    check(backend, U.model([U.lightning(1, 8, 8, ff=200)], eps=1.0, residual_mult=-0.5, logit_scale=3.0), dtype=dtype)
    check(backend, U.model([U.latent(2, 8, 8, 8, 16, 16)], width=200, vocab=3), dtype=dtype)


def mixed(width=88, vocab=210, ff=104):
    """Every layer another size; layers with and without feed-forward, with and without a window."""
    return U.model([U.latent(3, 16, 8, 24, 40, 48, window=21, ff=ff), U.lightning(2, 24, 40, decay=[0.8, 0.995], ff=None),
                    U.lightning(4, 8, 16, ff=ff + 40), U.latent(2, 32, 16, 16, 24, 32, ff=None), U.latent(5, 8, 8, 40, 56, 24, window=64, ff=ff)],
                   width=width, vocab=vocab, residual_mult=0.4)


PORTIONS = [(1,), (2,), (3, 2), (5, 7, 2), (9,), (16, 1), (17, 2, 33), (63, 1, 1, 65), (64,), (65, 3), (100, 1), (140, 2, 2, 1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", PORTIONS)
def test_portions(backend, dtype, sizes):
    check(backend, mixed(), n=180, sizes=sizes, dtype=dtype, seed=5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 2, 7, 32, 64])
def test_small_rings(backend, dtype, chunk):
    """Short prefill chunks: windowed caches hold window - 1 + chunk positions and wrap many times."""
    check(backend, mixed(), n=200, sizes=(50, 3, 1, 1, 1, 90, 1), dtype=dtype, seed=6, chunk=chunk)


def test_cut_independence(backend):
    """The same tokens in other portions, after other sequences, in another slot."""
    for dtype in DTYPES:
        cfg, n = mixed(), 150
        w, toks = U.weights(cfg, 7), tokens(150, 210, 7)
        eng = U.engine(backend, cfg, w, dtype, max_seq=n, max_batch=3)
        base = U.run_portions(eng, toks, [n])
        hold = eng.open_sequence()  # the next sequence gets another slot
        eng.extend([(hold, tokens(60, 210, 8), [])])
        for sizes in ([1], [2], [31, 2, 1], [149, 1]):
            assert U.error(U.run_portions(eng, toks, sizes), base) < U.TOL[dtype] / 2, (dtype, sizes)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(backend, dtype):
    """Prompts of several lengths and decode rows in the same steps against each request alone; slots are reused."""
    cfg = mixed()
    w = U.weights(cfg, 9)
    lens = [1, 2, 19, 40, 64, 97, 33, 5, 80, 23, 50, 12]
    reqs = [tokens(n + 6, cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    want = [orc.forward(cfg, w, r) for r in reqs]
    eng = U.engine(backend, cfg, w, dtype, max_seq=128, max_batch=10)
    live, at, got = {}, {}, {i: [] for i in range(len(reqs))}
    waiting = list(range(len(reqs)))
    while waiting or live:
        while waiting and len(live) < 10:
            i = waiting.pop(0)
            live[i] = eng.open_sequence()
            at[i] = 0
        entries, took = [], []
        for i, s in live.items():
            n = min(max(lens[i] - at[i], 1), 37)  # the prompt in portions, then one token at a time
            entries.append((s, reqs[i][at[i]:at[i] + n], list(range(n))))
            took.append((i, n))
        lg = eng.extend(entries)
        row = 0
        for i, n in took:
            got[i].append(lg[row:row + n])
            row += n
            at[i] += n
            if at[i] == len(reqs[i]):
                eng.close_sequence(live.pop(i))
    eng.close()
    for i, x in got.items():
        assert U.error(np.concatenate(x), want[i]) < U.TOL[dtype], i


def test_decode_batch_beyond_the_small_kernel(backend):
    """20 sequences decode together: the tensor-core GEMM with a 32-row tile, and 3 with the small-batch kernel."""
    cfg = mixed()
    w = U.weights(cfg, 10)
    for B in (3, 20):
        reqs = [tokens(30 + i, cfg["vocab"], 60 + i) for i in range(B)]
        want = [orc.forward(cfg, w, r) for r in reqs]
        eng = U.engine(backend, cfg, w, "bfloat16", max_seq=64, max_batch=B)
        seqs = [eng.open_sequence() for _ in range(B)]
        eng.extend([(s, r[:-6], []) for s, r in zip(seqs, reqs)])
        for k in range(6):  # eager, captured, replayed
            lg = eng.extend([(s, [r[len(r) - 6 + k]], [0]) for s, r in zip(seqs, reqs)])
            for i in range(B):
                assert U.error(lg[i:i + 1], want[i][len(reqs[i]) - 6 + k][None]) < 1.5 * U.TOL["bfloat16"], (B, k, i)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes_and_wanted_places_in_any_order(backend, dtype):
    cfg = U.model([U.latent(3, 10, 6, 14, 23, 19, window=11, ff=37), U.lightning(3, 9, 5, ff=61), U.lightning(1, 5, 3)], width=45, vocab=101)
    check(backend, cfg, n=90, sizes=(33, 2, 1), dtype=dtype, seed=17)
    w, toks = U.weights(cfg, 18), tokens(40, 101, 18)
    want = orc.forward(cfg, w, toks)
    eng = U.engine(backend, cfg, w, dtype, max_seq=64, chunk=16)  # the places fall into several chunks
    s = eng.open_sequence()
    places = [38, 3, 3, 17, 16, 0, 30]
    assert U.error(eng.extend([(s, toks[:39], places)]), want[places]) < U.TOL[dtype]
    assert U.error(eng.extend([(s, toks[39:], [0, 0])]), want[[39, 39]]) < U.TOL[dtype]
    eng.close()


def test_unfused_path_agrees(backend):
    """Option fuse = 0: separate norms and the tensor-core GEMM at every size, one row included."""
    backend.set_option("fuse", 0)
    try:
        check(backend, mixed(), n=60, sizes=(20, 1, 2), dtype="bfloat16", seed=12)
    finally:
        backend.set_option("fuse", 1)


@pytest.mark.parametrize("rows", [9, 17, 40, 100, 129, 200, 300])
def test_token_tiles_of_the_gemm(backend, rows):
    """A feed-forward of 150 row tiles: every token tile (16 .. 256) of the tensor-core GEMM, full and ragged."""
    check(backend, U.model([U.lightning(1, 8, 8, ff=19200)], width=64), n=rows, dtype="bfloat16", seed=rows)


# ---- keys that stand out ---------------------------------------------------------------------------------

def _spiked(window, heads=2, expand=True):
    """One latent layer whose query of the filler token strongly prefers the key of one other token, whatever the
    distance; returns (config, weights, filler, special)."""
    dim, rot, vdim = (16, 8, 16) if expand else (20, 4, 12)
    cfg = U.model([U.latent(heads, dim, rot, vdim, 24, 32, window=window, scale=2.5)], width=64, vocab=97, residual_mult=1.0)
    w = U.weights(cfg, 31)
    kv = 32
    w["l0.mix.dkv"] = w["l0.mix.dkv"].copy()
    w["l0.mix.dkv"][kv:] *= 0.02  # the rotated part says almost nothing
    w["l0.mix.dkv"] = U.round_bf16(w["l0.mix.dkv"])[1]
    h = orc.rms_norm(w["embed"].astype(np.float64), w["l0.norm1"], 1e-5)
    q = (orc.rms_norm(h @ w["l0.mix.dq"].T, w["l0.mix.dq.norm"], 1e-5) @ w["l0.mix.uq"].T).reshape(97, heads, -1)[:, :, :dim]
    k = (orc.rms_norm((h @ w["l0.mix.dkv"].T)[:, :kv], w["l0.mix.dkv.norm"], 1e-5) @ w["l0.mix.uk"].T).reshape(97, heads, dim)
    s = np.einsum("ahd,bhd->abh", q, k) * 2.5
    gain = (s - np.einsum("aah->ah", s)[:, None, :]).min(axis=2)  # how much filler a prefers b over itself, in every head
    a, b = np.unravel_index(np.argmax(gain), gain.shape)
    assert gain[a, b] > 6.0
    return cfg, w, int(a), int(b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("expand", [True, False])
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100])
def test_window_edges(backend, dtype, expand, window):
    """The last token that sees the special key and the first that does not, in prompts and decoded, with the
    special token at several places relative to tiles, portions and the ring."""
    cfg, w, fill, special = _spiked(window, expand=expand)
    wrong = json.loads(json.dumps(cfg))
    for place in (0, 1, 37, 64):
        n = place + window + 3
        toks = [fill] * n
        toks[place] = special
        want = orc.forward(cfg, w, toks)
        if window > 1:  # the edge shows: a window one token off is far outside the tolerance
            for off, pos in ((-1, place + window - 1), (1, place + window)):
                wrong["layers"][0]["mixer"]["mask"]["size"] = window + off
                assert U.error(orc.forward(wrong, w, toks)[pos:pos + 1], want[pos:pos + 1]) > 5 * U.TOL[dtype]
        eng = U.engine(backend, cfg, w, dtype, max_seq=n, chunk=48)
        for sizes in ([n], [max(1, n - 6), 1], [place + 1, max(1, window - 2), 2], [1 if n < 40 else 33]):
            assert U.error(U.run_portions(eng, toks, sizes), want) < U.TOL[dtype], (place, sizes)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_without_window(backend, dtype):
    """One key hundreds of tokens back decides the output; a cache that loses or misplaces it is caught."""
    cfg, w, fill, special = _spiked(None)
    n = 420
    toks = [fill] * n
    toks[3] = special
    want = orc.forward(cfg, w, toks)
    lost = orc.forward(cfg, w, [fill] * n)
    assert U.error(lost[-1:], want[-1:]) > 5 * U.TOL[dtype]
    eng = U.engine(backend, cfg, w, dtype, max_seq=n, chunk=128)
    for sizes in ([n], [300, 1], [130, 5, 200, 2]):
        assert U.error(U.run_portions(eng, toks, sizes), want) < U.TOL[dtype], sizes
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_state_reaches_far(backend, dtype):
    """Decay 1 and almost 1: the first tokens' contribution survives hundreds of tokens, over chunk edges of 64 and
    portions; a lost state shows in the oracle by far more than the tolerance."""
    cfg = U.model([U.lightning(2, 16, 24, decay=[1.0, 0.9995])], width=64, residual_mult=1.5)
    w = U.weights(cfg, 41)
    h = orc.rms_norm(w["embed"][5].astype(np.float64), w["l0.norm1"], 1e-5)
    # the filler's own keys vanish (silu of a large negative number), so what the first tokens left is what it reads
    w["l0.mix.k"] = U.round_bf16(w["l0.mix.k"] - np.outer(w["l0.mix.k"] @ h + 12.0, h) / (h @ h))[1]
    n = 330
    toks = tokens(20, 131, 1) + [5] * (n - 20)
    want = orc.forward(cfg, w, toks)
    lost = orc.forward(cfg, w, toks[20:])
    assert U.error(lost[-1:], want[-1:]) > 5 * U.TOL[dtype]
    eng = U.engine(backend, cfg, w, dtype, max_seq=n)
    for sizes in ([n], [64], [63, 65, 2, 1], [20, 1], [300, 1]):
        assert U.error(U.run_portions(eng, toks, sizes), want) < U.TOL[dtype], sizes
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_start_empty(backend, dtype):
    """A reused slot carries nothing over: same logits as on a fresh engine, bit for bit."""
    cfg = mixed()
    w, toks = U.weights(cfg, 13), tokens(60, 210, 13)
    eng = U.engine(backend, cfg, w, dtype, max_seq=128, max_batch=2)
    first = U.run_portions(eng, toks, [40, 1])
    for seed in (1, 2, 3):
        U.run_portions(eng, tokens(100, 210, seed), [50])
        assert np.array_equal(U.run_portions(eng, toks, [40, 1]), first)
    eng.close()


def test_long_decoding(backend):
    cfg = mixed(vocab=61)
    w = U.weights(cfg, 14)
    toks = tokens(400, 61, 14)
    want = orc.forward(cfg, w, toks)
    for dtype in DTYPES:
        eng = U.engine(backend, cfg, w, dtype, max_seq=400, chunk=16)
        assert U.error(U.run_portions(eng, toks, [5, 1]), want) < U.TOL[dtype]
        eng.close()


# ---- entry points ------------------------------------------------------------------------------------------

def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(orc.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def test_generate_batch_and_steps(backend):
    cfg = mixed(vocab=90)
    w = U.weights(cfg, 15)
    prompts = [tokens(25, 90, 70 + i) for i in range(3)]
    want = [greedy(cfg, w, q, 12) for q in prompts]
    eng = U.engine(backend, cfg, w, "float32", max_seq=64, max_batch=3)
    assert eng.generate(prompts, 12).tolist() == want
    assert eng.generate(prompts[1], 12).tolist() == want[1]
    out, lg = eng.generate(prompts[0][:1], 3, return_logits=True)  # a prompt of one token
    assert out.tolist() == greedy(cfg, w, prompts[0][:1], 3) and lg.shape == (90,)
    eng.reset(2)  # step() and decode() drive the same loop
    for t in range(24):
        eng.step([prompts[0][t], prompts[2][t]])
    nxt = eng.step([prompts[0][24], prompts[2][24]])
    rest = eng.decode(nxt, 5)
    assert [[int(a)] + b.tolist() for a, b in zip(nxt, rest)] == [want[0][:6], want[2][:6]]
    # greedy token of prompt portions and of decode rows through extend()
    eng.reset(0)
    s = eng.open_sequence()
    _, nx = eng.extend([(s, prompts[0], [])], want_next=True)
    got = [int(nx[0])]
    while len(got) < 12:
        _, nx = eng.extend([(s, [got[-1]], [])], want_next=True)
        got.append(int(nx[0]))
    assert got == want[0]
    assert eng.step_bytes() > 0 and eng.kernels_per_step() > 0
    eng.close()


def test_errors_are_reported(backend):
    import prism_engine_b200 as p

    cfg = U.model([U.lightning(1, 8, 8), U.latent(1, 8, 8, 12, 8, 8, window=4)])
    w = U.weights(cfg)
    lacking = {k: v for k, v in w.items() if k != "l1.mix.uv"}
    eng = U.engine(backend, cfg, lacking, max_seq=16)
    with pytest.raises(p.PrismCudaError, match="l1.mix.uv"):
        eng.generate([1, 2], 1)
    with pytest.raises(p.PrismCudaError, match="miss l9"):
        eng.set_tensor("l9.norm1", U.bits(w["l0.norm1"]))
    with pytest.raises(p.PrismCudaError, match="needs"):
        eng.set_tensor("l1.mix.uv", U.bits(w["l1.mix.uv"].T))
    eng.set_tensor("l1.mix.uv", U.bits(w["l1.mix.uv"]))
    s = eng.open_sequence()
    with pytest.raises(p.PrismCudaError, match="in use"):
        eng.open_sequence()
    for bad in ([(s, [], [])], [(s, [131], [])], [(s, [1, 2], [2])], [(s, [1], [1])], [(3, [1], [])], [(s, [1], []), (s, [2], [])]):
        with pytest.raises(p.PrismCudaError):
            eng.extend(bad)
    with pytest.raises(p.PrismCudaError, match="max_seq"):
        eng.extend([(s, [1] * 17, [])])
    assert eng.sequence_position(s) == 0
    eng.close_sequence(s)
    with pytest.raises(p.PrismCudaError, match="not open"):
        eng.close_sequence(s)
    with pytest.raises(p.PrismCudaError):
        eng.profile_gemv()
    eng.close()


def test_loading_generation_and_trace_from_a_folder(backend, tmp_path):
    """safetensors + config.json through the registry, the command line and the trace replay."""
    import prism_engine_b200 as p

    cfg = mixed(vocab=77)
    w = U.weights(cfg, 16)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    path = str(tmp_path / "model.safetensors")
    prompt = tokens(21, 77, 3)
    want = greedy(cfg, w, prompt, 5)
    for pad in (0, 1):  # the data section at an even and at an odd address
        U.write_safetensors(path, w, pad=pad)
        eng = p.load_model(backend, str(tmp_path), dtype="float32", max_seq=64)
        assert eng.generate(prompt, 5).tolist() == want
        eng.close()
    out = subprocess.run([sys.executable, "-m", "prism_engine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                          "--prompt", ",".join(map(str, prompt)), "--max-new", "5"], capture_output=True, text=True, cwd=ROOT, check=True)
    assert [int(t) for t in out.stdout.split()] == want
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[20:], "want": [0]}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": prompt[:3], "want": []}], "end": ["y"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "32"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, check=True)
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = orc.forward(cfg, w, prompt)
    assert U.error(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 77), ref[[0, 19]]) < U.TOL["float32"]
    assert U.error(np.fromfile(tmp_path / "1.f32", "<f4").reshape(1, 77), ref[[20]]) < U.TOL["float32"]
    assert not (tmp_path / "2.f32").exists()
    U.write_safetensors(path, w, dtype="F16")
    with pytest.raises(p.PrismCudaError, match="expected BF16"):
        p.load_model(backend, str(tmp_path))
    U.write_safetensors(path, {k: v for k, v in w.items() if k != "head"})
    with pytest.raises(p.PrismCudaError, match="head"):
        p.load_model(backend, str(tmp_path))
    (tmp_path / "model.safetensors").write_bytes(b"\xff" * 40)
    with pytest.raises(p.PrismCudaError, match="safetensors"):
        p.load_model(backend, str(tmp_path))
