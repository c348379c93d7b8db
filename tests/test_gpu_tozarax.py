"""Sequential layers (Tozarax) on the GPU against the plain restatement (oracle/layered.py): each mechanism alone,
portions, decoding, batches, slots, window and chunk edges, routing, generation, loading, command line."""
import ctypes as C
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
MOE = U.moe(6, 2, 24, (3, 2))


def tokens(n, vocab, seed=0):
    return np.random.default_rng([12, seed]).integers(0, vocab, n).tolist()


def compare(be, cfg, w, toks, portions, dtype, **kw):
    want = U.expected(cfg, w, toks, dtype)
    eng = U.engine(be, cfg, w, dtype, max_seq=len(toks), **kw)
    try:
        for sizes in portions:
            err = U.error(U.run_portions(eng, toks, list(sizes)), want)
            assert err < U.TOL[dtype], (sizes, err)
    finally:
        eng.close()


def weights_for(cfg, dtype, seed):
    """Independent experts in 32-bit; in bf16 similar ones, for a choice may fall either way when scores almost meet."""
    return U.sequential_weights(cfg, seed, apart=1.0 if dtype == "float32" else 0.02)


def check(be, cfg, n, portions, dtype, seed=0, without=(), **kw):
    w = weights_for(cfg, dtype, seed)
    for name in w:
        if any(name.endswith(x) for x in without):
            w[name] = 0.0 * w[name]
    compare(be, cfg, w, tokens(n, cfg["vocab"], seed), portions, dtype, **kw)


WHOLE_AND_STEPS = [(10 ** 9,), (50, 1), (9, 40, 2)]
ATTENTION = [
    U.attention(4, 2, 16, 24, window=20), U.attention(1, 1, 8, 8), U.attention(3, 3, 20, 12, window=1, scale=0.7),
    U.attention(6, 1, 7, 13, window=33),                      # nothing a multiple of 8, an odd value size
    U.attention(12, 1, 24, 40, window=2),                     # more query heads per key head than go together
    U.attention(8, 2, 40, 64, window=65), U.attention(2, 1, 136, 200, window=64), U.attention(5, 5, 256, 256, window=70),
    U.attention(2, 2, 264, 16, window=50), U.attention(2, 1, 16, 300, window=90), U.attention(4, 1, 9, 6)]
DELTA = [
    U.delta(2, 1, 16, 24), U.delta(1, 1, 8, 8, conv=1), U.delta(4, 2, 20, 36, conv=2), U.delta(3, 3, 7, 13, conv=5), U.delta(2, 2, 64, 32, conv=4),
    U.delta(6, 2, 128, 40), U.delta(1, 1, 136, 64, conv=9), U.delta(2, 1, 200, 33), U.delta(1, 1, 256, 64), U.delta(1, 1, 272, 24, conv=4),
    U.delta(2, 2, 24, 300)]
TINY_A, TINY_D = U.attention(1, 1, 8, 8, window=5), U.delta(1, 1, 8, 8)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(ATTENTION)))
def test_attention_alone(backend, dtype, i):
    cfg = U.tozarax([U.pair(ATTENTION[i], TINY_D)], width=40 + 8 * i)
    check(backend, cfg, 150, WHOLE_AND_STEPS, dtype, seed=i, without=["right.out"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(DELTA)))
def test_gated_delta_alone(backend, dtype, i):
    cfg = U.tozarax([U.pair(TINY_A, DELTA[i])], width=40 + 8 * i)
    check(backend, cfg, 150, WHOLE_AND_STEPS, dtype, seed=i, without=["left.out"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decay", [-9.0, 0.0, 2.5, 6.0])
def test_decays_from_almost_one_to_nothing(backend, dtype, decay):
    """From a state that lasts for the whole sequence to one that is gone at the next token."""
    cfg = U.tozarax([U.pair(TINY_A, U.delta(2, 2, 24, 40, conv=4))], width=64)
    w = weights_for(cfg, dtype, 3)
    w["l0.mix.right.A_log"] = U.round_bf16(np.array([decay, decay - 0.5]))[1]
    w["l0.mix.left.out"] *= 0.0
    compare(backend, cfg, w, tokens(200, 131, 3), WHOLE_AND_STEPS + [(64,), (63, 2, 65)], dtype)


MOES = [U.moe(1, 1, 8), U.moe(5, 5, 20), U.moe(8, 3, 40, (2, 1)), U.moe(12, 2, 33, (6, 2)), U.moe(40, 7, 24, (4, 3)), U.moe(6, 2, 200, (6, 6)),
        U.moe(130, 9, 16, (10, 4)), U.moe(3, 2, 130, (3, 2))]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(MOES)))
def test_experts_alone(backend, dtype, i):
    cfg = U.tozarax([U.pair(TINY_A, TINY_D, MOES[i])], width=40 + 8 * i)
    check(backend, cfg, 120, WHOLE_AND_STEPS + [(4, 8, 7)], dtype, seed=20 + i, without=["left.out", "right.out"])


def _clear_choices(cfg, w, n, margin, seed):
    """Token ids whose choices (groups and experts) stand out by `margin` at every place; layer 0, mixers silent."""
    mlp, eps, taps = cfg["layers"][0]["mlp"], cfg["norm"]["eps"], cfg["canon"]["taps"]
    r, g = mlp["router"], mlp["router"]["groups"]
    per = r["experts"] // g["count"]
    rng, out, hs = np.random.default_rng(seed), [], []
    while len(out) < n:
        tok = int(rng.integers(cfg["vocab"]))
        h = orc.rms_norm(w["embed"][tok].astype(np.float64) + w["pos"][len(out)], 1.0 + w["l0.norm2"], eps)
        x = h + orc.causal_conv(np.stack((hs + [h])[-taps:]), w["l0.canon2"])[-1]
        z = w["l0.mlp.router"] @ x
        choice = orc.sigmoid(z) + w["l0.mlp.correction"]
        score = np.sort(np.sort(choice.reshape(g["count"], -1), axis=1)[:, -2:].sum(axis=1))[::-1]
        chosen, _ = orc.route(z, w["l0.mlp.correction"], r["top"], g)
        all_kept, _ = orc.route(z, w["l0.mlp.correction"], per * g["keep"], g)
        rest = [choice[e] for e in all_kept if e not in chosen]
        if score[g["keep"] - 1] - score[g["keep"]] < margin or min(choice[chosen]) - max(rest) < margin:
            continue
        out.append(tok)
        hs.append(h)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i,correction", [(0, 0.0), (1, 1.0), (2, -3.0)])
def test_choice_of_experts(backend, dtype, i, correction):
    """Independent experts, choices that stand out: a wrong expert, weight or group would show.  Corrections of all
    sizes, also ones that make every choice score negative."""
    cfg = U.tozarax([U.pair(TINY_A, TINY_D, U.moe(16, 3, 24, (4, 2)))], width=64)
    w = U.sequential_weights(cfg, 30 + i, apart=1.0)
    for name in ("left", "right"):
        w[f"l0.mix.{name}.out"] *= 0.0
    w["l0.mlp.correction"] = U.round_bf16(np.random.default_rng(i).normal(correction, abs(correction) / 3, 16))[1]
    toks = _clear_choices(cfg, w, 90, 0.03, i)
    want = orc.forward(cfg, w, toks)
    # what the choice is worth: experts by score alone, or all groups open
    free = json.loads(json.dumps(cfg))
    free["layers"][0]["mlp"]["router"]["groups"]["keep"] = 4
    assert U.error(orc.forward(free, w, toks), want) > 5 * U.TOL[dtype]
    if correction:
        plain = dict(w, **{"l0.mlp.correction": 0 * w["l0.mlp.correction"]})
        assert U.error(orc.forward(cfg, plain, toks), want) > 5 * U.TOL[dtype]
    compare(backend, cfg, w, toks, WHOLE_AND_STEPS + [(8, 3, 1)], dtype)


@pytest.mark.parametrize("rows", [9, 17, 40, 100, 129, 200, 300, 520])
@pytest.mark.parametrize("ff", [72, 512])
def test_row_tiles_of_the_expert_gemm(backend, rows, ff):
    """One and several row tiles per expert, few and many rows each, independent experts, some of them without a row."""
    cfg = U.tozarax([U.pair(TINY_A, TINY_D, U.moe(12, 3, ff, (4, 2)))], width=256)
    w = U.sequential_weights(cfg, rows, apart=1.0)
    for name in ("left", "right"):
        w[f"l0.mix.{name}.out"] *= 0.0
    w["l0.mlp.correction"] = U.round_bf16(np.linspace(-0.4, 0.4, 12))[1]
    compare(backend, cfg, w, _clear_choices(cfg, w, rows, 0.02, rows), [(10 ** 9,)], "bfloat16")


# ---- around the sublayers ----------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_input_convolution(backend, dtype, taps):
    cfg = U.tozarax([U.pair(U.attention(2, 1, 8, 8, window=9), U.delta(1, 1, 8, 8, conv=2), MOE)] * 2, width=72, taps=taps)
    w = weights_for(cfg, dtype, taps)
    toks = tokens(60, 131, taps)
    want = orc.forward(cfg, w, toks)
    for name in ("canon1", "canon2"):  # each of them counts
        lost = dict(w, **{f"l1.{name}": 0 * w[f"l1.{name}"]})
        assert U.error(orc.forward(cfg, lost, toks), want) > 2 * U.TOL[dtype]
    compare(backend, cfg, w, toks, [(10 ** 9,), (1,), (2,), (3, 5), (17, 1), (16, 40)], dtype)


def test_gate_position_and_depth_average_count(backend):
    """Dropping any one of them changes the restatement's logits by far more than the 32-bit tolerance, which the
    engine meets with all of them; every width and constant differs from the other tests."""
    cfg = U.tozarax([U.pair(TINY_A, TINY_D, MOE), U.pair(TINY_A, TINY_D), U.pair(TINY_A, TINY_D, MOE)], width=52, eps=0.2, vocab=67, max_positions=80)
    w = U.sequential_weights(cfg, 4, apart=1.0)
    toks = tokens(80, 67, 4)
    want = orc.forward(cfg, w, toks)
    for name in ("pos", "l0.rg1", "l0.rg1.b", "l2.rg2", "l2.rg2.b", "l0.dwa", "l1.dwa", "l2.dwa", "l1.norm1", "l2.norm2", "final.norm"):
        if name.endswith("dwa"):  # only the layer's own result goes on
            lost = dict(w, **{name: np.eye(len(w[name]))[-1]})
        else:
            lost = dict(w, **{name: 0 * w[name]})
        assert U.error(orc.forward(cfg, lost, toks), want) > 1e-2, name
    for dtype in DTYPES:
        compare(backend, cfg, weights_for(cfg, dtype, 4), toks, [(10 ** 9,), (70, 1), (7, 2)], dtype)


def mixed(width=88, vocab=210, max_positions=600):
    """Every layer other sizes; with and without feed-forward, windows shorter and longer than a tile, none."""
    return U.tozarax([
        U.pair(U.attention(4, 2, 16, 24, window=21), U.delta(2, 1, 24, 16, conv=4), U.moe(8, 2, 40, (4, 2))),
        U.pair(U.attention(3, 1, 8, 40), U.delta(4, 4, 8, 24, conv=2)),
        U.pair(U.attention(2, 2, 24, 8, window=70), U.delta(3, 3, 40, 32, conv=3), U.moe(5, 3, 72))],
        width=width, vocab=vocab, max_positions=max_positions)


PORTIONS = [(1,), (2,), (3, 2), (5, 7, 2), (9,), (16, 1), (17, 2, 33), (63, 1, 1, 65), (64,), (65, 3), (100, 1), (140, 2, 2, 1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", PORTIONS)
def test_portions(backend, dtype, sizes):
    check(backend, mixed(), 180, [sizes], dtype, seed=5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 2, 7, 32, 64])
def test_small_rings(backend, dtype, chunk):
    """Short prefill chunks: windowed caches hold window - 1 + chunk positions and wrap many times."""
    check(backend, mixed(), 200, [(50, 3, 1, 1, 1, 90, 1)], dtype, seed=6, chunk=chunk)


@pytest.mark.parametrize("dtype", DTYPES)
def test_cut_independence(backend, dtype):
    """The same tokens in other portions, after other sequences, in another slot."""
    cfg, n = mixed(), 150
    w, toks = weights_for(cfg, dtype, 7), tokens(150, 210, 7)
    base = U.expected(cfg, w, toks, dtype)
    eng = U.engine(backend, cfg, w, dtype, max_seq=n, max_batch=3)
    assert U.error(U.run_portions(eng, toks, [n]), base) < U.TOL[dtype] / 2
    hold = eng.open_sequence()  # the next sequence gets another slot
    eng.extend([(hold, tokens(60, 210, 8), [])])
    for sizes in ([1], [2], [31, 2, 1], [149, 1]):
        assert U.error(U.run_portions(eng, toks, sizes), base) < U.TOL[dtype] / 2, sizes
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(backend, dtype):
    """Prompts of several lengths and decode rows in the same steps against each request alone; slots are reused."""
    cfg = mixed()
    w = weights_for(cfg, dtype, 9)
    lens = [1, 2, 19, 40, 64, 97, 33, 5, 80, 23, 50, 12]
    reqs = [tokens(n + 6, cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    want = [U.expected(cfg, w, r, dtype) for r in reqs]
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


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [2, 5, 8, 20])
def test_decode_batches(backend, dtype, B):
    """Several sequences decode together: the small-batch kernels with experts shared by some rows, and the sorted plan."""
    cfg = mixed()
    w = weights_for(cfg, dtype, 10)
    reqs = [tokens(30 + i, cfg["vocab"], 60 + i) for i in range(B)]
    want = [U.expected(cfg, w, r, dtype) for r in reqs]
    eng = U.engine(backend, cfg, w, dtype, max_seq=64, max_batch=B)
    seqs = [eng.open_sequence() for _ in range(B)]
    eng.extend([(s, r[:-6], []) for s, r in zip(seqs, reqs)])
    for k in range(6):  # eager, captured, replayed
        lg = eng.extend([(s, [r[len(r) - 6 + k]], [0]) for s, r in zip(seqs, reqs)])
        for i in range(B):
            assert U.error(lg[i:i + 1], want[i][len(reqs[i]) - 6 + k][None]) < 1.5 * U.TOL[dtype], (B, k, i)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes_and_wanted_places_in_any_order(backend, dtype):
    cfg = U.tozarax([U.pair(U.attention(3, 3, 10, 7, window=11), U.delta(3, 1, 9, 5, conv=2), U.moe(7, 2, 37)),
                     U.pair(U.attention(5, 1, 11, 14), U.delta(1, 1, 5, 3, conv=6))], width=45, vocab=101, taps=2)
    check(backend, cfg, 90, [(33, 2, 1)], dtype, seed=17)
    w, toks = weights_for(cfg, dtype, 18), tokens(40, 101, 18)
    want = U.expected(cfg, w, toks, dtype)
    eng = U.engine(backend, cfg, w, dtype, max_seq=64, chunk=16)  # the places fall into several chunks
    s = eng.open_sequence()
    places = [38, 3, 3, 17, 16, 0, 30]
    assert U.error(eng.extend([(s, toks[:39], places)]), want[places]) < U.TOL[dtype]
    assert U.error(eng.extend([(s, toks[39:], [0, 0])]), want[[39, 39]]) < U.TOL[dtype]
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_rows_shared_by_a_cluster(backend, dtype):
    """A width at which several CTAs share a row of the row-wise kernel."""
    cfg = U.tozarax([U.pair(U.attention(4, 2, 32, 32, window=30), U.delta(2, 2, 32, 32), U.moe(4, 2, 96))], width=2056, vocab=64)
    check(backend, cfg, 40, [(10 ** 9,), (30, 1), (3,)], dtype, seed=40)


def test_unfused_path_agrees(backend):
    """Option fuse = 0: the tensor-core GEMM at every size, one row included, and the sorted plan of the experts."""
    backend.set_option("fuse", 0)
    try:
        check(backend, mixed(), 60, [(20, 1, 2)], "bfloat16", seed=12)
    finally:
        backend.set_option("fuse", 1)


# ---- the parts in another design -----------------------------------------------------------------------------

def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


OTHER = [
    U.sequential([layer("attention", U.attention(4, 2, 16, 24, window=9)), layer("gated_delta", U.delta(2, 1, 16, 24), {"kind": "dense", "ff": 56})]),
    U.sequential([U.lightning(2, 16, 24), U.latent(2, 16, 8, 16, 24, 32, window=12)], width=56, norm_offset=0.5, canon_taps=2),
    U.sequential([layer("attention", U.attention(2, 2, 8, 8), U.moe(4, 2, 24)), U.lightning(1, 8, 16, ff=40)], gated_residual=True, depth_average=True),
    U.sequential([layer("gated_delta", U.delta(2, 2, 8, 12), U.moe(5, 1, 16)), U.pair(TINY_A, TINY_D)], norm_offset=1.0, max_positions=200,
                 gated_residual=True, canon_taps=4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("i", range(len(OTHER)))
def test_parts_in_other_designs(backend, dtype, i):
    check(backend, OTHER[i], 100, WHOLE_AND_STEPS, dtype, seed=50 + i)


# ---- keys that stand out ---------------------------------------------------------------------------------

def _spiked(window, dim=16, heads=4, kv_heads=2):
    """One layer in which the query of the filler token strongly prefers the key of one other token, whatever the
    distance; everything but the attention is silent.  Returns (config, weights, filler, special)."""
    cfg = U.tozarax([U.pair(U.attention(heads, kv_heads, dim, 12, window=window, scale=2.5), TINY_D)], width=64, vocab=97, max_positions=500)
    w = U.sequential_weights(cfg, 31)
    for name in ("pos", "l0.canon1", "l0.mix.right.out"):
        w[name] = 0 * w[name]
    h = orc.rms_norm(w["embed"].astype(np.float64), 1.0 + w["l0.norm1"], 1e-5)
    q = (h @ w["l0.mix.left.q"].T).reshape(97, kv_heads, heads // kv_heads, dim)
    k = (h @ w["l0.mix.left.k"].T).reshape(97, kv_heads, dim)
    s = np.einsum("agnd,bgd->abgn", q, k) * 2.5
    gain = (s - np.einsum("aagn->agn", s)[:, None]).min(axis=(2, 3))  # how much filler a prefers b over itself, in every head
    a, b = np.unravel_index(np.argmax(gain), gain.shape)
    assert gain[a, b] > 6.0
    return cfg, w, int(a), int(b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 264])
@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100, 129])
def test_window_edges(backend, dtype, dim, window):
    """The last token that sees the special key and the first that does not, in prompts and decoded, with the
    special token at several places relative to tiles, portions and the ring."""
    cfg, w, fill, special = _spiked(window, dim, *((4, 2) if dim == 16 else (2, 2)))
    wrong = json.loads(json.dumps(cfg))
    for place in (0, 1, 37, 64):
        n = place + window + 3
        toks = [fill] * n
        toks[place] = special
        want = U.expected(cfg, w, toks, dtype)
        if window > 1:  # the edge shows: a window one token off is far outside the tolerance
            for off, pos in ((-1, place + window - 1), (1, place + window)):
                wrong["layers"][0]["mixer"]["left"]["mask"]["size"] = window + off
                assert U.error(U.expected(wrong, w, toks, dtype)[pos:pos + 1], want[pos:pos + 1]) > 5 * U.TOL[dtype]
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
    compare(backend, cfg, w, toks, [(n,), (300, 1), (130, 5, 200, 2)], dtype, chunk=128)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_state_reaches_far(backend, dtype):
    """Hardly any decay, and later tokens that hardly write: what the first tokens left is read hundreds of tokens on,
    over chunk edges and portions; a lost state shows in the oracle by far more than the tolerance."""
    cfg = U.tozarax([U.pair(TINY_A, U.delta(2, 2, 16, 24, conv=2))], width=64, max_positions=400)
    w = U.sequential_weights(cfg, 41)
    for name in ("pos", "l0.canon1", "l0.mix.left.out"):
        w[name] = 0 * w[name]
    w["l0.mix.right.A_log"] = np.full(2, -10.0, np.float32)
    h = orc.rms_norm(w["embed"][5].astype(np.float64), 1.0 + w["l0.norm1"], 1e-5)
    w["l0.mix.right.b"] = U.round_bf16(w["l0.mix.right.b"] - np.outer(w["l0.mix.right.b"] @ h + 9.0, h) / (h @ h))[1]
    n = 330
    toks = tokens(20, 131, 1) + [5] * (n - 20)
    want = orc.forward(cfg, w, toks)
    lost = orc.forward(cfg, w, toks[20:])
    assert U.error(lost[-1:], want[-1:]) > 5 * U.TOL[dtype]
    compare(backend, cfg, w, toks, [(n,), (64,), (63, 65, 2, 1), (20, 1), (300, 1)], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_replaces_what_a_key_held(backend, dtype):
    """The same keys written again and again with full step size: the state holds the last value, not the sum, which a
    linear attention would give.  The keys repeat inside and across the chunks of 64."""
    cfg = U.tozarax([U.pair(TINY_A, U.delta(1, 1, 16, 24, conv=1))], width=64, max_positions=400)
    w = U.sequential_weights(cfg, 43)
    for name in ("pos", "l0.canon1", "l0.mix.left.out"):
        w[name] = 0 * w[name]
    w["l0.mix.right.A_log"] = np.full(1, -10.0, np.float32)
    w["l0.mix.right.b"] *= 0.0
    w["l0.mix.right.b"][:, 0] = 40.0                                    # step size 1 ..
    w["embed"][:, 0] = U.round_bf16(np.abs(w["embed"][:, 0]) + 1.0)[1]  # .. for every token
    w["l0.norm1"][0] = 0.0
    toks = np.tile(tokens(3, 131, 5), 70).tolist()
    compare(backend, cfg, w, toks, [(10 ** 9,), (64, 1, 70), (100, 1)], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_start_empty(backend, dtype):
    """A reused slot carries nothing over: same logits as on a fresh engine, bit for bit."""
    cfg = mixed()
    w, toks = weights_for(cfg, dtype, 13), tokens(60, 210, 13)
    eng = U.engine(backend, cfg, w, dtype, max_seq=128, max_batch=2)
    first = U.run_portions(eng, toks, [40, 1])
    for seed in (1, 2, 3):
        U.run_portions(eng, tokens(100, 210, seed), [50])
        assert np.array_equal(U.run_portions(eng, toks, [40, 1]), first)
    for n in (1, 2):  # the very first tokens, right after another sequence
        U.run_portions(eng, tokens(100, 210, 4), [50, 1])
        assert U.error(U.run_portions(eng, toks[:n], [n]), U.expected(cfg, w, toks[:n], dtype)) < U.TOL[dtype]
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(backend, dtype):
    cfg = mixed(vocab=61)
    compare(backend, cfg, weights_for(cfg, dtype, 14), tokens(400, 61, 14), [(5, 1)], dtype, chunk=16)


# ---- entry points ------------------------------------------------------------------------------------------

def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(orc.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


def test_generate_batch_and_steps(backend):
    cfg = mixed(vocab=90)
    w = U.sequential_weights(cfg, 15, apart=1.0)
    prompts = [tokens(25, 90, 70 + i) for i in range(3)]
    want = [greedy(cfg, w, q, 12) for q in prompts]
    eng = U.engine(backend, cfg, w, "float32", max_seq=64, max_batch=3)
    assert eng.generate(prompts, 12).tolist() == want
    assert eng.generate(prompts[1], 12).tolist() == want[1]
    eng.reset(2)  # step() and decode() drive the same loop
    for t in range(24):
        eng.step([prompts[0][t], prompts[2][t]])
    nxt = eng.step([prompts[0][24], prompts[2][24]])
    rest = eng.decode(nxt, 5)
    assert [[int(a)] + b.tolist() for a, b in zip(nxt, rest)] == [want[0][:6], want[2][:6]]
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

    cfg = mixed(max_positions=40)
    w = U.sequential_weights(cfg)
    with pytest.raises(p.PrismCudaError, match="position table"):
        U.engine(backend, cfg, {}, max_seq=41)
    lacking = {k: v for k, v in w.items() if k != "l2.mlp.e4.down"}
    eng = U.engine(backend, cfg, lacking, max_seq=40)
    with pytest.raises(p.PrismCudaError, match="l2.mlp.e4.down"):
        eng.generate([1, 2], 1)
    eng.set_tensor("l1.norm2", U.bits(w["l0.norm1"]))  # of a layer without feed-forward: taken, not needed
    for bad in ("l2.mlp.e5.down", "l1.mlp.router", "l0.mlp.up"):
        with pytest.raises(p.PrismCudaError, match="miss"):
            eng.set_tensor(bad, U.bits(w["l0.norm1"]))
    with pytest.raises(p.PrismCudaError, match="needs"):
        eng.set_tensor("l0.canon1", U.bits(w["l0.canon1"].T))
    eng.set_tensor("l2.mlp.e4.down", U.bits(w["l2.mlp.e4.down"]))
    s = eng.open_sequence()
    with pytest.raises(p.PrismCudaError, match="max_seq"):
        eng.extend([(s, [1] * 41, [])])
    assert eng.extend([(s, [1] * 40, [39])]).shape == (1, 210)
    eng.close()
    for field, value in (("expert_groups", 3), ("top", 9), ("groups_keep", 5)):
        mc, arr, keep = p.LayeredConfig.from_dict(cfg).to_c("float32", 8, 1)
        setattr(arr[0], field, value)
        h = C.c_void_p()
        assert backend.L.prism_cuda_engine_create_layered(backend.ctx, C.byref(mc), arr, C.byref(h)) == -2 and not h
        del keep


def test_loading_generation_and_trace_from_a_folder(backend, tmp_path):
    """safetensors + config.json through the registry, the command line and the trace replay."""
    import prism_engine_b200 as p

    cfg = mixed(vocab=77, max_positions=48)
    w = U.sequential_weights(cfg, 16, apart=1.0)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    U.write_safetensors(str(tmp_path / "model.safetensors"), w)
    prompt = tokens(21, 77, 3)
    want = greedy(cfg, w, prompt, 5)
    eng = p.load_model(backend, str(tmp_path), dtype="float32")  # the position table bounds the sequence length
    assert eng.generate(prompt, 5).tolist() == want
    eng.close()
    out = subprocess.run([sys.executable, "-m", "prism_engine_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                          "--prompt", ",".join(map(str, prompt)), "--max-new", "5"], capture_output=True, text=True, cwd=ROOT, check=True)
    assert [int(t) for t in out.stdout.split()] == want
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": prompt[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": prompt[20:], "want": [0]}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": prompt[:3], "want": []}], "end": ["y"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, check=True)
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = orc.forward(cfg, w, prompt)
    assert U.error(np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 77), ref[[0, 19]]) < U.TOL["float32"]
    assert U.error(np.fromfile(tmp_path / "1.f32", "<f4").reshape(1, 77), ref[[20]]) < U.TOL["float32"]
