"""Sipelorn on the GPU against the plain implementation (tests/plain_sipelorn.py): every mechanism alone with inputs made
so that a fault shows, then whole models through the step function in every cut (whole, a long tail decoded token by
token, portions down to two tokens, mixed batches over a pool so small that pages and slots are used again), in 32-bit
and in bfloat16, and greedy generation through the engine's entry point and scheduler."""

import os
import subprocess
import tempfile

import numpy as np
import pytest
import torch

import plain_sipelorn as plain
from replay_util import (ROOT, compare, plan_chunks, plan_many_rows, plan_mixed, plan_tail, plan_whole, random_requests,
                         run_plan_in_process, run_plan_trace_run)
from sipelorn_configs import ONE_KIND, SIPELORN

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# float32: (absolute, relative to the row's largest logit) on every logit. bfloat16: the spread of a row's difference
# against the spread of its logits, (bound of the median row, bound of every row).
TOL = {"float32": (3e-5, 3e-5), "bfloat16": (0.05, 0.35)}
SPREAD = {"float32": False, "bfloat16": True}
LENGTHS = {"sa": [5, 70, 150, 33, 210, 129], "sb": [1, 7, 64, 100, 129, 40], "sc": [3, 48, 95, 200, 16, 331]}
SIZES = [16, 7, 2, 5, 3, 2, 11, 32, 2, 9, 64, 2]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """dtype -> name -> model folder whose file holds that dtype."""
    from dynalm_b200.weights import write_model_folder
    out = {"float32": {}, "bfloat16": {}}
    for name, (cfg, seed) in SIPELORN.items():
        for dtype, t in (("float32", torch.float32), ("bfloat16", torch.bfloat16)):
            d = tmp_path_factory.mktemp(f"sipelorn_{name}_{dtype}")
            write_model_folder(str(d), cfg, seed, dtype=t)
            out[dtype][name] = str(d)
    return out


@pytest.fixture(scope="module")
def plain_logits(folders):
    made = {}

    class Lookup:
        def __getitem__(self, key):
            name, dtype = key
            if key not in made:
                reqs = random_requests(SIPELORN[name][0]["vocab"], LENGTHS[name], seed=271 + len(made))
                model = plain.PlainSipelorn(folders[dtype][name])
                made[key] = (reqs, {r: model.logits(t) for r, t in reqs.items()})
            return made[key]
    return Lookup()


def _built(folder, dtype, kv_tokens, max_batch, max_requests=8):
    from dynalm_b200.engine import build
    return build(folder, dtype=dtype, kv_tokens=kv_tokens, max_batch_tokens=max_batch, max_requests=max_requests,
                 context=max(kv_tokens, 256))


def _t(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV, dtype)


def _np(t):
    return t.double().cpu().numpy()


def _ints(v):
    return torch.tensor(list(v), dtype=torch.int32, device=DEV)


def _close(got, want, tol, what=""):
    err = np.abs(got - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), f"{what}: {err:.3g}"


class Batch:
    """The arrays of a step for (slot, first position, tokens) runs."""

    def __init__(self, runs):
        self.runs = runs
        self.num_requests = len(runs)
        self.num_tokens = sum(n for _, _, n in runs)
        self.positions = _ints(p + i for _, p, n in runs for i in range(n))
        self.row_request = _ints(r for r, (_, _, n) in enumerate(runs) for _ in range(n))
        self.row_slot = _ints(s for s, _, n in runs for _ in range(n))
        self.state_slots = _ints(s for s, _, _ in runs)
        self.pos_start = _ints(p for _, p, _ in runs)
        self.q_start = _ints(np.cumsum([0] + [n for _, _, n in runs]))
        self.decode_only = all(n == 1 for _, _, n in runs)


# ---------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [30, 72, 96, 512, 1001, 2048, 4096, 5000])
def test_residual_update_and_norm(dtype, width):
    """A gated result as partial sums, a result that joins normed, a plain one; both norms and none; the copy of the
    stream; the gather of wanted rows without a write; a row with a large mean."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(width)
    rows = 7
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    x0 = rng.randn(rows, width)
    x0[3] += 30.0
    w, b, gb, pw = 1 + 0.2 * rng.randn(width), 0.3 * rng.randn(width), rng.randn(width), 1 + 0.3 * rng.randn(width)
    eps = 1e-5
    x = _t(x0)
    out, copy = torch.zeros(rows, width, dtype=dtype, device=DEV), torch.zeros(rows, width, dtype=dtype, device=DEV)
    # nothing pending: the norm alone
    ops.residual_norm(x, out, "layer", _t(w), _t(b), eps)
    _close(_np(out), plain.layer_norm(x0, w, b, eps), tol, "layer norm")
    assert np.array_equal(_np(x), _np(_t(x0)))
    # a gated result in three partial sums; the gate's values lie inside wider rows
    delta = rng.randn(3, rows, width)
    wide_gate = _np(_t(3 * rng.randn(rows, width + 8), dtype))
    ops.residual_norm(x, out, "layer", _t(w), _t(b), eps, delta=_t(delta), gate=_t(wide_gate, dtype)[:, 8:], gate_bias=_t(gb), copy=copy)
    want = _np(_t(x0)) + plain.sigmoid(wide_gate[:, 8:] + gb) * delta.sum(0)
    _close(_np(x), want, 1e-5, "the stream after a gated result")
    _close(_np(copy), want, 1e-5 if dtype == torch.float32 else 1e-2, "the copy")
    _close(_np(out), plain.layer_norm(want, w, b, eps), tol, "the norm after a gated result")
    # a result that joins normed, in the compute dtype, then an RMS norm
    d2 = _np(_t(rng.randn(rows, width) * 5.0, dtype))
    ops.residual_norm(x, out, "rms", _t(w), None, eps, delta=_t(d2, dtype), post_weight=_t(pw), post_eps=0.01)
    want = want + plain.rms_norm(d2, pw, 0.01)
    _close(_np(x), want, 1e-5, "the stream after a normed result")
    _close(_np(out), plain.rms_norm(want, w, eps), tol, "the norm after a normed result")
    # the wanted rows only: nothing is written back
    pick = [5, 0, 3]
    out2, before = torch.zeros(3, width, dtype=dtype, device=DEV), x.clone()
    gate = _np(_t(rng.randn(rows, width), dtype))
    ops.residual_norm(x, out2, "layer", _t(w), _t(b), eps, delta=_t(d2, dtype), delta_scale=0.5, gate=_t(gate, dtype), rows=_ints(pick))
    assert torch.equal(x, before)
    _close(_np(out2), plain.layer_norm((want + 0.5 * plain.sigmoid(gate) * d2)[pick], w, b, eps), tol, "the gathered rows")
    # the sum alone
    ops.residual_norm(x, None, delta=_t(d2, dtype))
    _close(_np(x), want + d2, 1e-5, "a plain sum")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,K", [(4, 2, 32, 16, 4), (3, 3, 20, 12, 2), (2, 1, 8, 40, 6), (5, 1, 12, 28, 1), (2, 2, 16, 16, 0),
                                       (4, 0, 24, 8, 3)])
def test_convolutions_into_shuffled_pages_keep_their_inputs(dtype, H, G, d, e, K):
    """Two requests in different cuts side by side (single tokens, portions shorter and longer than the taps) against the
    convolution over each whole sequence; q into its own array, k and v into the token's place. The first inputs are large:
    one that is lost, kept twice or carries no bias shows. Then a slot that is used again. G = 0: queries only."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H * 100 + d + K)
    page, n_pages, slots = 8, 24, 4
    widths = (H * d, G * d, G * e)
    C = sum(widths)
    taps = rng.randn(C, K) if K else None
    bias = rng.randn(C) * 2.0
    cuts = {1: [1, 2, 9, 8, 1, 1, 33, 6], 3: [7, 1, 1, 2, 12]}
    kept = torch.zeros(slots, max(1, (K - 1) * C) + 3, device=DEV) if K > 1 else None
    table = torch.full((slots, 12), -1, dtype=torch.int32, device=DEV)
    perm = rng.permutation(n_pages)
    table[1], table[3] = _ints(perm[:12]), _ints(perm[12:])
    record = max(8, G * (d + e))
    cache = torch.zeros(n_pages, page, record, dtype=dtype, device=DEV)
    flat = cache.view(-1)
    taps_t = _t(taps.T) if K else None
    tol = 3e-5 if dtype == torch.float32 else 2e-2
    for again in range(2):
        seqs = {s: _np(_t(rng.randn(sum(c), C + 5) * 1.5, dtype)) for s, c in cuts.items()}
        for s in seqs:
            seqs[s][:2] *= 8.0
            seqs[s] = _np(_t(seqs[s], dtype))
            if kept is not None:
                kept[s].zero_()
        want = {}
        for s, u in seqs.items():
            want[s] = plain.convolve(u[:, :C] + bias, taps, np.zeros((K - 1, C)))[0] if K else u[:, :C] + bias
        at = {1: 0, 3: 0}
        for step in range(8):
            batch = Batch([(s, at[s], cuts[s][step]) for s in (3, 1) if step < len(cuts[s])])
            proj = torch.cat([_t(seqs[s][p:p + n], dtype) for s, p, n in batch.runs])
            q = torch.zeros(batch.num_tokens, H * d, dtype=dtype, device=DEV)
            ops.conv_cache(proj, widths, taps_t, _t(bias), kept, batch, table, page, q, cache if G else None, record,
                           flat[G * d:] if G else None, record)
            row = 0
            for s, p, n in batch.runs:
                _close(_np(q[row:row + n]), want[s][p:p + n, :H * d], tol, f"queries, step {step} slot {s}")
                for i in range(p, p + n) if G else ():
                    rec = _np(cache[int(table[s, i // page]), i % page])[:G * (d + e)]
                    _close(rec, want[s][i, H * d:], tol, f"keys and values, step {step} slot {s} position {i}")
                row += n
                at[s] += n
        assert kept is None or float(kept[0].abs().max()) == 0.0 and float(kept[:, (K - 1) * C:].abs().max()) == 0.0


@pytest.mark.parametrize("K", [2, 3, 4])
def test_convolutions_over_many_rows(K):
    """A step of several hundred rows (a thread walks eight of them): three requests, one of a single token in the middle of
    a thread's rows, all with kept inputs from before; then the inputs that are kept."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(K)
    H, G, d, e, page = 2, 1, 32, 16, 16
    widths = (H * d, G * d, G * e)
    C = sum(widths)
    taps, bias = rng.randn(C, K), rng.randn(C)
    runs = [(2, 5, 203), (0, 9, 1), (1, 0, 131)]
    seqs = {s: _np(_t(rng.randn(p + n, C) * 2, torch.bfloat16)) for s, p, n in runs}
    kept = torch.zeros(3, (K - 1) * C, device=DEV)
    for s, p, _ in runs:
        if p:
            kept[s] = _t(seqs[s][p - K + 1:p].ravel())
    table = _ints(rng.permutation(60)).view(3, 20)
    rec = G * (d + e)
    cache = torch.zeros(60, page, rec, dtype=torch.bfloat16, device=DEV)
    batch = Batch(runs)
    q = torch.zeros(batch.num_tokens, H * d, dtype=torch.bfloat16, device=DEV)
    proj = torch.cat([_t(seqs[s][p:p + n], torch.bfloat16) for s, p, n in runs])
    ops.conv_cache(proj, widths, _t(taps.T), _t(bias), kept, batch, table, page, q, cache, rec, cache.view(-1)[G * d:], rec)
    row = 0
    for s, p, n in runs:
        want = plain.convolve(seqs[s] + bias, taps, np.zeros((K - 1, C)))[0][p:]
        _close(_np(q[row:row + n]), want[:, :H * d], 2e-2, f"queries of slot {s}")
        pos = torch.arange(p, p + n, device=DEV)
        got = cache[table[s].long()[pos // page], pos % page]
        _close(_np(got), want[:, H * d:], 2e-2, f"keys and values of slot {s}")
        _close(_np(kept[s]).reshape(K - 1, C), seqs[s][-(K - 1):], 1e-6, f"kept inputs of slot {s}")
        row += n


def _attention_case(rng, n, H, G, d, e, dtype, page):
    """Keys and values of one request in slot 1 as records on shuffled pages, and queries that point at one key each: the
    newest, the first of the window, the one just outside it, one far away."""
    k, v = _np(_t(rng.randn(n, G, d), dtype)), _np(_t(rng.randn(n, G, e), dtype))
    n_pages = -(-n // page) + 3
    perm = rng.permutation(n_pages)
    table = torch.full((2, -(-n // page)), -1, dtype=torch.int32, device=DEV)
    cache = torch.zeros(n_pages, page, G * (d + e), dtype=dtype, device=DEV)
    for i in range(n):
        table[1, i // page] = int(perm[i // page])
        cache[int(perm[i // page]), i % page] = _t(np.concatenate([k[i].ravel(), v[i].ravel()]), dtype)
    return k, v, table, cache


def _pointed_queries(rng, k, H, positions, window, dtype, strength):
    q = rng.randn(len(positions), H, k.shape[2]) * 0.3
    for i, p in enumerate(positions):
        j = [p, p - window + 1, p - window, p - 64, p // 2, 0][i % 6] if window else [p, p // 2, 0, p - 64, p - 63, 1][i % 6]
        if 0 <= j <= p:
            for h in range(H):
                kk = k[j, h // (H // k.shape[1])]
                q[i, h] += kk * (strength / max(1e-6, (kk ** 2).sum()))
    return _np(_t(q, dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,window", [(4, 2, 32, 16, 20), (3, 3, 20, 12, 64), (5, 1, 12, 28, 0), (4, 1, 64, 64, 100), (2, 2, 200, 8, 33)])
def test_plain_attention_with_a_distance_bias(dtype, H, G, d, e, window):
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H * 10 + d)
    n, page = 530, 16
    k, v, table, cache = _attention_case(rng, n, H, G, d, e, dtype, page)
    rate, step = rng.rand(H) * 1.5 + 0.1, rng.rand(H) * 2 + 0.05
    positions = sorted({0, 1, 2, 15, 16, 17, 63, 64, 65, 99, 100, 101, 130, 255, 256, 511, 512, 513, 529})
    q = _pointed_queries(rng, k, H, positions, window, dtype, 12.0)
    out = torch.zeros(len(positions), H * e, dtype=dtype, device=DEV)
    rec = G * (d + e)
    ops.paged_attention_generic_kv(_t(q.reshape(len(positions), H * d), dtype), cache, rec, cache.view(-1)[G * d:], rec, table,
                                   _ints(positions), _ints([1] * len(positions)), out, H, G, d, e, page, 0.9, window,
                                   rate=_t(rate), step=_t(step))
    want = plain.attend(q, k, v, positions, list(range(n)), 0.9, window, rate, step)
    _close(_np(out).reshape(-1, H, e), want, 3e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("gated", [False, True])
@pytest.mark.parametrize("H,G,d,e,window", [(4, 2, 32, 16, 20), (8, 2, 48, 48, 0), (4, 4, 64, 64, 100), (6, 2, 64, 32, 37), (2, 1, 128, 128, 160)])
def test_masked_flash_attention_with_a_distance_bias(H, G, d, e, window, gated):
    """Portions that begin inside key tiles, then the same rows as single tokens (heads of a key head in one tile, with the
    keys in one piece and dealt over four), with and without the output gate."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H + d + window)
    n, page = 333, 16
    k, v, table, cache = _attention_case(rng, n, H, G, d, e, torch.bfloat16, page)
    rate, step = rng.rand(H) * 1.5 + 0.1, rng.rand(H) * 2 + 0.05
    q = _pointed_queries(rng, k, H, list(range(n)), window, torch.bfloat16, 12.0)
    gate = _np(_t(rng.randn(n, H * e + 8) * 2, torch.bfloat16))
    want = plain.attend(q, k, v, list(range(n)), list(range(n)), 0.6, window, rate, step)
    if gated:
        want = want * plain.sigmoid(gate[:, 8:]).reshape(n, H, e)
    rec = G * (d + e)
    kw = dict(rate=_t(rate), step=_t(step))
    order = list(range(200, n)) + list(range(200))
    tiles = [(1, 0, 128, 200), (1, 128, 5, 328), (1, 133, 128, 0), (1, 261, 72, 128)]
    out = torch.zeros(n, H * e, dtype=torch.bfloat16, device=DEV)
    g = _t(gate[order], torch.bfloat16)[:, 8:] if gated else None
    ops.masked_flash_attention(_t(q[order].reshape(n, H * d), torch.bfloat16), cache, rec, cache.view(-1)[G * d:], rec, table,
                               _ints([x for t in tiles for x in t]), len(tiles), out, H, G, d, e, page, 0.6, window, gate=g, **kw)
    _close(_np(out).reshape(n, H, e), want[order], 2e-2, "portions")
    picked = [0, 1, 19, 20, 21, 36, 37, 38, 63, 64, 65, 99, 100, 101, 159, 160, 161, 255, 256, 300, 332]
    for parts in (1, 4):
        m = len(picked)
        out = torch.zeros(m, H * e, dtype=torch.bfloat16, device=DEV)
        scratch = torch.zeros(ops.masked_flash_partial_floats(m, H, e, parts), device=DEV) if parts > 1 else None
        g = _t(gate[picked], torch.bfloat16)[:, 8:] if gated else None
        ops.masked_flash_attention(_t(q[picked].reshape(m, H * d), torch.bfloat16), cache, rec, cache.view(-1)[G * d:], rec, table,
                                   _ints([x for i, p in enumerate(picked) for x in (1, i, 1, p)]), m, out, H, G, d, e, page, 0.6,
                                   window, one_token_tiles=True, parts=parts, partial=scratch, gate=g, **kw)
        _close(_np(out).reshape(m, H, e), want[picked], 2e-2, f"single tokens in {parts} parts")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("R,r,rot,mag", [(40, 16, 16, 1.3), (21, 6, 6, 1.0), (64, 8, 8, 1.7), (9, 0, 0, 1.0)])
def test_latent_records_and_rotated_queries_with_a_magnitude(dtype, R, r, rot, mag):
    """The record without a query latent, at positions up to 100,000: normed latent, rotated part times the magnitude; and
    the rotated part of every head's query."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(R)
    page, positions = 8, [0, 1, 7, 8, 9, 99_990, 99_991]
    rows = len(positions)
    freq = plain.yarn(700.0, rot, {"factor": 6.0, "original": 128, "fast": 16.0, "slow": 1.0})[0] if rot else np.zeros(0)
    low = _np(_t(rng.randn(rows, R + r + 3) * 3, dtype))
    w = 1 + 0.2 * rng.randn(R)
    table = torch.full((2, 99_992 // page + 1), -1, dtype=torch.int32, device=DEV)
    for i, blk in enumerate(sorted({p // page for p in positions})):
        table[1, blk] = [2, 0, 1][i % 3]
    cache = torch.zeros(3, page, R + r, dtype=dtype, device=DEV)
    f = _t(freq, torch.float64) if rot else None
    ops.latent_prep(_t(low, dtype), 0, R, r, rot, None, _t(w), 1e-5, f, _ints(positions), _ints([1] * rows), table, cache, page,
                    None, mag)
    c, kr = plain.rms_norm(low[:, :R], w, 1e-5), plain.rotate_pairs(low[:, R:R + r], positions, freq, mag)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for i, p in enumerate(positions):
        rec = _np(cache[int(table[1, p // page]), p % page])
        _close(rec, np.concatenate([c[i], kr[i]]), tol, f"record of position {p}")
    if r:
        H, d = 3, 10
        q = _np(_t(rng.randn(rows, H * (d + r)), dtype))
        out = torch.zeros(rows, H * (R + r), dtype=dtype, device=DEV)
        ops.rotate_pairs(_t(q, dtype), d + r, d, out, R + r, R, r, rot, f, _ints(positions), H, mag)
        want = plain.rotate_pairs(q.reshape(rows, H, d + r)[..., d:], positions, freq, mag)
        _close(_np(out).reshape(rows, H, R + r)[..., R:], want, tol, "queries")


@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (8, 3, 2, 1), (5, 5, 1, 1), (8, 2, 4, 2), (1, 1, 1, 1), (12, 3, 3, 3),
                                               (64, 6, 8, 3), (4, 2, 4, 2), (256, 8, 8, 4), (40, 4, 2, 1)])
def test_router_with_corrections_and_the_sum_of_two(E, top, groups, keep):
    """Sigmoid scores; corrections that are large and of both signs (choice scores far below zero in a kept group), and rows
    made so that the best expert of all sits in a group that loses by the sum of its two best."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(E * 10 + top)
    rows, per = 40, E // groups
    z = rng.randn(rows, E) * 2.0
    corr = rng.randn(E) * 0.5
    corr[: E // 2] -= 3.0
    if groups > keep and per > 1:
        z[0] = -6.0
        z[0, 0] = 6.0
        z[0, per:2 * per] = 1.5
        corr[:2 * per] = 0.0
        corr[2 * per:] = -5.0
    logits = _t(np.concatenate([z, np.full((rows, 3), 50.0)], axis=1))[:, :E]         # (rows with more behind them)
    ids = torch.zeros(rows, top, dtype=torch.int32, device=DEV)
    w = torch.zeros(rows, top, device=DEV)
    for renorm in (False, True):
        ops.moe_route(logits, top, groups, keep, 1.5, ids, w, _t(corr), "sigmoid", "top2", renorm)
        for r in range(rows):
            chosen, weights = plain.route(_np(logits[r]), _np(_t(corr)), top, groups, keep)
            assert [int(i) for i in ids[r]] == chosen, f"row {r}"
            _close(_np(w[r]), 1.5 * (weights / weights.sum() if renorm else weights), 3e-6, f"weights of row {r}")
    if groups > keep and per > 1 and keep == 1 and top <= per:
        assert 0 not in [int(i) for i in ids[0]], "the best expert's group loses"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,width,inner,rows", [(6, 2, 96, 40, 50), (4, 1, 64, 32, 7), (5, 5, 72, 17, 33), (8, 3, 256, 128, 300),
                                                    (3, 2, 128, 64, 1), (16, 2, 160, 224, 130), (4, 2, 192, 320, 700)])
def test_gated_experts_and_the_shared_one(dtype, E, top, width, inner, rows):
    """Pairs grouped by expert, gate and up rows in turn in one product (every kernel that takes it), the weighted sum, and
    a shared expert's output in partial sums times the sigmoid of one number a token."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(E + width)
    x = _np(_t(rng.randn(rows, width), dtype))
    gate, up = (_np(_t(rng.randn(E, inner, width) * 0.2, dtype)) for _ in range(2))
    down = _np(_t(rng.randn(E, width, inner) * 0.2, dtype))
    ids = np.stack([rng.permutation(E)[:top] for _ in range(rows)])
    weights = rng.rand(rows, top) + 0.1
    pairs = rows * top
    shared, sz = rng.randn(2, rows, width), rng.randn(rows, 3) * 2
    want = plain.sigmoid(sz[:, 1:2]) * shared.sum(0)
    for r in range(rows):
        for k in range(top):
            j = ids[r, k]
            want[r] += weights[r, k] * plain.gated_expert(x[r], gate[j], up[j], down[j])
    w1 = _t(np.stack([gate, up], axis=2).reshape(E, 2 * inner, width), dtype)
    wide = dtype == torch.bfloat16 and width % 64 == 0 and inner % 64 == 0
    for tile_rows in ((ops.MOE_TILE_ROWS, ops.MOE_WIDE_TILE_ROWS) if wide else (ops.MOE_TILE_ROWS,)):
        place_of, pair_at = (torch.zeros(pairs, dtype=torch.int32, device=DEV) for _ in range(2))
        max_tiles = ops.moe_max_tiles(pairs, E, tile_rows)
        tiles = torch.zeros(3 * max_tiles, dtype=torch.int32, device=DEV)
        n_tiles = torch.zeros(1, dtype=torch.int32, device=DEV)
        ops.moe_group(_ints(ids.reshape(-1)), pairs, E, place_of, pair_at, tiles, n_tiles, tile_rows)
        act = torch.zeros(pairs, inner, dtype=dtype, device=DEV)
        ops.moe_linear(_t(x, dtype), pair_at, top, w1, act, tiles, n_tiles, max_tiles, "pairs", tile_rows)
        ways = [act]
        if tile_rows == ops.MOE_WIDE_TILE_ROWS and ops.moe_linear_tcgen05_applies(_t(x, dtype), w1, act, "pairs"):
            rows_sorted = torch.zeros(pairs, width, dtype=dtype, device=DEV)
            ops.moe_gather(_t(x, dtype), pair_at, top, rows_sorted)
            act2 = torch.zeros(pairs, inner, dtype=dtype, device=DEV)
            ops.moe_linear_tcgen05(rows_sorted, w1, act2, tiles, n_tiles, max_tiles, "pairs")
            assert ops.gemm_tcgen05_status() == 0
            ways.append(act2)
        for i, a in enumerate(ways):
            out = torch.zeros(pairs, width, device=DEV)
            ops.moe_linear(a, None, 1, _t(down, dtype), out, tiles, n_tiles, max_tiles, "none", tile_rows)
            y = torch.zeros(rows, width, dtype=dtype, device=DEV)
            ops.moe_combine(out, place_of, _t(weights), top, y, _t(shared), _t(sz)[:, 1:2])
            _close(_np(y), want, 3e-5 if dtype == torch.float32 else 3e-2, f"experts, tiles of {tile_rows}, way {i}")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,inner", [(1, 96, 40), (5, 256, 136), (12, 512, 128), (40, 72, 33), (300, 256, 1024), (700, 512, 2048)])
def test_xielu_behind_the_product(dtype, rows, width, inner):
    """xIELU of a product over few rows and over many, with inputs on both sides of zero, near it and far below it."""
    from dynalm_b200.engine.runtime import Runtime
    from dynalm_b200.kernels.gemm import linear_xielu
    rng = np.random.RandomState(rows)
    x = _np(_t(rng.randn(rows, width), dtype))
    w = _np(_t(rng.randn(inner, width) * 0.2, dtype))
    w[0] *= 4.0
    w[1] *= 1e-4
    w = _np(_t(w, dtype))
    p, q = 0.4, -1.1
    coeffs = _t([plain.softplus(p), 0.5 + plain.softplus(q)])
    rt = Runtime(DEV, dtype, max_tokens=rows)
    got = _np(linear_xielu(_t(x, dtype), _t(w, dtype), rt, inner, coeffs))
    want = plain.xielu(x @ w.T, p, q)
    err = np.abs(got - want) / (1.0 + np.abs(want))
    assert err.max() <= (6e-5 if dtype == torch.float32 else 1.5e-2), err.max()
    assert np.abs(got[:, 1] - want[:, 1]).max() <= 1e-2 * np.abs(want[:, 1]).max() + 5e-7, "near zero"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 70, 1024])
def test_a_table_of_token_pairs_keeps_the_last_token(dtype, width):
    """First tokens, portions, single tokens and a slot used again, with multipliers whose products leave 32 bits."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(width)
    vocab, table = 300, {"buckets": 97, "mul_prev": 1 << 31, "mul_cur": 987_654_321}
    emb, pairs = _np(_t(rng.randn(vocab, width), dtype)), _np(_t(rng.randn(98, width), dtype))
    state = torch.zeros(4, 1, dtype=torch.int32, device=DEV)
    state[2] = 77
    cuts = {1: [1, 2, 9, 1, 1, 5], 3: [7, 1, 1, 2]}
    for again in range(2):
        seqs = {s: [int(t) for t in rng.randint(0, vocab, sum(c))] for s, c in cuts.items()}
        rows = {s: plain.bigram_rows(t, None, table) for s, t in seqs.items()}
        at = {1: 0, 3: 0}
        for step in range(6):
            batch = Batch([(s, at[s], cuts[s][step]) for s in (3, 1) if step < len(cuts[s])])
            ids = [t for s, p, n in batch.runs for t in seqs[s][p:p + n]]
            out = torch.zeros(len(ids), width, device=DEV)
            ops.embed_pairs(_t(emb, dtype), _t(pairs, dtype), _ints(ids), batch.positions, batch.row_request, batch.row_slot,
                            batch.q_start, state, out, 2.5, table["mul_prev"], table["mul_cur"])
            want = emb[ids] * 2.5 + pairs[[r for s, p, n in batch.runs for r in rows[s][p:p + n]]]
            _close(_np(out), want, 1e-6, f"step {step}")
            for s, _, n in batch.runs:
                at[s] += n
                assert int(state[s, 0]) == seqs[s][at[s] - 1]
    assert int(state[2, 0]) == 77


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_tokens_gate_reads_its_piece_of_the_table(dtype):
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(1)
    z, table = _np(_t(rng.randn(9, 12) * 2, dtype)), _np(_t(rng.randn(50, 36), dtype))
    ids = rng.randint(0, 50, 9)
    out = torch.zeros(9, 12, dtype=dtype, device=DEV)
    ops.token_gate(_t(z, dtype), _t(table, dtype)[:, 12:24], _ints(ids), out)
    _close(_np(out), plain.gelu_tanh(z) * table[ids, 12:24], 1e-5 if dtype == torch.float32 else 1e-2)


# ---------------------------------------------------------------------------------------------
# whole models through the step function
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SIPELORN))
def test_replay_all_cuts(name, dtype, folders, plain_logits):
    reqs, logits = plain_logits[name, dtype]
    tol = TOL[dtype]
    plans = {
        "whole": plan_whole(reqs),
        "tail48": plan_tail(reqs, 48),
        "chunks": plan_chunks(reqs, SIZES),
        "mixed": plan_mixed(reqs, seed=5),
        "mixed2": plan_mixed(reqs, seed=6, max_live=3, decode_tail=20),
    }
    for what, plan in plans.items():
        need = plan.max_live_tokens(64)          # just what the plan needs: pages of finished requests are used again
        built = _built(folders[dtype][name], dtype, need, max(need, 64), max_requests=4)
        got = run_plan_in_process(built.step_fn, plan)
        compare(plan, got, logits, tol[0], tol[1], f"{name}/{dtype}/{what}", spread=SPREAD[dtype])
        assert built.cache.free_pages == built.cache.num_pages, "pages were lost"


@pytest.mark.parametrize("name", sorted(SIPELORN))
def test_layers_follow_the_plain_implementation(name, folders, monkeypatch):
    """The residual stream behind every layer of a short prompt in 32-bit, what a layer leaves pending included."""
    import copy
    from dynalm_b200.engine import launch_memo
    monkeypatch.setattr(launch_memo, "ENABLED", False)
    reqs = random_requests(SIPELORN[name][0]["vocab"], [29], seed=2)
    toks = reqs["r0"]
    _, layers = plain.PlainSipelorn(folders["float32"][name]).logits(toks, layers=True)
    built = _built(folders["float32"][name], "float32", 64, 64, max_requests=1)
    seen = []
    for blk in built.model.blocks:
        def fwd(stream, ctx, cache, owns, orig=blk.forward):
            s = orig(stream, ctx, cache, owns)
            c = copy.copy(s)
            c.x = s.x.clone()
            seen.append(_np(c.flush()[:len(toks)]))
            return s
        blk.forward = fwd
    run_plan_in_process(built.step_fn, plan_whole(reqs))
    assert len(seen) == len(layers)
    for i, (g, w) in enumerate(zip(seen, layers)):
        _close(g, w, 2e-5, f"layer {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_issued_by_address_equal_layers_run_through_their_parts(dtype, monkeypatch):
    """A model whose layers repeat: with the layers after the first of a kind re-issued by address (each with its own piece
    of the token table, its own gates and coefficients, the norm of the layer in front of it) the logits are bit for bit
    those of every layer run through its parts."""
    import copy
    from dynalm_b200.engine import launch_memo
    from dynalm_b200.weights import write_model_folder
    cfg = copy.deepcopy(SIPELORN["sa"][0])
    cfg["layers"] = [copy.deepcopy(cfg["layers"][i]) for i in (0, 0, 0, 4, 4, 1)]
    cfg["layers"][5]["mixer"]["kv_from"] = 1
    reqs = random_requests(cfg["vocab"], [40, 9], seed=4)
    plan = plan_chunks(reqs, [16, 3, 2])
    outs = []
    with tempfile.TemporaryDirectory() as d:
        write_model_folder(d, cfg, 5, dtype=torch.float32 if dtype == "float32" else torch.bfloat16)
        for enabled in (True, False):
            monkeypatch.setattr(launch_memo, "ENABLED", enabled)
            before = launch_memo.REPLAYED_LAYERS
            built = _built(d, dtype, 128, 64, max_requests=2)
            outs.append(run_plan_in_process(built.step_fn, plan))
            assert (launch_memo.REPLAYED_LAYERS > before) == enabled
        model = plain.PlainSipelorn(d)
        compare(plan, outs[0], {r: model.logits(t) for r, t in reqs.items()}, *TOL[dtype], "repeated layers", spread=SPREAD[dtype])
    assert all(np.array_equal(outs[0][k], outs[1][k]) for k in outs[0])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_single_token_rows_beside_a_portion(dtype, folders):
    """A couple of dozen live requests decoding beside portions of long prompts: unequal requests in one batch
    against each alone, with more state slots than the other tests use."""
    name = "sa"
    vocab = SIPELORN[name][0]["vocab"]
    short = {f"s{k}": v for k, v in random_requests(vocab, [12 + (5 * i) % 29 for i in range(20)], seed=8).items()}
    long = {f"l{k}": v for k, v in random_requests(vocab, [150, 90], seed=9).items()}
    model = plain.PlainSipelorn(folders[dtype][name])
    logits = {r: model.logits(t) for r, t in {**short, **long}.items()}
    plan = plan_many_rows(short, long, seed=3, tail_lo=4, tail_hi=10)
    built = _built(folders[dtype][name], dtype, plan.max_live_tokens(64), 256, max_requests=24)
    got = run_plan_in_process(built.step_fn, plan)
    compare(plan, got, logits, *TOL[dtype], f"{name}/{dtype}/many rows", spread=SPREAD[dtype])


@pytest.mark.parametrize("name", sorted(ONE_KIND))
def test_models_of_one_kind_of_layer(name, tmp_path):
    from dynalm_b200.weights import write_model_folder
    cfg, seed = ONE_KIND[name]
    write_model_folder(str(tmp_path), cfg, seed, dtype=torch.float32)
    reqs = random_requests(cfg["vocab"], [5, 200, 77, 130, 64], seed=3)
    model = plain.PlainSipelorn(str(tmp_path))
    logits = {r: model.logits(t) for r, t in reqs.items()}
    for what, plan in (("whole", plan_whole(reqs)), ("mixed", plan_mixed(reqs, seed=4))):
        need = plan.max_live_tokens(64)
        built = _built(str(tmp_path), "float32", need, max(need, 64), max_requests=4)
        got = run_plan_in_process(built.step_fn, plan)
        compare(plan, got, logits, *TOL["float32"], f"{name}/{what}")
        assert built.cache.free_pages == built.cache.num_pages


@pytest.mark.parametrize("name,dtype", [("sa", "float32"), ("sc", "float32"), ("sc", "bfloat16")])
def test_long_decoding_keeps_its_place(name, dtype, folders):
    """300 tokens decoded one by one after a 3-token prompt: every window passes over decoded tokens many times, a reader's
    longer window still finds its keys, and kept inputs and the last token are carried through every step (also through
    steps replayed from a captured graph)."""
    reqs = random_requests(SIPELORN[name][0]["vocab"], [303], seed=12)
    model = plain.PlainSipelorn(folders[dtype][name])
    logits = {r: model.logits(t) for r, t in reqs.items()}
    plan = plan_tail(reqs, 300)
    built = _built(folders[dtype][name], dtype, 320, 64, max_requests=2)
    got = run_plan_in_process(built.step_fn, plan)
    assert built.step_fn.graph_captures > 0 or not built.step_fn.use_graphs
    compare(plan, got, logits, *TOL[dtype], "long decoding", spread=SPREAD[dtype])
    assert built.cache.free_pages == built.cache.num_pages


def test_a_forked_request_takes_its_state_along(folders):
    """A request forked in mid-sequence continues as its parent would have: kept inputs and the last token are copied."""
    from dynalm_b200.engine import StepEntry
    name = "sa"
    toks = random_requests(SIPELORN[name][0]["vocab"], [60], seed=21)["r0"]
    other = toks[:31] + [(t + 7) % 310 for t in toks[31:]]
    model = plain.PlainSipelorn(folders["float32"][name])
    want = {"a": model.logits(toks), "b": model.logits(other)}
    sf = _built(folders["float32"][name], "float32", 256, 64, max_requests=4).step_fn
    sf.step([StepEntry("a", toks[:31], [])])
    sf.fork("a", "b")
    for lo, hi in ((31, 32), (32, 40), (40, 41), (41, 60)):
        got = _np(sf.step([StepEntry("a", toks[lo:hi], [hi - lo - 1]), StepEntry("b", other[lo:hi], [hi - lo - 1])]))
        _close(got[0], want["a"][hi - 1], 6e-5, f"parent at {hi}")
        _close(got[1], want["b"][hi - 1], 6e-5, f"child at {hi}")


def test_trace_run_replays_a_plan(folders, tmp_path):
    name = "sb"
    reqs = random_requests(SIPELORN[name][0]["vocab"], [40, 7, 90], seed=13)
    model = plain.PlainSipelorn(folders["float32"][name])
    logits = {r: model.logits(t) for r, t in reqs.items()}
    plan = plan_mixed(reqs, seed=2)
    got = run_plan_trace_run(folders["float32"][name], "float32", plan, str(tmp_path), plan.max_live_tokens(64),
                             SIPELORN[name][0]["vocab"])
    compare(plan, got, logits, *TOL["float32"], "trace_run")


# ---------------------------------------------------------------------------------------------
# generation through the entry point
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(SIPELORN))
def test_greedy_generation_through_the_engine(name, folders):
    """Decoding runs a step ahead, so the token in front of a new one is known on the device alone."""
    from dynalm_b200 import Engine
    folder = folders["float32"][name]
    model = plain.PlainSipelorn(folder)
    reqs = random_requests(SIPELORN[name][0]["vocab"], [5, 17, 33, 70], seed=14)
    eng = Engine(folder, dtype="float32", ctx=512, batch=64, max_running=4)
    outs = eng.generate(list(reqs.values()), max_tokens=12)
    for prompt, g in zip(reqs.values(), outs):
        assert g.status == "finished" and len(g.tokens) == 12
        seq = list(prompt) + list(g.tokens)
        rows = model.logits(seq[:-1])
        for i, tok in enumerate(g.tokens):
            row = rows[len(prompt) - 1 + i]
            assert row[tok] >= row.max() - 3e-5, f"token {i}: chose {tok} at {row[tok]:.6f}, best {row.max():.6f}"
    alone = [eng.generate(p, max_tokens=12).tokens for p in reqs.values()]
    assert alone == [g.tokens for g in outs]


def test_few_pages_give_the_same_tokens(folders):
    """An engine whose pool is too small for its requests preempts and recomputes (a state cannot be rewound, so a
    preempted request starts again from its first token), and gives the tokens of a roomy one."""
    from dynalm_b200 import Engine, SchedulerConfig
    name = "sa"
    reqs = list(random_requests(SIPELORN[name][0]["vocab"], [40, 90, 17, 100, 64, 33], seed=15).values())

    def run(ctx):
        eng = Engine(folders["float32"][name], dtype="float32", ctx=ctx, batch=128, max_running=8,
                     scheduler=SchedulerConfig(max_running=6, decode_token_budget=8, prefill_token_budget=64,
                                               max_prefill_chunk=32, max_batch_tokens=128))
        out = eng.generate(reqs, max_tokens=40)
        assert eng.built.cache.free_pages == eng.built.cache.num_pages
        return [g.tokens for g in out], eng.scheduler.stats.preemptions

    roomy, p0 = run(4096)
    tight, p1 = run(320)
    assert p0 == 0 and p1 > 0
    assert tight == roomy


def test_command_line_generates(folders):
    proc = subprocess.run([os.path.join(ROOT, "bin", "dynalm"), "run", folders["bfloat16"]["sa"], "--tokens", "5,9,200,31",
                           "-n", "8", "--ctx", "256", "--batch", "64", "--no-stream"], capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    ids = [int(t) for t in proc.stdout.split()]
    assert len(ids) == 8 and all(0 <= t < SIPELORN["sa"][0]["vocab"] for t in ids)
    from dynalm_b200 import Engine
    assert Engine(folders["bfloat16"]["sa"], ctx=256, batch=64).generate([5, 9, 200, 31], max_tokens=8).tokens == ids
