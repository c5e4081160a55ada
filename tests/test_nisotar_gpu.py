"""Nisotar on the GPU against the plain implementation (tests/plain_nisotar.py): every mechanism alone with inputs made
so that a fault shows, then whole models through the step function in every cut (whole, a long tail decoded token by
token, portions down to two tokens, mixed batches over a pool so small that pages and slots are used again), in 32-bit
and in bfloat16, and greedy generation through the engine's entry point and scheduler."""

import os
import subprocess
import tempfile

import numpy as np
import pytest
import torch

import plain_nisotar as plain
from replay_util import (ROOT, compare, plan_chunks, plan_many_rows, plan_mixed, plan_tail, plan_whole, random_requests,
                         run_plan_in_process, run_plan_trace_run)
from nisotar_configs import NISOTAR, ONE_KIND, write_loud_folder

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# float32: (absolute, relative to the row's largest logit) on every logit. bfloat16: the spread of a row's difference
# against the spread of its logits, (bound of the median row, bound of every row).
TOL = {"float32": (3e-5, 3e-5), "bfloat16": (0.05, 0.35)}
SPREAD = {"float32": False, "bfloat16": True}
LENGTHS = {"na": [5, 70, 150, 33, 210, 129], "nb": [1, 7, 64, 100, 129, 40], "nc": [3, 48, 95, 200, 16, 331]}
SIZES = [16, 7, 2, 5, 3, 2, 11, 32, 2, 9, 64, 2]


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    """dtype -> name -> model folder whose file holds that dtype."""
    out = {"float32": {}, "bfloat16": {}}
    for name, (cfg, seed) in NISOTAR.items():
        for dtype, t in (("float32", torch.float32), ("bfloat16", torch.bfloat16)):
            d = tmp_path_factory.mktemp(f"nisotar_{name}_{dtype}")
            write_loud_folder(str(d), cfg, seed, t)
            out[dtype][name] = str(d)
    return out


@pytest.fixture(scope="module")
def plain_logits(folders):
    made = {}

    class Lookup:
        def __getitem__(self, key):
            name, dtype = key
            if key not in made:
                reqs = random_requests(NISOTAR[name][0]["vocab"], LENGTHS[name], seed=271 + len(made))
                model = plain.PlainNisotar(folders[dtype][name])
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

def _pages(rng, n, page, slots=2, slot=1):
    """A block table in which `slot` holds n tokens on shuffled pages, and the number of pages."""
    blocks, n_pages = -(-n // page), -(-n // page) + 3
    table = torch.full((slots, blocks), -1, dtype=torch.int32, device=DEV)
    table[slot] = _ints(rng.permutation(n_pages)[:blocks])
    return table, n_pages


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,rot,mag,own", [(4, 2, 64, 64, 32, 1.0, False), (6, 1, 48, 32, 48, 1.2, True), (3, 3, 20, 12, 6, 1.0, True),
                                                 (5, 1, 12, 12, 2, 1.0, False), (2, 2, 128, 128, 128, 1.4, True),
                                                 (8, 4, 96, 96, 16, 1.1, False), (2, 1, 256, 200, 64, 1.0, True), (1, 1, 21, 21, 0, 1.0, False),
                                                 (32, 8, 128, 64, 64, 1.3, True), (3, 1, 32, 48, 0, 1.0, True)])
def test_heads_normed_then_turned_into_shuffled_pages(dtype, H, G, d, e, rot, mag, own):
    """Every head by itself with a weight for each number, then the rotation by halves, at positions up to 120,000; values of
    their own or the keys as they were projected. One head is a hundred times larger: a statistic shared between heads shows."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H * 100 + d + rot)
    page, positions = 8, [0, 1, 7, 8, 9, 119_990, 119_991, 3]
    rows = len(positions)
    cols = H * d + G * d + (G * e if own else 0)
    x = rng.randn(rows, cols + 8)
    x[:, :d] *= 100.0
    x[:, H * d:H * d + d] *= 0.01
    x = _np(_t(x, dtype))
    freq, _ = plain.yarn(700.0, rot, {"factor": 6.0, "original": 128, "fast": 16.0, "slow": 1.0}) if rot else (np.zeros(0), 1.0)
    wq, wk = 1 + 0.3 * rng.randn(d), 1 + 0.3 * rng.randn(d)
    table = torch.full((2, 119_992 // page + 1), -1, dtype=torch.int32, device=DEV)
    for i, blk in enumerate(sorted({p // page for p in positions})):
        table[1, blk] = [2, 0, 1][i % 3]
    k_cache = torch.zeros(3, page, G, d, dtype=dtype, device=DEV)
    v_cache = torch.zeros(3, page, G, e, dtype=dtype, device=DEV)
    proj = _t(x, dtype)
    eps = 1e-5
    ops.qk_norm_turn_cache(proj, _t(wq), _t(wk), eps, _t(freq, torch.float64) if rot else None, rot, mag, _ints(positions),
                           _ints([1] * rows), table, k_cache, G * d, v_cache, G * e, H, G, d, e, page, values_are_keys=not own)
    q = plain.rotate_halves(plain.rms_norm(x[:, :H * d].reshape(rows, H, d), wq, eps), positions, freq, mag)
    k_raw = x[:, H * d:(H + G) * d].reshape(rows, G, d)
    k = plain.rotate_halves(plain.rms_norm(k_raw, wk, eps), positions, freq, mag)
    v = x[:, (H + G) * d:cols].reshape(rows, G, e) if own else k_raw
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    _close(_np(proj)[:, :H * d].reshape(rows, H, d), q, tol, "queries")
    assert np.array_equal(_np(proj)[:, H * d:], x[:, H * d:]), "columns behind the queries stay"
    for i, p in enumerate(positions):
        at = int(table[1, p // page])
        _close(_np(k_cache[at, p % page]), k[i], tol, f"key of position {p}")
        assert np.array_equal(_np(v_cache[at, p % page]), v[i]), f"values of position {p}"


def _chunk_case(rng, n, H, G, d, e, chunk, dtype, page, strength):
    """One request's keys and values on shuffled pages, and queries each of which points at one key: the chunk's first, the
    one in front of it (of another chunk), its own, the chunk's last that it may see, one far away."""
    k, v = _np(_t(rng.randn(n, G, d), dtype)), _np(_t(rng.randn(n, G, e) * 2 + 1, dtype))
    table, n_pages = _pages(rng, n, page)
    k_cache = torch.zeros(n_pages, page, G, d, dtype=dtype, device=DEV)
    v_cache = torch.zeros(n_pages, page, G, e, dtype=dtype, device=DEV)
    at = table[1].long()[torch.arange(n, device=DEV) // page]
    k_cache[at, torch.arange(n, device=DEV) % page] = _t(k, dtype)
    v_cache[at, torch.arange(n, device=DEV) % page] = _t(v, dtype)
    q = rng.randn(n, H, d) * 0.3
    for i in range(n):
        first = i // chunk * chunk if chunk else 0
        j = [first, first - 1, i, max(first, i - 63), first - chunk, 0, i - 1][i % 7]
        if i % 11 == 3:
            q[i] = 0.0                                       # every score 0: as likely as the sink
        elif i % 11 == 7:
            q[i] = -k[i].mean(axis=0) * 3.0                  # scores far below zero: the sink takes the weight
        elif 0 <= j <= i:
            for h in range(H):
                kk = k[j, h // (H // G)]
                q[i, h] += kk * (strength / max(1e-6, (kk ** 2).sum()))
    return k, v, table, k_cache, v_cache, _np(_t(q, dtype))


CHUNK_CASES = [(4, 2, 32, 32, 37), (3, 3, 20, 12, 64), (5, 1, 12, 28, 1), (4, 1, 64, 64, 100), (2, 2, 200, 8, 33), (6, 2, 48, 16, 200),
               (6, 1, 96, 96, 80)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e,chunk", CHUNK_CASES)
def test_plain_attention_inside_chunks_with_a_sink(dtype, H, G, d, e, chunk):
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H * 10 + d)
    n, page = 530, 16
    k, v, table, k_cache, v_cache, q = _chunk_case(rng, n, H, G, d, e, chunk, dtype, page, 12.0)
    positions = sorted({0, 1, 2, 15, 16, 32, 33, 36, 37, 38, 63, 64, 65, 73, 74, 79, 80, 99, 100, 101, 128, 199, 200, 201, 255, 256, 511, 512,
                        513, 529})
    out = torch.zeros(len(positions), H * e, dtype=dtype, device=DEV)
    ops.paged_attention_generic_kv(_t(q[positions].reshape(len(positions), H * d), dtype), k_cache, G * d, v_cache, G * e, table,
                                   _ints(positions), _ints([1] * len(positions)), out, H, G, d, e, page, 0.9, sink=True, chunk=chunk)
    want = plain.attend(q[positions], k, v, positions, list(range(n)), 0.9, chunk=chunk, sink=True)
    _close(_np(out).reshape(-1, H, e), want, 3e-5 if dtype == torch.float32 else 2e-2)


@pytest.mark.parametrize("H,G,d,e,chunk", [(4, 2, 32, 32, 37), (8, 2, 48, 48, 64), (4, 4, 64, 64, 100), (6, 2, 64, 32, 1), (2, 1, 128, 128, 160),
                                           (6, 1, 96, 96, 80), (3, 3, 16, 16, 0), (4, 1, 64, 128, 300)])
def test_masked_flash_attention_inside_chunks_with_a_sink(H, G, d, e, chunk):
    """Portions that begin inside key tiles and chunks and go over several of them, then the same rows as single tokens (heads
    of a key head in one tile, with the keys in one piece and dealt over four). Pages behind the chunk hold numbers that are
    not numbers: they must not be read."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H + d + chunk)
    n, page = 333, 16
    k, v, table, k_cache, v_cache, q = _chunk_case(rng, n, H, G, d, e, chunk, torch.bfloat16, page, 12.0)
    want = plain.attend(q, k, v, list(range(n)), list(range(n)), 0.6, chunk=chunk, sink=True)
    order = list(range(200, n)) + list(range(200))
    tiles = [(1, 0, 128, 200), (1, 128, 5, 328), (1, 133, 128, 0), (1, 261, 72, 128)]
    out = torch.zeros(n, H * e, dtype=torch.bfloat16, device=DEV)
    ops.masked_flash_attention(_t(q[order].reshape(n, H * d), torch.bfloat16), k_cache, G * d, v_cache, G * e, table,
                               _ints([x for t in tiles for x in t]), len(tiles), out, H, G, d, e, page, 0.6, sink=True, chunk=chunk)
    _close(_np(out).reshape(n, H, e), want[order], 2e-2, "portions")
    picked = [0, 1, 19, 36, 37, 38, 63, 64, 65, 74, 79, 80, 99, 100, 101, 159, 160, 161, 255, 256, 299, 300, 301, 332]
    for parts in (1, 4):
        m = len(picked)
        out = torch.zeros(m, H * e, dtype=torch.bfloat16, device=DEV)
        scratch = torch.zeros(ops.masked_flash_partial_floats(m, H, e, parts), device=DEV) if parts > 1 else None
        ops.masked_flash_attention(_t(q[picked].reshape(m, H * d), torch.bfloat16), k_cache, G * d, v_cache, G * e, table,
                                   _ints([x for i, p in enumerate(picked) for x in (1, i, 1, p)]), m, out, H, G, d, e, page, 0.6,
                                   sink=True, one_token_tiles=True, parts=parts, partial=scratch, chunk=chunk)
        _close(_np(out).reshape(m, H, e), want[picked], 2e-2, f"single tokens in {parts} parts")
    if chunk > 1:
        # a decoded token whose chunk has just begun, with every page in front of its own poisoned
        p = max(x for x in range(0, n, chunk))
        for blk in range(p // page):
            k_cache[table[1, blk].long()] = float("nan")
            v_cache[table[1, blk].long()] = float("nan")
        out = torch.zeros(1, H * e, dtype=torch.bfloat16, device=DEV)
        ops.masked_flash_attention(_t(q[[p]].reshape(1, H * d), torch.bfloat16), k_cache, G * d, v_cache, G * e, table, _ints([1, 0, 1, p]),
                                   1, out, H, G, d, e, page, 0.6, sink=True, one_token_tiles=True, chunk=chunk)
        _close(_np(out).reshape(1, H, e), want[[p]], 2e-2, "the first token of a chunk")


def _delta_reference(q, k, v, z, a_log, dt_bias, b, S):
    """q, k [T, G, d] and v [T, H, e] after convolution and silu, z [T, H, d] the decays' raw numbers; S [H, d, e] goes on."""
    T, H, e = v.shape
    G, d = q.shape[1], q.shape[2]
    g = np.exp(-np.exp(a_log)[None, :, None] * plain.softplus(z + dt_bias.reshape(H, d)))
    beta = plain.sigmoid(b)
    q, k = plain.unit(q) * d ** -0.5, plain.unit(k)
    out = np.zeros((T, H, e))
    for t in range(T):
        for h in range(H):
            j = h // (H // G)
            S[h], out[t, h] = plain.delta_step(S[h], q[t, j], k[t, j], v[t, h], g[t, h], beta[t, h])
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,e", [(2, 2, 32, 32), (4, 1, 24, 16), (3, 3, 10, 7), (2, 1, 128, 64), (4, 4, 64, 128), (1, 1, 8, 40), (2, 2, 200, 12),
                                     (2, 1, 16, 33), (1, 1, 300, 20), (6, 2, 40, 24), (1, 1, 512, 8)])
def test_delta_rule_with_a_decay_per_channel(dtype, H, G, d, e):
    """Two requests in different cuts side by side (single tokens, pairs, portions shorter and longer than a tile), from and
    into their states, then a slot that is used again. Neighbouring channels forget very differently, from hardly at all to
    nearly everything, so that a decay at the wrong row shows; write strengths near one correct what the state holds."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(H * 1000 + d + e)
    qk = G * d
    C = 2 * qk + H * e
    cuts = {1: [1, 2, 37, 16, 1, 1, 33, 6, 1], 3: [7, 1, 1, 2, 49, 3, 4, 1, 1]}
    a_log, dt = rng.randn(H) * 0.4, rng.randn(H * d)
    state = torch.zeros(4, H * d * e + 5, device=DEV)
    state[0] = 3.0
    tol = 5e-5 if dtype == torch.float32 else 3e-4
    for again in range(2):
        state[1], state[3] = 0.0, 0.0
        data = {s: dict(u=_np(_t(rng.randn(sum(c), C + 3), dtype)), b=_np(_t(rng.randn(sum(c), H + 4) * 2 + 1, dtype)),
                        z=_np(_t(rng.randn(sum(c), H * d + 8) * 3 - 2))) for s, c in cuts.items()}
        want = {}
        for s, x in data.items():
            T = len(x["u"])
            q, k = x["u"][:, :qk].reshape(T, G, d), x["u"][:, qk:2 * qk].reshape(T, G, d)
            want[s] = _delta_reference(q, k, x["u"][:, 2 * qk:C].reshape(T, H, e), x["z"][:, :H * d].reshape(T, H, d), _np(_t(a_log)),
                                       _np(_t(dt)), x["b"][:, 3:3 + H], np.zeros((H, d, e))).reshape(T, H * e)
        at = {1: 0, 3: 0}
        for step in range(9):
            batch = Batch([(s, at[s], cuts[s][step]) for s in (3, 1)])
            rows = lambda key, t: torch.cat([_t(data[s][key][p:p + n], t) for s, p, n in batch.runs])
            out = torch.zeros(batch.num_tokens, H * e, device=DEV)
            ops.delta_rule(rows("u", dtype), 0, qk, 2 * qk, rows("b", dtype), 3, 0, _t(a_log), _t(dt), state, batch.q_start,
                           batch.state_slots, out, batch.num_requests, H, G, d, e, channel_decay=rows("z", torch.float32))
            row = 0
            for s, p, n in batch.runs:
                _close(_np(out[row:row + n]), want[s][p:p + n], tol, f"step {step} slot {s}")
                row += n
                at[s] += n
        assert float(state[0].min()) == 3.0 and float(state[0].max()) == 3.0 and float(state[2].abs().max()) == 0.0
        assert float(state[1:, H * d * e:].abs().max()) == 0.0


@pytest.mark.parametrize("H,G,d,e", [(2, 1, 128, 64), (3, 3, 40, 24)])
def test_delta_rule_over_many_tokens(H, G, d, e):
    """A portion of a thousand tokens beside one of 3 and a single token, with decays near one: what is kept adds up."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(d)
    qk = G * d
    runs = [(0, 0, 1000), (2, 4, 3), (1, 9, 1)]
    batch = Batch(runs)
    u, b = _np(_t(rng.randn(1004, 2 * qk + H * e))), _np(_t(rng.randn(1004, H) * 2))
    z = _np(_t(rng.randn(1004, H * d) - 5.0))
    a_log, dt = _np(_t(rng.randn(H) * 0.3)), _np(_t(rng.randn(H * d) * 0.3))
    S0 = _np(_t(rng.randn(3, H, d, e)))
    state = _t(S0.reshape(3, -1))
    out = torch.zeros(1004, H * e, device=DEV)
    ops.delta_rule(_t(u), 0, qk, 2 * qk, _t(b), 0, 0, _t(a_log), _t(dt), state, batch.q_start, batch.state_slots, out, 3, H, G, d, e,
                   channel_decay=_t(z))
    row = 0
    for s, _, n in runs:
        r = slice(row, row + n)
        S = S0[s].copy()
        want = _delta_reference(u[r, :qk].reshape(n, G, d), u[r, qk:2 * qk].reshape(n, G, d), u[r, 2 * qk:].reshape(n, H, e),
                                z[r].reshape(n, H, d), a_log, dt, b[r], S)
        _close(_np(out[r]).reshape(n, H, e), want, 1e-4, f"outputs of slot {s}")
        _close(_np(state[s]).reshape(H, d, e), S, 1e-4, f"state of slot {s}")
        row += n


@pytest.mark.parametrize("dtype,gate_dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)])
@pytest.mark.parametrize("H,e", [(2, 32), (3, 7), (4, 128), (1, 200)])
def test_head_norm_with_a_sigmoid_gate(dtype, gate_dtype, H, e):
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(e)
    rows = 9
    o = _np(_t(rng.randn(rows, H * e) * np.array([1e-3, 1.0, 50.0] * 3)[:, None]))
    gate, w = _np(_t(rng.randn(rows, H * e + 8) * 3, gate_dtype)), 1 + 0.2 * rng.randn(e)
    for act, f in (("sigmoid", plain.sigmoid), ("silu", plain.silu)):
        out = torch.zeros(rows, H * e, dtype=dtype, device=DEV)
        ops.head_norm_gate(_t(o), _t(gate, gate_dtype), 8, _t(w), 1e-6, out, H, e, act=act)
        want = plain.rms_norm(o.reshape(rows, H, e), w, 1e-6) * f(gate[:, 8:]).reshape(rows, H, e)
        _close(_np(out).reshape(rows, H, e), want, 2e-5 if dtype == torch.float32 else 1e-2, act)


@pytest.mark.parametrize("width", [30, 72, 512, 1001, 1024, 2048, 4096, 5000])
def test_half_the_sum_of_two_normed_results(width):
    """Partial sums, either dtype, results of very different size, each with a weight of its own."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(width)
    rows, eps = 5, 1e-4
    wa, wb = 1 + 0.3 * rng.randn(width), 1 + 0.3 * rng.randn(width)
    for parts_a, parts_b, ta, tb in ((0, 0, torch.bfloat16, torch.bfloat16), (3, 0, torch.float32, torch.bfloat16),
                                     (0, 2, torch.bfloat16, torch.float32), (4, 5, torch.float32, torch.float32)):
        a = _np(_t(rng.randn(*([parts_a] if parts_a else []), rows, width) * 40.0, ta))
        b = _np(_t(rng.randn(*([parts_b] if parts_b else []), rows, width) * 0.01, tb))
        out = torch.zeros(rows, width, device=DEV)
        ops.normed_sum(_t(a, ta), _t(wa), 0.5, _t(b, tb), _t(wb), 0.5, eps, out)
        want = plain.half_sum(a.sum(0) if parts_a else a, b.sum(0) if parts_b else b, wa, wb, eps)
        _close(_np(out), want, 1e-5, f"{parts_a}, {parts_b} parts")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,inner", [(1, 96, 40), (5, 256, 136), (8, 128, 64), (12, 512, 128), (16, 64, 200), (40, 72, 33), (64, 128, 192),
                                              (130, 256, 1024), (300, 256, 1024), (700, 512, 2048)])
@pytest.mark.parametrize("limit", [0.6, 7.0])
def test_clamped_gated_product(dtype, rows, width, inner, limit):
    """Gate and up products with biases, many of them beyond the limit on both sides, over few rows and over many."""
    from dynalm_b200.engine.runtime import Runtime
    from dynalm_b200.kernels import ops
    from dynalm_b200.kernels.gemm import linear_clamped_swiglu, linear_partial_biased
    rng = np.random.RandomState(rows + inner)
    x = _np(_t(rng.randn(rows, width), dtype))
    w = _np(_t(rng.randn(2 * inner, width) * 2.5 / np.sqrt(width), dtype))
    bias = _np(_t(rng.randn(2 * inner) * 1.5))
    rt = Runtime(DEV, dtype, max_tokens=rows)
    got = _np(linear_clamped_swiglu(_t(x, dtype), _t(w, dtype), ops.clamped_coeffs(limit, 1.702, _t(bias), inner, DEV), rt, inner))
    z = x @ w.T + bias
    want = plain.clamped_gate(z[:, :inner], z[:, inner:], limit)
    assert ops.gemm_tcgen05_status() == 0
    _close(got, want, 3e-5 if dtype == torch.float32 else 3e-2)
    none = _np(linear_clamped_swiglu(_t(x, dtype), _t(w, dtype), ops.clamped_coeffs(limit, 1.702, None, inner, DEV), rt, inner))
    z = x @ w.T
    _close(none, plain.clamped_gate(z[:, :inner], z[:, inner:], limit), 3e-5 if dtype == torch.float32 else 3e-2, "without biases")
    down, b2 = _np(_t(rng.randn(width, inner) * 0.2, dtype)), _np(_t(rng.randn(width) * 30.0))
    got = _np(linear_partial_biased(_t(want, dtype), _t(down, dtype), _t(b2), rt, "t"))
    got = got.sum(0) if got.ndim == 3 else got
    _close(got, want @ down.T + b2, 3e-5 if dtype == torch.float32 else 1e-2, "down with its bias")


@pytest.mark.parametrize("rows", [1, 7, 12, 40, 64, 65, 200])
@pytest.mark.parametrize("K,N", [(8, 96), (40, 72), (128, 1024)])
def test_a_short_product_over_a_slice_of_wider_rows(rows, K, N):
    from dynalm_b200.kernels import ops
    from dynalm_b200.kernels.gemm import linear_short
    rng = np.random.RandomState(rows + K)
    x, w = _np(_t(rng.randn(rows, K + 24), torch.bfloat16)), _np(_t(rng.randn(N, K), torch.bfloat16))
    out = torch.zeros(rows, N, device=DEV)
    linear_short(_t(x, torch.bfloat16)[:, 8:8 + K], _t(w, torch.bfloat16), out)
    assert ops.gemm_tcgen05_status() == 0
    _close(_np(out), x[:, 8:8 + K] @ w.T, 1e-5)


@pytest.mark.parametrize("E,top", [(8, 2), (5, 1), (4, 4), (40, 7), (256, 8), (1, 1), (33, 3)])
def test_router_with_a_bias_on_the_logits(E, top):
    """Biases that change which experts are chosen AND how they weigh; logits of a few and of many nats."""
    from dynalm_b200.kernels import ops
    rng = np.random.RandomState(E)
    rows = 40
    z, bias = rng.randn(rows, E) * np.linspace(0.1, 12.0, rows)[:, None], rng.randn(E) * 3.0
    z, bias = _np(_t(z)), _np(_t(bias))
    logits = _t(np.concatenate([z, np.full((rows, 3), 50.0)], axis=1))[:, :E]         # (rows with more behind them)
    ids, w = torch.zeros(rows, top, dtype=torch.int32, device=DEV), torch.zeros(rows, top, device=DEV)
    ops.moe_route(logits, top, 1, 1, 1.0, ids, w, bias=_t(bias))
    for r in range(rows):
        chosen, weights = plain.route(z[r] + bias, top)
        assert [int(i) for i in ids[r]] == chosen, f"row {r}"
        _close(_np(w[r]), weights, 3e-6, f"weights of row {r}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,r,e,R,window", [(3, 16, 16, 24, 40, 29), (2, 10, 6, 7, 21, 5), (4, 32, 32, 32, 128, 65), (6, 64, 8, 16, 64, 0)])
def test_latent_attention_turned_by_halves_inside_a_window(dtype, H, d, r, e, R, window):
    """The whole mixer with weights so large that one key takes most of a query's weight, in portions and token by token: the
    keys just inside and just outside the window decide, and a pair of the rotation that is not one shows."""
    from dynalm_b200.config.plan import MixerSpec, PositionSpec
    from dynalm_b200.engine import build
    cfg = {"architecture": "Nisotar", "vocab": 150, "width": 96, "norm": {"eps": 1e-5},
           "layers": [{"type": "latent_attention", "mlp": None,
                       "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": e, "kv_rank": R, "scale": (d + r) ** -0.5,
                                 "rot": {"base": 500.0, "dims": r}, **({"mask": {"size": window}} if window else {})}}]}
    from dynalm_b200.registry import find_architecture
    from dynalm_b200.weights.random_init import random_tensors
    arch = find_architecture(cfg)
    t = random_tensors(arch.plan(arch.read_config(cfg)), 5, torch.float32)
    t["l0.mix.q"] *= 18.0
    t["l0.mix.uk"] *= 12.0
    t["l0.mix.dkv"] *= 12.0
    t["l0.mix.uv"] *= 20.0
    t["l0.mix.o"] *= 20.0
    t["embed"] *= 50.0
    t = {n: x.to(torch.bfloat16) for n, x in t.items()}
    model = plain.PlainNisotar(config=cfg, tensors={n: x.float().numpy() for n, x in t.items()})
    reqs = random_requests(150, [90, 33], seed=6)
    logits = {n: model.logits(x) for n, x in reqs.items()}
    for plan in (plan_whole(reqs), plan_chunks(reqs, [16, 3, 2, 7]), plan_tail(reqs, 40)):
        built = build(config_obj=cfg, tensors=t, dtype=dtype, kv_tokens=160, max_batch_tokens=128, max_requests=2, context=128)
        got = run_plan_in_process(built.step_fn, plan)
        compare(plan, got, logits, *TOL[dtype], "latent", spread=SPREAD[dtype])


# ---------------------------------------------------------------------------------------------
# whole models through the step function
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(NISOTAR))
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


@pytest.mark.parametrize("name", sorted(NISOTAR))
def test_layers_follow_the_plain_implementation(name, folders, monkeypatch):
    """The residual stream behind every layer of a short prompt in 32-bit, what a layer leaves pending included."""
    import copy
    from dynalm_b200.engine import launch_memo
    monkeypatch.setattr(launch_memo, "ENABLED", False)
    reqs = random_requests(NISOTAR[name][0]["vocab"], [29], seed=2)
    toks = reqs["r0"]
    _, layers = plain.PlainNisotar(folders["float32"][name]).logits(toks, layers=True)
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
    """A model whose layers repeat: with the layers after the first of a kind re-issued by address (each with its own norms,
    biases, decays and states) the logits are bit for bit those of every layer run through its parts."""
    import copy
    from dynalm_b200.engine import launch_memo
    cfg = copy.deepcopy(NISOTAR["na"][0])
    cfg["layers"] = [copy.deepcopy(cfg["layers"][i]) for i in (0, 0, 0, 4, 4, 1)]
    reqs = random_requests(cfg["vocab"], [40, 9], seed=4)
    plan = plan_chunks(reqs, [16, 3, 2])
    outs = []
    with tempfile.TemporaryDirectory() as d:
        write_loud_folder(d, cfg, 5, torch.float32 if dtype == "float32" else torch.bfloat16)
        for enabled in (True, False):
            monkeypatch.setattr(launch_memo, "ENABLED", enabled)
            before = launch_memo.REPLAYED_LAYERS
            built = _built(d, dtype, 128, 64, max_requests=2)
            outs.append(run_plan_in_process(built.step_fn, plan))
            assert (launch_memo.REPLAYED_LAYERS > before) == enabled
        model = plain.PlainNisotar(d)
        compare(plan, outs[0], {r: model.logits(t) for r, t in reqs.items()}, *TOL[dtype], "repeated layers", spread=SPREAD[dtype])
    assert all(np.array_equal(outs[0][k], outs[1][k]) for k in outs[0])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_single_token_rows_beside_a_portion(dtype, folders):
    """A couple of dozen live requests decoding beside portions of long prompts: unequal requests in one batch
    against each alone, with more state slots than the other tests use."""
    name = "na"
    vocab = NISOTAR[name][0]["vocab"]
    short = {f"s{k}": v for k, v in random_requests(vocab, [12 + (5 * i) % 29 for i in range(20)], seed=8).items()}
    long = {f"l{k}": v for k, v in random_requests(vocab, [150, 90], seed=9).items()}
    model = plain.PlainNisotar(folders[dtype][name])
    logits = {r: model.logits(t) for r, t in {**short, **long}.items()}
    plan = plan_many_rows(short, long, seed=3, tail_lo=4, tail_hi=10)
    built = _built(folders[dtype][name], dtype, plan.max_live_tokens(64), 256, max_requests=24)
    got = run_plan_in_process(built.step_fn, plan)
    compare(plan, got, logits, *TOL[dtype], f"{name}/{dtype}/many rows", spread=SPREAD[dtype])


@pytest.mark.parametrize("name", sorted(ONE_KIND))
def test_models_of_one_kind_of_layer(name, tmp_path):
    cfg, seed = ONE_KIND[name]
    write_loud_folder(str(tmp_path), cfg, seed, torch.float32)
    reqs = random_requests(cfg["vocab"], [5, 200, 77, 130, 64], seed=3)
    model = plain.PlainNisotar(str(tmp_path))
    logits = {r: model.logits(t) for r, t in reqs.items()}
    for what, plan in (("whole", plan_whole(reqs)), ("mixed", plan_mixed(reqs, seed=4))):
        need = plan.max_live_tokens(64)
        built = _built(str(tmp_path), "float32", need, max(need, 64), max_requests=4)
        got = run_plan_in_process(built.step_fn, plan)
        compare(plan, got, logits, *TOL["float32"], f"{name}/{what}")
        assert built.cache.free_pages == built.cache.num_pages


@pytest.mark.parametrize("name,dtype", [("na", "float32"), ("nc", "float32"), ("nc", "bfloat16")])
def test_long_decoding_keeps_its_place(name, dtype, folders):
    """300 tokens decoded one by one after a 3-token prompt: every window passes over decoded tokens and every chunk begins many
    times, and states and kept inputs are carried through every step (also through steps replayed from a captured graph)."""
    reqs = random_requests(NISOTAR[name][0]["vocab"], [303], seed=12)
    model = plain.PlainNisotar(folders[dtype][name])
    logits = {r: model.logits(t) for r, t in reqs.items()}
    plan = plan_tail(reqs, 300)
    built = _built(folders[dtype][name], dtype, 320, 64, max_requests=2)
    got = run_plan_in_process(built.step_fn, plan)
    assert built.step_fn.graph_captures > 0 or not built.step_fn.use_graphs
    compare(plan, got, logits, *TOL[dtype], "long decoding", spread=SPREAD[dtype])
    assert built.cache.free_pages == built.cache.num_pages


def test_a_forked_request_takes_its_state_along(folders):
    """A request forked in mid-sequence continues as its parent would have: states and kept inputs are copied."""
    from dynalm_b200.engine import StepEntry
    name = "na"
    toks = random_requests(NISOTAR[name][0]["vocab"], [60], seed=21)["r0"]
    other = toks[:31] + [(t + 7) % 301 for t in toks[31:]]
    model = plain.PlainNisotar(folders["float32"][name])
    want = {"a": model.logits(toks), "b": model.logits(other)}
    sf = _built(folders["float32"][name], "float32", 256, 64, max_requests=4).step_fn
    sf.step([StepEntry("a", toks[:31], [])])
    sf.fork("a", "b")
    for lo, hi in ((31, 32), (32, 40), (40, 41), (41, 60)):
        got = _np(sf.step([StepEntry("a", toks[lo:hi], [hi - lo - 1]), StepEntry("b", other[lo:hi], [hi - lo - 1])]))
        _close(got[0], want["a"][hi - 1], 6e-5, f"parent at {hi}")
        _close(got[1], want["b"][hi - 1], 6e-5, f"child at {hi}")


def test_trace_run_replays_a_plan(folders, tmp_path):
    name = "nb"
    reqs = random_requests(NISOTAR[name][0]["vocab"], [40, 7, 90], seed=13)
    model = plain.PlainNisotar(folders["float32"][name])
    logits = {r: model.logits(t) for r, t in reqs.items()}
    plan = plan_mixed(reqs, seed=2)
    got = run_plan_trace_run(folders["float32"][name], "float32", plan, str(tmp_path), plan.max_live_tokens(64),
                             NISOTAR[name][0]["vocab"])
    compare(plan, got, logits, *TOL["float32"], "trace_run")


# ---------------------------------------------------------------------------------------------
# generation through the entry point
# ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name", sorted(NISOTAR))
def test_greedy_generation_through_the_engine(name, folders):
    """Through the engine's entry point and scheduler, together and alone."""
    from dynalm_b200 import Engine
    folder = folders["float32"][name]
    model = plain.PlainNisotar(folder)
    reqs = random_requests(NISOTAR[name][0]["vocab"], [5, 17, 33, 70], seed=14)
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
    name = "na"
    reqs = list(random_requests(NISOTAR[name][0]["vocab"], [40, 90, 17, 100, 64, 33], seed=15).values())

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
    proc = subprocess.run([os.path.join(ROOT, "bin", "dynalm"), "run", folders["bfloat16"]["na"], "--tokens", "5,9,200,31",
                           "-n", "8", "--ctx", "256", "--batch", "64", "--no-stream"], capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    ids = [int(t) for t in proc.stdout.split()]
    assert len(ids) == 8 and all(0 <= t < NISOTAR["na"][0]["vocab"] for t in ids)
    from dynalm_b200 import Engine
    assert Engine(folders["bfloat16"]["na"], ctx=256, batch=64).generate([5, 9, 200, 31], max_tokens=8).tokens == ids
