"""Pogarax on the GPU: replay through bin/trace_run against the plain implementation (whole prompts,
tails decoded token by token, portions down to two tokens, mixed batches in a pool so small that pages
and slots are used again, windows that give pages back), every new kernel and option alone against
NumPy, keys planted just inside and just outside a window, far away and at page borders, states and
kept rows across steps and slots used again, and greedy generation through the Python entry point,
the scheduler and the command line."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_pogarax as pp
import tiny_pogarax as tp
import trace_tools as tt

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
SMALL = ["PA", "PB", "PC", "PD"]
LENGTHS = {"PA": [1, 2, 19, 100, 65, 48, 33], "PB": [5, 41, 97, 150, 34, 64], "PC": [3, 70, 130, 17], "PD": [2, 110, 31, 16, 77],
           "PL": [7, 150, 320, 64]}


@pytest.fixture(scope="module")
def cases(model_folders):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            folder = model_folders(name, dtype)
            rng = np.random.default_rng(1200 + ord(name[1]))
            reqs = tt.make_requests(rng, tp.TINY[name]["config"]["vocab"], LENGTHS[name[:2]])
            cfg, w = pp.load_folder(folder)
            made[(name, dtype)] = (folder, reqs, {r: pp.logits_all(cfg, w, t) for r, t in reqs.items()})
        return made[(name, dtype)]
    return get


# In bfloat16 a router's choice between two experts whose logits differ by less than its input's rounding is a
# toss-up, and since only the results are normed the other expert's output counts in full; states and cached
# rows carry it on.  So bfloat16 whole-model logits are compared at the same configurations with every expert
# chosen ("-all"), and at the others loosely.
def _compare(got, tb, plain, dtype, label, tol_rms=3e-5):
    errs = []
    for sid in sorted(tb.rows):
        want = tt.expected_rows(tb.rows[sid], plain)
        have = got[sid]
        assert have.shape == want.shape and np.isfinite(have).all(), (label, sid)
        errs.extend(np.sqrt(((have - want) ** 2).mean(axis=1)) / np.sqrt((want ** 2).mean(axis=1)))
    errs = np.sort(np.asarray(errs))
    print(f"{label} {dtype}: {len(errs)} rows, relative rms error median {np.median(errs):.2e}, "
          f"90 % {errs[int(0.9 * (len(errs) - 1))]:.2e}, worst {errs[-1]:.2e}")
    if dtype == "float32":
        assert errs[-1] <= tol_rms, (label, errs[-1])
    elif "PC" in label:          # (heads of 8 elements whose read-outs are normed: rounding of 32-bit, too, shows tenfold there)
        assert np.median(errs) <= 6e-2, label
    elif label.split()[1].endswith("-all"):
        assert np.median(errs) <= 2.5e-2 and errs[int(0.98 * (len(errs) - 1))] <= 6e-2, label
    else:
        assert np.median(errs) <= 0.1, label


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in SMALL] + [(n + "-all", "bfloat16") for n in SMALL] + [("PA", "bfloat16")])
def test_alone_whole_tail_portions(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tp.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_whole(tb, reqs)
    tt.trace_tail_decode(tb, reqs)
    tt.trace_portions(tb, reqs, np.random.default_rng(7))
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"))
    _compare(got, tb, plain, dtype, f"config {name}")
    if dtype == "float32":
        tt.compare_cuts([(got, tb)], dtype, f"config {name}", tol=2e-5)


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in SMALL] + [(n + "-all", "bfloat16") for n in SMALL] + [("PA", "bfloat16")])
def test_mixed_with_page_and_slot_reuse(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tp.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_mixed(tb, reqs, np.random.default_rng(11), max_live=3)
    assert tb.pages_taken > tb.peak_tokens // ps, "the trace must make the pool hand pages out again"
    assert max(len(s["entries"]) for s in tb.steps) >= 3
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"),
                       extra_args=["--max-live", "3"])          # three slots for all requests
    _compare(got, tb, plain, dtype, f"config {name} mixed")


@pytest.mark.parametrize("name", ["PA", "PB"])
def test_long_decoding(name, cases, tmp_path):
    """Decoded past every window many times over."""
    folder, reqs, plain = cases(name, "float32")
    ps = tp.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_tail_decode(tb, {"r3": reqs["r3"]}, tail=len(reqs["r3"]) - 3)
    got = tt.run_trace(folder, "float32", tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"))
    _compare(got, tb, plain, "float32", f"config {name} decoded")


@pytest.mark.parametrize("name, dtype", [("PL", "float32"), ("PL", "bfloat16"), ("PL-all", "bfloat16")])
def test_layer_sizes_of_the_tensor_core_kernels(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tp.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_whole(tb, reqs)
    tt.trace_tail_decode(tb, reqs, tail=40)
    tt.trace_portions(tb, reqs, np.random.default_rng(3))
    tt.trace_mixed(tb, reqs, np.random.default_rng(5))
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"))
    _compare(got, tb, plain, dtype, f"config {name}", tol_rms=6e-5)
    if dtype == "float32":
        tt.compare_cuts([(got, tb)], dtype, "config PL", tol=6e-5)


def test_a_window_gives_pages_back(model_folders):
    """A model all of whose caches have windows decodes further than its pool holds pages for."""
    from crane_b200.config import EngineConfig
    from crane_b200.engine import ModelRunner, StepEntry
    folder = model_folders("PA", "float32")
    cfg, w = pp.load_folder(folder)
    ps = 8
    runner = ModelRunner(folder, EngineConfig(dtype="float32", page_size=ps, num_pages=6, max_concurrent=2,
                                              max_batched_tokens=64, max_seq_len=256))
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 120).tolist()
    want = pp.logits_all(cfg, w, toks)
    pos = 0
    for n in [20, 9, 2] + [1] * 89:
        got = runner.step([StepEntry(1, toks[pos:pos + n], [n - 1])]).cpu().numpy()[0]
        pos += n
        assert np.abs(got - want[pos - 1]).max() < 5e-5 * np.abs(want).max(), pos
    runner.rt.check_errors()
    runner.table.check()
    assert pos == 120 > 6 * ps


# ------------------------------------------------------------------ kernels
@pytest.fixture(scope="module")
def K():
    from crane_b200.kernels import get_kernels
    return get_kernels()


def _dev(a, dtype=torch.float32):
    return torch.as_tensor(np.asarray(a), dtype=dtype).to(DEV)


def _i32(a):
    return _dev(a, torch.int32)


def _err():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def _np(t):
    return t.double().cpu().numpy()


# three requests and a fourth that takes the second one's slot; portions, single tokens, a request left out of a
# step; slots in no order
PLAN = [[(0, 20, 2), (1, 1, 0), (2, 4, 1)], [(2, 5, 1), (0, 1, 2)], [(0, 1, 2)], [(0, 15, 2), (3, 2, 0)], [(3, 9, 0)]]
PLAN_LENS = [37, 1, 9, 11]
PLAN_LONG = [[(0, 70, 2), (1, 2, 0), (2, 1, 1), (3, 6, 3)], [(2, 66, 1), (0, 1, 2), (3, 1, 3)], [(0, 3, 2), (3, 67, 3)], [(0, 1, 2), (3, 2, 3)],
             [(2, 1, 1), (0, 1, 2)], [(0, 1, 2), (2, 1, 1), (3, 1, 3)], [(2, 3, 1), (0, 1, 2)]]
PLAN_LONG_LENS = [78, 2, 72, 77]


def _steps_of(lens, plan, pad=0):
    """Per step the kernels' metadata and, per entry, (request, first position, count).  ``pad``: that many
    rows of no entry and one entry without rows (of slot 3) behind the real ones."""
    done = [0] * len(lens)
    for step in plan:
        ents = []
        for r, take, slot in step:
            ents.append((r, done[r], take, slot))
            done[r] += take
        q_lens = [t for _, _, t, _ in ents] + ([0] if pad else [])
        ctx = SimpleNamespace(cu_q=_i32(np.concatenate([[0], np.cumsum(q_lens)])),
                              kv_len=_i32([b + t for _, b, t, _ in ents] + ([0] if pad else [])),
                              slots=_i32([s for _, _, _, s in ents] + ([3] if pad else [])),
                              tok_entry=_i32(np.concatenate([np.full(t, i) for i, t in enumerate(q_lens)] + [np.full(pad, -1)])))
        yield ctx, ents
    assert done == list(lens)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden, mixes", [(48, 5), (68, 5), (1000, 2), (7, 1)])
def test_token_shift_mix(K, dtype, hidden, mixes):
    """Every mix over the plan of steps, from slots full of another request's numbers, with padding rows."""
    rng = np.random.default_rng(hidden)
    mu = rng.standard_normal((mixes, hidden))
    rows = [_dev(rng.standard_normal((n, hidden)), dtype) for n in PLAN_LENS]
    off, pad = 3, 2
    state = torch.full((4, off + hidden + 2), 1e3, device=DEV)
    err = _err()
    tol = 1e-5 if dtype == torch.float32 else 3e-2
    for ctx, ents in _steps_of(PLAN_LENS, PLAN, pad):
        h = torch.cat([rows[r][b:b + t] for r, b, t, _ in ents] + [torch.full((pad, hidden), 9.0, dtype=dtype, device=DEV)])
        n = h.shape[0]
        out = torch.full((mixes, n, hidden), 5.0, dtype=dtype, device=DEV)
        K.token_shift_mix(h, _dev(mu), ctx, state, off, out, err)
        got = _np(out)
        at = 0
        for r, b, t, slot in ents:
            x = _np(rows[r])
            for g in range(mixes):
                want = pp.token_mix(x, mu[g])[b:b + t]
                assert np.abs(got[g, at:at + t] - want).max() < tol * max(1.0, np.abs(want).max()), (r, b, g)
            assert np.abs(state[slot, off:off + hidden].cpu().numpy() - x[b + t - 1]).max() == 0
            at += t
        assert (got[:, at:] == 5.0).all()
    assert (state[:, :off] == 1e3).all() and (state[:, off + hidden:] == 1e3).all() and (state[3] == 1e3).all()
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, d, dv", [(3, 16, 16), (1, 40, 24), (5, 8, 8), (2, 128, 128)])
def test_bonus_prep(K, dtype, H, d, dv):
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(d)
    n, hd, hv = 9, H * d, H * dv
    cols = 2 * hd + hv + (6 if d == 40 else 5)
    u = rng.standard_normal((H, d))
    ent = np.zeros(n, dtype=np.int32)
    ent[4] = -1
    for form in ("whole", "parts"):
        parts = _dev(rng.standard_normal((2, n, cols)))
        x = parts.sum(0).to(dtype)
        extra = (2 * hd + hv + H) % 2             # (rows of even length take two neighbours a lane)
        aux = torch.full((n, 2 * hd + hv + H + 6 + extra), 5.0, device=DEV)
        K.bonus_prep(x if form == "whole" else Partials(parts), cols, _i32(ent), _dev(u), aux, 2 * hd + hv + 6, H, d, dv, dtype)
        xn, got = _np(x), _np(aux)
        b = (xn[:, :hd].reshape(n, H, d) * u * xn[:, hd:2 * hd].reshape(n, H, d)).sum(-1)
        keep = ent >= 0
        assert np.abs(got[keep, :2 * hd + hv] - xn[keep, :2 * hd + hv]).max() < 1e-6, form
        assert np.abs(got[keep, 2 * hd + hv + 6:2 * hd + hv + 6 + H] - b[keep]).max() < 2e-5 * max(1.0, np.abs(b).max()), form
        assert (got[4] == 5.0).all() and (got[:, 2 * hd + hv:2 * hd + hv + 6] == 5.0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n", [1, 13, 70, 131])
@pytest.mark.parametrize("ranks, outs", [((5, 9), (48, 20)), ((24, 24), (64, 64)), ((128, 1), (200, 130)), ((300, 17), (33, 90)),
                                         ((256, 33), (65, 1))])
def test_low_rank_expand(K, dtype, n, ranks, outs):
    """Both decays, the plain product, tanh on the way in, two products in one launch, columns off the blocks'
    borders, ranks off the steps of 16 and beyond what the tensor-core kernel takes."""
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(n + ranks[0])
    exact = dtype == torch.float32
    offs = (3, 3 + ranks[0] + 2)
    cols = offs[1] + ranks[1] + 1
    parts = _dev(rng.standard_normal((3, n, cols)) * 0.7)
    low = parts.sum(0).to(dtype)
    ln = _np(low)
    ws = [_dev(rng.standard_normal((o, r)) * r ** -0.5, dtype) for o, r in zip(outs, ranks)]
    wn = [_np(w) for w in ws]
    ent = np.zeros(n, dtype=np.int32)
    if n > 2:
        ent[1] = -1
    keep = ent >= 0
    per = 4
    bias, rate = rng.standard_normal(outs[0]), rng.standard_normal(-(-outs[0] // per)) * 0.5
    packed = [K.pack_low_rank(w, exact) for w in ws]
    if not exact:
        assert [m for _, m in packed] == [-(-r // 16) * 16 <= 256 for r in ranks]
    for kind, tanh in (("soft_decay", False), ("exp_decay", True), ("plain", False)):
        out0 = torch.full((n, outs[0] + 3), 5.0, dtype=dtype if kind == "plain" else torch.float32, device=DEV)
        out1 = torch.full((n, outs[1]), 5.0, dtype=dtype, device=DEV)
        a = K.LowRank(packed[0][0], ranks[0], offs[0], outs[0], out=out0, kind=kind, bias=_dev(bias), rate=_dev(rate), per_rate=per,
                      tanh=tanh, mma=packed[0][1])
        b = K.LowRank(packed[1][0], ranks[1], offs[1], outs[1], out=out1, mma=packed[1][1])
        src = Partials(parts) if kind == "exp_decay" else low
        if a.mma == b.mma:
            K.low_rank_expand(src, cols, _i32(ent), n, dtype, a, b)
        else:
            K.low_rank_expand(src, cols, _i32(ent), n, dtype, a)
            K.low_rank_expand(src, cols, _i32(ent), n, dtype, b)
        x0 = ln[:, offs[0]:offs[0] + ranks[0]]
        z = (np.tanh(x0) if tanh else x0) @ wn[0].T
        if kind == "soft_decay":
            want = np.exp(-np.exp(rate[np.arange(outs[0]) // per]) * pp.softplus(z + bias))
        else:
            want = np.exp(-np.exp(z + bias)) if kind == "exp_decay" else z
        tol = 2e-5 if exact else 8e-3 if tanh or kind == "plain" else 2e-5       # (tanh is rounded once on the way in)
        g0, g1 = _np(out0), _np(out1)
        assert np.abs(g0[keep, :outs[0]] - want[keep]).max() < tol * max(1.0, np.abs(want).max()), kind
        assert (g0[:, outs[0]:] == 5.0).all() and (g0[~keep] == 5.0).all() and (g1[~keep] == 5.0).all()
        want1 = ln[:, offs[1]:offs[1] + ranks[1]] @ wn[1].T
        assert np.abs(g1[keep] - want1[keep]).max() < (2e-5 if exact else 8e-3) * max(1.0, np.abs(want1).max()), kind


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, H, d", [(1, 3, 16), (8, 5, 40), (70, 2, 64), (200, 33, 8)])
def test_bonus_rides_along_with_the_low_rank_product(K, dtype, n, H, d):
    """One launch for the decay and for r, k, v and the bonus gives what two launches give, row by row."""
    rng = np.random.default_rng(n)
    hd, rank = H * d, 10
    cols = 3 * hd + rank
    proj = _dev(rng.standard_normal((n, cols)), dtype)
    u = _dev(rng.standard_normal((H, d)))
    w, mma = K.pack_low_rank(_dev(rng.standard_normal((hd, rank)) * 0.3, dtype), dtype == torch.float32)
    bias = _dev(rng.standard_normal(hd))
    ent = np.zeros(n, dtype=np.int32)
    if n > 4:
        ent[3] = -1
    one, two = (torch.full((n, 4 * hd + H), 5.0, device=DEV) for _ in range(2))
    part = lambda aux: K.LowRank(w, rank, 3 * hd, hd, out=aux[:, 3 * hd:], kind="exp_decay", bias=bias, tanh=True, mma=mma)
    K.low_rank_expand(proj, cols, _i32(ent), n, dtype, part(one), bonus=K.Bonus(u, one, 4 * hd, H, d, d))
    K.bonus_prep(proj, cols, _i32(ent), u, two, 4 * hd, H, d, d, dtype)
    K.low_rank_expand(proj, cols, _i32(ent), n, dtype, part(two))
    assert torch.equal(one, two)
    if n > 4:
        assert (one[3] == 5.0).all()


@pytest.mark.parametrize("mode", ["delta", "bonus"])
@pytest.mark.parametrize("H, G, dk, dv", [(2, 2, 16, 8), (4, 2, 24, 40), (1, 1, 64, 32), (6, 3, 48, 16), (2, 1, 128, 128),
                                          (1, 1, 300, 20), (3, 1, 32, 12), (2, 2, 256, 4), (5, 5, 8, 8)])
def test_matrix_state_scan_with_a_decay_per_channel(K, mode, H, G, dk, dv):
    """The delta rule whose decay differs between key channels and between heads that share a query and a key,
    and the recurrence whose read-out comes before its write, over portions, single tokens and a slot used
    again, from a pool full of another request's numbers.  Decays near 1 and a large first token: a state
    that is lost or started anew shows at every later read-out."""
    rng = np.random.default_rng(dk + dv)
    Hq = G if mode == "delta" else H
    u = rng.standard_normal((H, dk))
    data = []
    for n in PLAN_LENS:
        q, k, v = rng.standard_normal((n, Hq, dk)), rng.standard_normal((n, Hq, dk)), rng.standard_normal((n, H, dv))
        v[0] *= 8.0
        w = 0.93 + 0.07 * rng.random((n, H, dk))
        if mode == "delta":
            k, q, b = pp.unit_vector(k), pp.unit_vector(q), rng.random((n, H))
            want = pp.channel_delta_scan(q, k, v, b, w)[0]
        else:
            k[0] *= 3.0
            want = pp.bonus_scan(q, k, v, w, u)[0]
            b = (q * u * k).sum(-1)
        at_w = -(-(2 * Hq * dk + H * dv + H) // 4) * 4
        row = np.zeros((n, at_w + H * dk))
        row[:, :2 * Hq * dk + H * dv + H] = np.concatenate([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), b], axis=1)
        row[:, at_w:] = w.reshape(n, -1)
        data.append((row.astype(np.float32), want))
    qk, hv = Hq * dk, H * dv
    rows_, lanes = K.matrix_state_plan(dk)
    floats = H * rows_ * lanes * dv
    state = torch.full((4, floats + 5), 1e3, device=DEV)
    err = _err()
    for ctx, ents in _steps_of(PLAN_LENS, PLAN, 1):
        aux = torch.cat([_dev(data[r][0][b:b + t]) for r, b, t, _ in ents] + [torch.full((1, data[0][0].shape[1]), 7.0, device=DEV)])
        n = aux.shape[0] - 1
        o = torch.full((n + 1, hv), 5.0, device=DEV)
        K.matrix_state_scan(aux, (0, qk, 2 * qk, at_w, 2 * qk + hv), True, mode, H // Hq, ctx, state, o, H, dk, dv, err)
        got = _np(o[:n]).reshape(n, H, dv)
        assert (o[n] == 5.0).all()
        at = 0
        for r, b, t, _ in ents:
            want = data[r][1][b:b + t]
            assert np.abs(got[at:at + t] - want).max() < 3e-5 * max(1.0, np.abs(want).max()), (r, b, t)
            at += t
    assert (state[:, floats:] == 1e3).all() and (state[3] == 1e3).all()
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shared, sigmoid", [(True, True), (False, False), (False, True)])
@pytest.mark.parametrize("dv, gate_off", [(40, 7), (40, 6), (300, 0), (128, 8)])
def test_head_norm_gate_options(K, dtype, shared, sigmoid, dv, gate_off):
    rng = np.random.default_rng(3)
    n, H, eps = 11, 3, 1e-3
    cols = gate_off + H * dv + 2
    o_raw = rng.standard_normal((n, H, dv)) * 0.03                 # small, so that eps counts
    proj = _dev(rng.standard_normal((n, cols)), dtype)
    nw = rng.standard_normal(dv if shared else H * dv)
    out = torch.empty(n, H * dv, dtype=dtype, device=DEV)
    K.head_norm_gate(_dev(o_raw.reshape(n, -1)), proj, cols, gate_off, _i32(np.zeros(n)), _dev(nw), eps, out, H, dv, sigmoid=sigmoid)
    gate = _np(proj)[:, gate_off:gate_off + H * dv].reshape(n, H, dv)
    want = pp.over_rms(o_raw, eps) * (nw if shared else nw.reshape(H, dv)) * (pp.sigmoid(gate) if sigmoid else pp.silu(gate))
    assert np.abs(_np(out).reshape(n, H, dv) - want).max() < (2e-5 if dtype == torch.float32 else 2e-2) * max(1.0, np.abs(want).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, d, dv, taps", [(4, 2, 16, 24, 3), (5, 1, 16, 8, 1), (3, 3, 24, 16, 5), (4, 4, 64, 128, 4),
                                               (6, 3, 128, 70, 4), (2, 1, 8, 130, 4), (3, 1, 66, 64, 2), (2, 2, 9, 7, 4)])
@pytest.mark.parametrize("plan, lens", [(PLAN, PLAN_LENS), (PLAN_LONG, PLAN_LONG_LENS)])
def test_conv_prep_without_a_decay(K, dtype, H, G, d, dv, taps, plan, lens):
    """Other columns for beta, no decay formed, the columns where it would be left alone; steps of many tokens,
    whose tiles of tokens hold the ends and beginnings of entries, beside steps of few."""
    rng = np.random.default_rng(taps)
    C = 2 * G * d + H * dv
    b_off = C + 5
    cols = b_off + H + 3
    cols += cols % 2
    conv_w = rng.standard_normal((C, taps))
    proj = [_dev(rng.standard_normal((n, cols)), dtype) for n in lens]
    state = torch.full((4, 2 + (taps - 1) * C), 1e3, device=DEV)
    err = _err()
    for ctx, ents in _steps_of(lens, plan):
        ctx.all_single = all(t == 1 for _, _, t, _ in ents)        # (the engine says so: the inputs then move on in one kernel)
        rows = torch.cat([proj[r][b:b + t] for r, b, t, _ in ents])
        n = rows.shape[0]
        wide = C + 4 + H + (C + H) % 2
        aux = torch.full((n, wide), 5.0, device=DEV)
        K.conv_delta_prep(rows, cols, ctx, state, 2, _dev(conv_w), taps, None, None, aux, H, G, d, dv, 1e-6, d ** -0.5, err, dtype,
                          b_off=b_off, a_off=-1, w_off=0, beta_off=C + 4)
        got = _np(aux)
        at = 0
        for r, b, t, _ in ents:
            x = _np(proj[r])
            y = pp.silu(pp.short_convolution(x[:, :C], conv_w)[0])
            q = pp.unit_vector(y[:, :G * d].reshape(-1, G, d)) * d ** -0.5
            k = pp.unit_vector(y[:, G * d:2 * G * d].reshape(-1, G, d))
            want = np.concatenate([q.reshape(len(x), -1), k.reshape(len(x), -1), y[:, 2 * G * d:]], axis=1)[b:b + t]
            assert np.abs(got[at:at + t, :C] - want).max() < 2e-5, (r, b)
            assert np.abs(got[at:at + t, C + 4:C + 4 + H] - pp.sigmoid(x[b:b + t, b_off:b_off + H])).max() < 1e-6
            at += t
        assert (got[:, C:C + 4] == 5.0).all()
    assert int(err.item()) == 0


@pytest.mark.parametrize("experts, top", [(3, 3), (12, 1), (6, 2), (64, 6), (40, 8)])
def test_route_by_sigmoid_scores(K, experts, top):
    rng = np.random.default_rng(experts)
    n = 29
    z = (rng.standard_normal((n, experts)) * 3).astype(np.float32)
    z[0] = 40.0 + np.arange(experts)                     # scores that all round to 1: the logits still order them
    z[1] = 0.25                                          # all equal: the lowest indices
    z[2] = -30.0 - np.arange(experts)                    # scores near zero
    from crane_b200.kernels import Partials
    route, route2 = torch.full((n, experts), 5.0, device=DEV), torch.full((n, experts), 5.0, device=DEV)
    K.route_grouped(_dev(z), None, route, experts, top, 1, 1, False, sigmoid=True)
    # the logits left as partial sums
    K.route_grouped(Partials(torch.stack([_dev(z), torch.zeros(n, experts, device=DEV)])), None, route2, experts, top, 1, 1, False,
                    sigmoid=True)
    assert torch.equal(route, route2)
    got = _np(route)
    for t in range(n):
        order = sorted(range(experts), key=lambda e: (-float(z[t, e]), e))[:top]
        want = np.zeros(experts)
        want[order] = pp.sigmoid(z[t, order].astype(np.float64))
        assert np.abs(got[t] - want).max() < 1e-6 and set(np.nonzero(got[t])[0]) == set(order), t


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("F", [6, 16, 264])
def test_weight_on_the_experts_input(K, dtype, F):
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(8)
    n, E = 7, 4
    cols = E * F
    route = rng.random((n, E)).astype(np.float32)
    route[:, 2] = 0.0
    for form in ("whole", "parts"):
        parts = _dev(rng.standard_normal((2, n, 2 * cols)) * 2)
        gu = parts.sum(0).to(dtype)
        gn = _np(gu)
        out = torch.empty(n, cols, dtype=dtype, device=DEV)
        K.gated_activation(gu if form == "whole" else Partials(parts), out, _dev(route), E, F, cols, on_input=True)
        w = np.repeat(route.astype(np.float64), F, axis=1)
        want = pp.silu(w * gn[:, :cols]) * (w * gn[:, cols:])
        assert np.abs(_np(out) - want).max() < (1e-5 if dtype == torch.float32 else 2e-2) * np.abs(want).max(), form
        assert (out[:, 2 * F:3 * F] == 0).all()
        K.gated_activation(gu if form == "whole" else Partials(parts), out, _dev(route), E, F, cols)
        want = pp.silu(gn[:, :cols]) * gn[:, cols:] * w
        assert np.abs(_np(out) - want).max() < (1e-5 if dtype == torch.float32 else 2e-2) * np.abs(want).max(), form


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M", [1, 9, 64, 130, 257, 600])
@pytest.mark.parametrize("groups, features, tail, width", [(5, 256, 48, 192), (3, 128, 128, 200), (4, 96, 8, 64), (2, 40, 12, 100),
                                                           (5, 512, 64, 1024)])
def test_grouped_products(K, dtype, M, groups, features, tail, width):
    """Every output column reads its group's rows, whole or as partial sums, at one token and at hundreds;
    tiles' rows behind a group's own belong to the next group and must not be stored."""
    from crane_b200.kernels import Partials
    from crane_b200.parts import Runtime
    rng = np.random.default_rng(M + width)
    rt = Runtime(DEV, dtype, 640)
    xs = _dev(rng.standard_normal((groups, M, width)), dtype)
    N = (groups - 1) * features + tail
    w = _dev(rng.standard_normal((N, width)) * width ** -0.5, dtype)
    got = rt.linear_grouped(xs, w, features, "t")
    got = _np(got.sum(dtype) if isinstance(got, Partials) else got)
    xn, wn = _np(xs), _np(w)
    want = np.concatenate([xn[g] @ wn[g * features:min(N, (g + 1) * features)].T for g in range(groups)], axis=1)
    assert np.abs(got - want).max() < (2e-5 if dtype == torch.float32 else 2e-2) * np.abs(want).max()
    assert int(rt.err.item()) == 0


def test_grouped_product_on_pairs_of_sms(K):
    """The largest products: a tile by two SMs together."""
    from crane_b200.parts import Runtime
    rng = np.random.default_rng(1)
    G, M, width, features = 4, 2048, 2048, 2048
    rt = Runtime(DEV, torch.bfloat16, 2048)
    assert rt.kernels.pair_plan(M, (G - 1) * features + 64, width, rt.num_sms)[0]
    xs = torch.randn((G, M, width), device=DEV).to(torch.bfloat16)
    w = (torch.randn(((G - 1) * features + 64, width), device=DEV) * width ** -0.5).to(torch.bfloat16)
    got = rt.linear_grouped(xs, w, features, "t").float()
    want = torch.cat([xs[g].float() @ w[g * features:(g + 1) * features].float().t() for g in range(G)], dim=1)
    assert float((got - want).abs().max()) < 2e-2 * float(want.abs().max())
    assert int(rt.err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_prep_with_a_query_latent(K, dtype):
    """First launch: cache rows and the normed query latent; second: the rotation of the queries made from it."""
    rng = np.random.default_rng(4)
    H, dim, rot, rank, rq, ps = 3, 10, 8, 24, 20, 8
    rotp = {"dims": rot, "base": 100.0, "scaling": {"factor": 2.0, "original": 16, "fast": 4.0, "slow": 1.0}}
    f, mult = pp.yarn(rot, 100.0, rotp["scaling"])
    ang = np.arange(40)[:, None] * f[None]
    cos, sin = _dev(np.cos(ang) * mult), _dev(np.sin(ang) * mult)
    cols = rq + rank + rot + 3
    pos, ent = [13, 14, 15, 16, 8, 0], [0, 0, 0, 0, 1, -1]
    table = np.array([[5, 2, 7], [0, 4, -1]], dtype=np.int32)
    proj = _dev(rng.standard_normal((len(pos), cols)) * 0.05, dtype)                 # small, so that eps counts
    nw, cw, eps = rng.standard_normal(rank), rng.standard_normal(rq), 1e-3
    pool = torch.zeros(9, 1, ps, rank + rot, dtype=dtype, device=DEV)
    cq = torch.full((len(pos), rq), 5.0, dtype=dtype, device=DEV)
    err = _err()
    meta = (cos, sin, _i32(pos), _i32(ent), _i32(table), pool, ps)
    K.latent_prep(proj, cols, -1, rq + 3, H, dim, rot, rank, rot, *meta, _dev(nw), eps, None, err, cq_off=0, cq_w=_dev(cw), cq_out=cq)
    p64, tol = _np(proj), 2e-5 if dtype == torch.float32 else 2e-2
    got = _np(cq)
    want = pp.over_rms(p64[:, :rq], eps) * cw
    assert np.abs(got[:5] - want[:5]).max() < tol * np.abs(want).max() and (got[5] == 5.0).all()
    for t, (p, e) in enumerate(zip(pos, ent)):
        if e < 0:
            continue
        row = _np(pool)[table[e, p // ps], 0, p % ps]
        c = pp.over_rms(p64[t, rq + 3:rq + 3 + rank], eps) * nw
        kr = pp.rotate_pairs(p64[t:t + 1, rq + 3 + rank:], [p], rotp)[0]
        assert np.abs(row - np.concatenate([c, kr])).max() < tol * max(1.0, np.abs(c).max())
    before = pool.clone()
    q = _dev(rng.standard_normal((len(pos), H * (dim + rot))), dtype)
    q_abs = torch.zeros(len(pos), H * (rank + rot), dtype=dtype, device=DEV)
    K.latent_prep(q, H * (dim + rot), 0, -1, H, dim, rot, rank, rot, *meta, None, eps, q_abs, err)
    qr = pp.rotate_pairs(_np(q).reshape(-1, H, dim + rot)[..., dim:], pos, rotp)
    got_q = _np(q_abs).reshape(-1, H, rank + rot)
    assert np.abs(got_q[:5, :, rank:] - qr[:5]).max() < tol * 4 and np.abs(got_q[5]).max() == 0
    assert torch.equal(pool, before) and int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [0, 1, 5, 64, 100, 65])
@pytest.mark.parametrize("rank, rot, heads, ps", [(32, 16, 4, 16), (72, 8, 5, 8), (80, 16, 7, 32), (128, 32, 8, 64), (176, 48, 20, 16),
                                                  (20, 6, 3, 8)])
def test_latent_attention_window_and_sinks(K, dtype, window, rank, rot, heads, ps):
    """A prompt portion deep in a request, single tokens and a short prompt.  For some queries one key stands
    out: the oldest that a window still shows, the one just outside it (which must change nothing), the
    newest, and without a window the first of all.  Pages that a window has passed are gone (-1), and what
    stands in their storage is large.  Sinks from negligible to larger than any score."""
    from crane_b200.parts.latent_attention import latent_attention_kernel
    rng = np.random.default_rng(rank + heads + window)
    width, scale = rank + rot, 0.2
    lens, q_lens = [700, 3 * ps + 1, 2 * ps, 45, 300], [37, 1, 1, 45, 1]
    sinks = np.linspace(-3.0, 6.0, heads)
    sinks[-1] = 60.0                                     # above a planted key's score
    rows = [rng.standard_normal((n, width)) * 0.5 for n in lens]
    n_pages = sum(-(-n // ps) for n in lens) + 2
    order = rng.permutation(n_pages)
    pool = (torch.randn(n_pages, 1, ps, width, device=DEV) * 30).to(dtype)
    table = -np.ones((len(lens), max(-(-n // ps) for n in lens)), dtype=np.int32)
    nxt = 0
    for e, r in enumerate(rows):
        first = max(0, lens[e] - q_lens[e] + 1 - window) // ps if window else 0       # the first page still held
        for b in range(-(-len(r) // ps)):
            page = order[nxt]; nxt += 1
            if b >= first:
                table[e, b] = page
                pool[int(page), 0, :len(r[b * ps:(b + 1) * ps])] = _dev(r[b * ps:(b + 1) * ps], dtype)
        rows[e] = _np(_dev(r, dtype))
    qs, pos, ent, cu = [], [], [], [0]
    for e, (n, ql) in enumerate(zip(lens, q_lens)):
        q = rng.standard_normal((ql, heads, width)) * 0.5
        for t in {0, ql // 2, ql - 1}:
            p = n - ql + t
            lo = max(0, p - window + 1) if window else 0
            for h, key in ((0, lo), (1, lo - 1), (2 % heads, p), (heads - 1, lo)):
                if key >= 0:
                    q[t, h] = rows[e][key] * 40.0 / max(1e-6, (rows[e][key] ** 2).sum() * scale)
        qs.append(q)
        pos += list(range(n - ql, n)); ent += [e] * ql; cu.append(cu[-1] + ql)
    q_all = _dev(np.concatenate(qs).reshape(-1, heads * width), dtype)
    out = torch.zeros(q_all.shape[0], heads * rank, dtype=dtype, device=DEV)
    err = _err()
    latent_attention_kernel(K, q_all, out, pool, _i32(pos), _i32(ent), _i32(cu), _i32(lens), np.asarray(cu), np.asarray(lens),
                            _i32(table), ps, heads, rank, rot, scale, err, exact=dtype == torch.float32, window=window,
                            sinks=_dev(sinks))
    got = _np(out).reshape(-1, heads, rank)
    q64 = _np(q_all).reshape(-1, heads, width)
    tol = 3e-5 if dtype == torch.float32 else 2.5e-2
    for i, (p, e) in enumerate(zip(pos, ent)):
        see = pp.visible(p, np.arange(p + 1), window)
        s = np.where(see[:, None], (rows[e][:p + 1] @ q64[i].T) * scale, -np.inf)
        want = np.stack([pp.sink_softmax(s[:, h], sinks[h]) @ rows[e][:p + 1, :rank] for h in range(heads)])
        assert np.abs(got[i] - want).max() < tol * max(1.0, np.abs(want).max()), (i, p, e)
    assert int(err.item()) == 0
    # the same as a captured graph's step would launch it: bounds by the shape alone
    if dtype == torch.bfloat16:
        out2 = torch.zeros_like(out)
        latent_attention_kernel(K, q_all, out2, pool, _i32(pos), _i32(ent), _i32(cu), _i32(lens), np.asarray(cu), np.asarray(lens),
                                _i32(table), ps, heads, rank, rot, scale, err, exact=False, padded=q_all.shape[0], window=window,
                                sinks=_dev(sinks))
        assert float((out2.float() - out.float()).abs().max()) < 2.5e-2 and int(err.item()) == 0


# ---------------------------------------------------------------- generation
def _load(folder, dtype, **opts):
    from crane_b200.generation import ModelForCausalLM
    return ModelForCausalLM.from_pretrained(folder, dtype, **opts)


def _greedy(n):
    from crane_b200.generation import GenerationConfig
    return GenerationConfig(max_new_tokens=n, temperature=None, eos_token_id=-1)


@pytest.mark.parametrize("name", SMALL)
def test_greedy_generation_float32_equals_plain(name, model_folders):
    folder = model_folders(name, "float32")
    cfg, w = pp.load_folder(folder)
    m = _load(folder, "fp32", page_size=tp.TINY[name]["page_size"], num_pages=24, max_concurrent=3,
              max_batched_tokens=64, max_seq_len=192)
    rng = np.random.default_rng(3)
    for n in (1, 5, 17):
        prompt = rng.integers(0, cfg["vocab"], n).tolist()
        assert m.generate(prompt, _greedy(8)) == pp.greedy_generate(cfg, w, prompt, 8)
    m.runner.table.check()
    assert m.runner.table.live() == 0


@pytest.mark.parametrize("name", ["PA", "PL"])
def test_greedy_batch_bfloat16_through_the_scheduler(name, model_folders):
    """Six prompts, three slots, portions of at most 16 tokens: requests wait, slots and pages are used
    again, and decode steps replay the batch-size buckets' graphs with the recurrent states in them."""
    folder = model_folders(name, "bfloat16")
    cfg, w = pp.load_folder(folder)
    m = _load(folder, "bf16", page_size=16, num_pages=40, max_concurrent=3, max_batched_tokens=48, chunk_size=16,
              max_seq_len=256)
    rng = np.random.default_rng(4)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (12, 3, 40, 1, 25, 7)]
    outs = m.generate_batch(prompts, _greedy(20))
    ok = 0
    for prompt, toks in zip(prompts, outs):
        assert len(toks) == len(prompt) + 20 and toks[:len(prompt)] == prompt
        logits = pp.logits_all(cfg, w, toks[:-1])
        for i in range(len(prompt), len(toks)):
            row = logits[i - 1]
            # (a token that another rounding would not have chosen does not end the comparison: every later one is
            # checked against the plain logits of the sequence as it was generated)
            ok += bool(row[toks[i]] >= row.max() - 3e-2 * np.abs(row).max())
    assert ok >= 0.95 * 20 * len(prompts), ok
    m.runner.table.check()
    assert m.runner.table.live() == 0
    assert m.runner.graph_replays > 0 and m.runner._pad_with_copies       # (the batch-size buckets)


def test_command_line(model_folders):
    """bin/crane picks the model class from config.json."""
    import os
    import subprocess
    import sys
    folder = model_folders("PA", "float32")
    cfg, w = pp.load_folder(folder)
    crane = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "crane")
    cmd = [sys.executable, crane, "-m", folder, "--dtype", "fp32", "--prompt-ids", "5,6,7", "--max-new-tokens", "6",
           "--eos-token-id", "-1", "--page-size", "16", "--num-pages", "8", "-c", "2", "--max-batched-tokens", "32",
           "--max-seq-len", "64"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-3000:]
    assert p.stdout.strip().splitlines()[-1] == ",".join(map(str, pp.greedy_generate(cfg, w, [5, 6, 7], 6)[3:]))
