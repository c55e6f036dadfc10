"""Mufalix on the GPU: replay through bin/trace_run against the plain implementation (whole prompts, tails
decoded token by token, portions down to two tokens, mixed batches in a pool so small that pages and slots
are used again, windows that give pages back), every new kernel and option alone against NumPy, keys
planted just inside and just outside a window, far away and at page borders, states and kept inputs across
steps and slots used again, and greedy generation through the Python entry point, the scheduler and the
command line."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_mufalix as pm
import tiny_mufalix as tm
import trace_tools as tt

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
SMALL = ["FA", "FB", "FC", "FD"]
LENGTHS = {"FA": [1, 2, 19, 100, 65, 48, 33], "FB": [5, 41, 97, 150, 34, 64], "FC": [3, 70, 140, 17], "FD": [2, 110, 31, 16, 77],
           "FL": [7, 150, 320, 64]}


@pytest.fixture(scope="module")
def cases(model_folders):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            folder = model_folders(name, dtype)
            rng = np.random.default_rng(1300 + ord(name[1]))
            reqs = tt.make_requests(rng, tm.TINY[name]["config"]["vocab"], LENGTHS[name[:2]])
            cfg, w = pm.load_folder(folder)
            made[(name, dtype)] = (folder, reqs, {r: pm.logits_all(cfg, w, t) for r, t in reqs.items()})
        return made[(name, dtype)]
    return get


# In bfloat16 a router's choice between two experts whose scores differ by less than its input's rounding is a
# toss-up, and the other expert's output counts in full.  So bfloat16 whole-model logits are compared closely at
# the same configurations with every expert chosen ("-all"), and at the others loosely.  (Heads whose read-out happens
# to be small are normed all the same, which shows rounding many times over in a few rows, in 32-bit too.)
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
    elif label.split()[1].endswith("-all"):
        assert np.median(errs) <= 2.5e-2 and errs[int(0.9 * (len(errs) - 1))] <= 6e-2, label
    else:
        assert np.median(errs) <= 0.1, label


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in SMALL] + [(n + "-all", "bfloat16") for n in SMALL] + [("FA", "bfloat16")])
def test_alone_whole_tail_portions(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tm.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_whole(tb, reqs)
    tt.trace_tail_decode(tb, reqs)
    tt.trace_portions(tb, reqs, np.random.default_rng(7))
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"))
    _compare(got, tb, plain, dtype, f"config {name}")
    if dtype == "float32":
        tt.compare_cuts([(got, tb)], dtype, f"config {name}", tol=2e-5)


@pytest.mark.parametrize("name, dtype", [(n, "float32") for n in SMALL] + [(n + "-all", "bfloat16") for n in SMALL] + [("FA", "bfloat16")])
def test_mixed_with_page_and_slot_reuse(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tm.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_mixed(tb, reqs, np.random.default_rng(11), max_live=3)
    assert tb.pages_taken > tb.peak_tokens // ps, "the trace must make the pool hand pages out again"
    assert max(len(s["entries"]) for s in tb.steps) >= 3
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"),
                       extra_args=["--max-live", "3"])          # three slots for all requests
    _compare(got, tb, plain, dtype, f"config {name} mixed")


@pytest.mark.parametrize("name, dtype", [("FA", "float32"), ("FC", "float32"), ("FL-all", "bfloat16")])
def test_long_decoding(name, dtype, cases, tmp_path):
    """Decoded past every window many times over."""
    folder, reqs, plain = cases(name, dtype)
    ps = tm.TINY[name]["page_size"]
    longest = max(reqs, key=lambda r: len(reqs[r]))
    tb = tt.TraceBuilder(ps)
    tt.trace_tail_decode(tb, {longest: reqs[longest]}, tail=len(reqs[longest]) - 3)
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"))
    _compare(got, tb, plain, dtype, f"config {name} decoded")


@pytest.mark.parametrize("name, dtype", [("FL", "float32"), ("FL", "bfloat16"), ("FL-all", "bfloat16")])
def test_layer_sizes_of_the_tensor_core_kernels(name, dtype, cases, tmp_path):
    folder, reqs, plain = cases(name, dtype)
    ps = tm.TINY[name]["page_size"]
    tb = tt.TraceBuilder(ps)
    tt.trace_whole(tb, reqs)
    tt.trace_tail_decode(tb, reqs, tail=40)
    tt.trace_portions(tb, reqs, np.random.default_rng(3))
    tt.trace_mixed(tb, reqs, np.random.default_rng(5))
    # (single tokens beside portions take the decode kernel from the first cached key on)
    got = tt.run_trace(folder, dtype, tb.steps, tb.peak_tokens, ps, str(tmp_path / "out"),
                       extra_args=["--mixed-decode-min-keys", "1"])
    _compare(got, tb, plain, dtype, f"config {name}", tol_rms=6e-5)
    if dtype == "float32":
        tt.compare_cuts([(got, tb)], dtype, "config FL", tol=6e-5)


def test_a_window_gives_pages_back(model_folders):
    """A model all of whose caches have windows decodes further than its pool holds pages for."""
    from crane_b200.config import EngineConfig
    from crane_b200.engine import ModelRunner, StepEntry
    folder = model_folders("FA", "float32")
    cfg, w = pm.load_folder(folder)
    ps = 8
    runner = ModelRunner(folder, EngineConfig(dtype="float32", page_size=ps, num_pages=5, max_concurrent=2,
                                              max_batched_tokens=64, max_seq_len=256))
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 120).tolist()
    want = pm.logits_all(cfg, w, toks)
    pos = 0
    for n in [20, 9, 2] + [1] * 89:
        got = runner.step([StepEntry(1, toks[pos:pos + n], [n - 1])]).cpu().numpy()[0]
        pos += n
        assert np.abs(got - want[pos - 1]).max() < 5e-5 * np.abs(want).max(), pos
    runner.rt.check_errors()
    runner.table.check()
    assert pos == 120 > 5 * ps


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
# step; slots in no order.  The long plan goes past the kernels' tiles and rounds of 128 tokens.
PLAN = [[(0, 20, 2), (1, 1, 0), (2, 4, 1)], [(2, 5, 1), (0, 1, 2)], [(0, 1, 2)], [(0, 15, 2), (3, 2, 0)], [(3, 9, 0)]]
PLAN_LENS = [37, 1, 9, 11]
PLAN_LONG = [[(0, 300, 2), (1, 2, 0), (2, 1, 1), (3, 6, 3)], [(2, 129, 1), (0, 1, 2), (3, 1, 3)], [(0, 3, 2), (3, 128, 3)],
             [(0, 1, 2), (3, 2, 3)], [(2, 1, 1), (0, 1, 2)], [(0, 1, 2), (2, 1, 1), (3, 1, 3)], [(2, 3, 1), (0, 131, 2)], [(0, 1, 2)]]
PLAN_LONG_LENS = [439, 2, 135, 138]
PLANS = [(PLAN, PLAN_LENS), (PLAN_LONG, PLAN_LONG_LENS)]


def _steps_of(lens, plan, pad=0):
    """Per step the kernels' metadata and, per entry, (request, first position, count, slot).  ``pad``: that many
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
                              tok_entry=_i32(np.concatenate([np.full(t, i) for i, t in enumerate(q_lens)] + [np.full(pad, -1)])),
                              all_single=all(t == 1 for _, _, t, _ in ents))
        yield ctx, ents
    assert done == list(lens)


def _rows(per_request, ents, pad, fill=0.0):
    rows = torch.cat([per_request[r][b:b + t] for r, b, t, _ in ents])
    if not pad:
        return rows
    return torch.cat([rows, torch.full((pad, rows.shape[1]), fill, dtype=rows.dtype, device=rows.device)])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, d, dv, cap", [(2, 16, 8, 5.0), (3, 24, 40, 15.0), (1, 64, 32, 2.0), (2, 128, 64, 15.0), (1, 300, 20, 9.0),
                                           (5, 9, 7, 30.0), (4, 32, 32, 15.0), (1, 256, 4, 1.0), (9, 8, 12, 15.0)])
@pytest.mark.parametrize("plan, lens", PLANS)
def test_exponential_gates_over_steps(K, dtype, H, d, dv, cap, plan, lens):
    """Gates, state, normaliser and running maximum over portions, single tokens, padding and a slot used again,
    from slots full of another request's numbers.  Forget gates near 1 and an early token with a large input
    gate: a state or a maximum that is lost shows at every later read-out; later a stretch of tiny input
    gates (the floor exp(-M) decides) and forget gates that forget."""
    rng = np.random.default_rng(d + dv)
    hd, hv = H * d, H * dv
    g_off = 2 * hd + hv + 3
    g_off += g_off % 2
    cols = g_off + 2 * H + 2
    cols += cols % 2 if d != 9 else 1 - cols % 2
    bi, bf = rng.standard_normal(H), rng.standard_normal(H) + 2.0
    nw = rng.standard_normal(hv)
    proj, want_rows = [], []
    for n in lens:
        x = rng.standard_normal((n, cols))
        x[:, g_off:g_off + H] *= 2.0
        x[:, g_off + H:g_off + 2 * H] = x[:, g_off + H:g_off + 2 * H] * 2 + 4.0
        x[0, g_off:g_off + H] += 6.0
        x[n // 2:n // 2 + 5, g_off:g_off + H] -= 30.0
        x[min(n - 1, n // 2 + 2), g_off + H:g_off + 2 * H] -= 30.0
        x = _dev(x, dtype)
        proj.append(x)
        x = _np(x)
        zi, zf = x[:, g_off:g_off + H] + bi, x[:, g_off + H:g_off + 2 * H] + bf
        o, _ = pm.stabilised_scan(x[:, :hd].reshape(n, H, d) * d ** -0.5, x[:, hd:2 * hd].reshape(n, H, d),
                                  x[:, 2 * hd:2 * hd + hv].reshape(n, H, dv), cap * np.tanh(zi / cap),
                                  pm.log_sigmoid(cap * np.tanh(zf / cap)))
        want_rows.append(pm.over_rms(o, 1e-5).reshape(n, hv) * nw * pm.sigmoid(x[:, :hv]))     # (q's columns serve as a gate)
    rows_, lanes = K.matrix_state_plan(d)
    m_off = H * rows_ * lanes * (dv + 1)
    state = torch.full((4, m_off + H + 3), 1e3, device=DEV)
    err, pad = _err(), 2
    w_at = 2 * hd + hv
    aux_cols = -(-(w_at + 3 * H) // 4) * 4
    gate_ok = hv <= cols
    assert gate_ok
    for ctx, ents in _steps_of(lens, plan, pad):
        x = _rows(proj, ents, pad, 9.0)
        n = x.shape[0]
        aux = torch.full((n, aux_cols), 5.0, device=DEV)
        K.exp_gate_prep(x, cols, ctx, state, m_off, _dev(bi), _dev(bf), cap, d ** -0.5, aux, H, d, dv, g_off, g_off + H, w_at, err, dtype)
        o_raw, den = torch.full((n, hv), 5.0, device=DEV), torch.full((n, H), 5.0, device=DEV)
        K.matrix_state_scan(aux, (0, hd, 2 * hd, w_at, w_at + H), False, "gated", 1, ctx, state, o_raw, H, d, dv, err, den=den)
        out = torch.full((n, hv), 5.0, dtype=dtype, device=DEV)
        K.head_norm_gate(o_raw, x, cols, 0, ctx.tok_entry, _dev(nw), 1e-5, out, H, dv, sigmoid=True, den=den,
                         floor=aux[:, w_at + 2 * H:], den_eps=1e-6)
        got, at = _np(out), 0
        for r, b, t, _ in ents:
            want = want_rows[r][b:b + t]
            tol = 1e-4 if dtype == torch.float32 else 2e-2
            assert np.abs(got[at:at + t] - want).max() < tol * max(1.0, np.abs(want).max()), (r, b, t)
            at += t
        assert (aux[at:] == 5.0).all() and (o_raw[at:] == 5.0).all() and (den[at:] == 5.0).all() and (out[at:] == 5.0).all()
    assert (state[:, m_off + H:] == 1e3).all() and (state[3] == 1e3).all() == (plan is PLAN)
    assert int(err.item()) == 0


@pytest.mark.parametrize("H, d, dv, lens", [(2, 16, 8, [64]), (3, 32, 24, [63, 1, 65, 23, 24, 200]), (1, 64, 64, [300]), (2, 128, 40, [130, 64]),
                                            (1, 256, 16, [97]), (1, 144, 48, [200, 30]), (4, 48, 136, [3, 70])])
@pytest.mark.parametrize("spread", [1.0, 6.0])
def test_chunks_of_the_matrix_memory_equal_the_walk(K, H, d, dv, lens, spread):
    """Portions in chunks of 64 tokens against the walk token by token, read-outs and normalisers in 32-bit and the
    states they leave, for fresh and continued requests; entries below the limit are left to the walk.  ``spread``
    1: forget gates near 1, so the first token shows in the last; 6: gates from one end to the other."""
    rng = np.random.default_rng(d + dv)
    hd, hv = H * d, H * dv
    cols = -(-(2 * hd + 2 * hv + 2 * H) // 8) * 8
    g_off = 2 * hd + 2 * hv
    n, w_at = sum(lens), 2 * hd + hv
    x = rng.standard_normal((n, cols))
    x[:, g_off:g_off + H] *= spread
    x[:, g_off + H:g_off + 2 * H] = x[:, g_off + H:g_off + 2 * H] * spread * 1.5 + (7.0 if spread == 1.0 else 2.0)
    cu = np.concatenate([[0], np.cumsum(lens)])
    x[cu[:-1], 2 * hd:2 * hd + hv] *= 8.0
    x = _dev(x, torch.bfloat16)
    start = [0 if i % 2 == 0 else 77 for i in range(len(lens))]
    ctx = SimpleNamespace(cu_q=_i32(cu), kv_len=_i32(np.asarray(lens) + start), slots=_i32(rng.permutation(len(lens))),
                          tok_entry=_i32(np.repeat(np.arange(len(lens)), lens)))
    rows_, lanes = K.matrix_state_plan(d)
    m_off = H * rows_ * lanes * (dv + 1)
    seed = torch.randn(len(lens), m_off + H + 1, device=DEV)
    if rows_ * lanes > d:                                    # rows past the keys are zeros and stay so
        st = seed[:, :m_off].view(len(lens), H, rows_, dv + 1, lanes)
        r = torch.arange(lanes, device=DEV)[None] * rows_ + torch.arange(rows_, device=DEV)[:, None]
        st *= (r < d)[None, None, :, None, :]
    err, bias = _err(), _dev(np.zeros(H))
    least = 24
    got = {}
    for way in ("walk", "chunks"):
        state = seed.clone()
        aux = torch.full((n, -(-(w_at + 3 * H) // 4) * 4), 5.0, device=DEV)
        o_raw, den = torch.full((n, hv), 5.0, device=DEV), torch.full((n, H), 5.0, device=DEV)
        logs = torch.full((n, 2 * H), 5.0, device=DEV) if way == "chunks" else None
        K.exp_gate_prep(x, cols, ctx, state, m_off, bias, bias, 15.0, d ** -0.5, aux, H, d, dv, g_off, g_off + H, w_at, err, torch.bfloat16,
                        logs=logs, logs_min=least)
        if logs is not None:
            assert K.memory_chunks_takes(x, cols, d, dv)
            K.memory_chunks(x, cols, (0, hd, 2 * hd), logs, ctx, state, o_raw, den, H, d, dv, d ** -0.5, least, err)
            short = np.repeat(np.asarray(lens) < least, lens)
            assert (o_raw[torch.from_numpy(short).to(DEV)] == 5.0).all()
        if logs is None or min(lens) < least:
            K.matrix_state_scan(aux, (0, hd, 2 * hd, w_at, w_at + H), False, "gated", 1, ctx, state, o_raw, H, d, dv, err, den=den,
                                max_len=least if logs is not None else 0)
        got[way] = (_np(o_raw), _np(den), _np(state), _np(aux)[:, w_at + 2 * H:w_at + 3 * H])
    for a, b, what in zip(got["walk"], got["chunks"], ("read-outs", "normalisers", "states", "floors")):
        assert np.abs(a - b).max() < 1e-4 * np.abs(a).max(), what
    o, den = got["walk"][:2]
    rms = lambda a: np.sqrt((a.reshape(n, H, -1) ** 2).mean(axis=(1, 2)))          # and token by token
    assert (rms(o - got["chunks"][0]) < 2e-3 * rms(o) + 1e-5 * rms(o).max()).all()
    assert int(err.item()) == 0


@pytest.mark.parametrize("n", [1, 3, 31, 128, 129, 700])
def test_exponential_gates_alone(K, n):
    """The three numbers per token against the walk in NumPy, from a maximum the request brings along, whole and
    as partial sums."""
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(n)
    H, d, dv, cap = 3, 2, 2, 15.0
    cols = 2 * H * d + H * dv + 2 * H
    parts = _dev(rng.standard_normal((2, n, cols)) * 4)
    x = _np(parts.sum(0))
    z = np.zeros(H)
    li = cap * np.tanh(x[:, -2 * H:-H] / cap)
    lf = pm.log_sigmoid(cap * np.tanh(x[:, -H:] / cap))
    M = np.array([-4.0, 0.5, 12.0])
    start = M.copy()
    want = np.zeros((n, 3, H))
    for t in range(n):
        new = np.maximum(lf[t] + M, li[t])
        want[t] = np.exp(lf[t] + M - new), np.exp(li[t] - new), np.exp(-new)
        M = new
    ctx = SimpleNamespace(cu_q=_i32([0, n]), kv_len=_i32([n + 5]), slots=_i32([1]), tok_entry=_i32(np.zeros(n)))
    err = _err()
    for form in ("whole", "parts"):
        state = torch.zeros((2, 7 + H), device=DEV)
        state[1, 7:] = _dev(start)
        aux = torch.zeros((n, 2 * H * d + H * dv + 3 * H), device=DEV)
        K.exp_gate_prep(parts.sum(0) if form == "whole" else Partials(parts), cols, ctx, state, 7, _dev(z), _dev(z), cap, 0.5, aux, H, d, dv,
                        cols - 2 * H, cols - H, 2 * H * d + H * dv, err, torch.float32)
        got = _np(aux)[:, -3 * H:].reshape(n, 3, H)
        assert np.abs(got - want).max() < 3e-5 * max(1.0, want.max()), form
        assert np.abs(_np(state)[1, 7:] - M).max() < 2e-5 and (state[0] == 0).all()
        assert np.abs(_np(aux)[:, :H * d] - 0.5 * x[:, :H * d]).max() < 1e-6
        assert np.abs(_np(aux)[:, H * d:2 * H * d + H * dv] - x[:, H * d:2 * H * d + H * dv]).max() < 1e-6
    assert int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C, parts, taps", [(40, 4, 3), (64, 1, 4), (512, 2, 4), (96, 3, 1), (60, 2, 5), (800, 2, 2), (33, 3, 16), (160, 2, 4),
                                            (336, 7, 2)])
@pytest.mark.parametrize("plan, lens", PLANS)
def test_gated_linear_recurrence_over_steps(K, dtype, C, parts, taps, plan, lens):
    """Convolution, gates, state and ring over portions, single tokens (one kernel), padding and a slot used again,
    from slots full of another request's numbers; decays from almost 1 (a large first input shows to the end)
    to almost 0."""
    rng = np.random.default_rng(C + taps)
    c = C // parts
    off = 2
    cols = 2 * C + off + 2
    conv_w, conv_b = rng.standard_normal((C, taps)), rng.standard_normal(C)
    mats = [_dev(rng.standard_normal((parts, c, c)) * c ** -0.5, dtype) for _ in range(2)]
    rb, ib = rng.standard_normal(C), rng.standard_normal(C)
    lam = np.where(np.arange(C) % 3 == 0, -9.0, rng.standard_normal(C) * 2)
    gates, mma = K.pack_gates(*mats, dtype == torch.float32)
    assert mma == (dtype == torch.bfloat16 and -(-c // 16) * 16 <= 384)
    scan = K.GateScan(y_off=off, x_off=off + C, s_off=1, ring_off=3 + C, conv_w=_dev(conv_w.T.copy()), conv_b=_dev(conv_b), gates=gates, mma=mma,
                      rb=_dev(rb), ib=_dev(ib), sp=_dev(pm.softplus(lam)), parts=parts)
    proj, want_rows, kept = [], [], []
    for n in lens:
        x = rng.standard_normal((n, cols))
        x[0, off + C:off + 2 * C] *= 20.0
        x = _dev(x, dtype)
        proj.append(x)
        x = _np(x)
        u, _ = pm.short_convolution(x[:, off + C:off + 2 * C], conv_w, conv_b)
        r = pm.sigmoid(pm.block_product(u, _np(mats[0]), rb.reshape(parts, c)))
        i = pm.sigmoid(pm.block_product(u, _np(mats[1]), ib.reshape(parts, c)))
        o, S = pm.linear_recurrence(u, r, i, lam)
        want_rows.append(o * pm.gelu_tanh(x[:, off:off + C]))
    state = torch.full((4, 3 + C + taps * C + 2), 1e3, device=DEV)
    err, pad = _err(), 3
    for ctx, ents in _steps_of(lens, plan, pad):
        x = _rows(proj, ents, pad, 9.0)
        n = x.shape[0]
        aux, out = torch.full((n, 2 * C), 5.0, device=DEV), torch.full((n, C), 5.0, dtype=dtype, device=DEV)
        K.gate_scan_prep(x, cols, ctx, state, scan, aux, out, err, dtype)
        if not ctx.all_single:
            assert (out == 5.0).all()
            K.channel_scan(aux, x, cols, ctx, state, scan, out, err)
        got, at = _np(out), 0
        for r, b, t, _ in ents:
            want = want_rows[r][b:b + t]
            tol = 2e-5 if dtype == torch.float32 else 1e-2
            assert np.abs(got[at:at + t] - want).max() < tol * max(1.0, np.abs(want).max()), (r, b, t)
            at += t
        assert (out[at:] == 5.0).all() and (aux[at:] == 5.0).all()
    assert plan is not PLAN or (state[3] == 1e3).all()
    assert (state[:, 0] == 1e3).all() and (state[:, 1 + C:3 + C] == 1e3).all() and (state[:, -2:] == 1e3).all()
    assert int(err.item()) == 0


@pytest.mark.parametrize("n", [1, 12, 17, 40])
def test_gated_linear_recurrence_batches_of_single_tokens(K, n):
    """Every tile shape of the single-token kernel, partial sums, entries without rows among them."""
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(n)
    C, parts, taps, c = 96, 2, 4, 48
    conv_w, conv_b, rb, ib, lam = rng.standard_normal((C, taps)), rng.standard_normal(C), rng.standard_normal(C), rng.standard_normal(C), rng.standard_normal(C)
    mats = [_dev(rng.standard_normal((parts, c, c)) * c ** -0.5, torch.bfloat16) for _ in range(2)]
    gates, mma = K.pack_gates(*mats, False)
    scan = K.GateScan(y_off=0, x_off=C, s_off=0, ring_off=C, conv_w=_dev(conv_w.T.copy()), conv_b=_dev(conv_b), gates=gates, mma=mma, rb=_dev(rb),
                      ib=_dev(ib), sp=_dev(pm.softplus(lam)), parts=parts)
    steps = 7
    slots = rng.permutation(n)
    state = torch.full((n + 1, C * (1 + taps)), 1e3, device=DEV)
    p = _dev(rng.standard_normal((steps, 3, n, 2 * C)))
    x = _np(p.sum(1).to(torch.bfloat16))
    err = _err()
    got = []
    for s in range(steps):
        ctx = SimpleNamespace(cu_q=_i32(list(range(n + 1)) + [n, n]), kv_len=_i32([s + 1] * n + [0, 0]), slots=_i32(list(slots) + [n, n]),
                              tok_entry=_i32(list(range(n)) + [-1, -1]), all_single=True)
        out = torch.full((n + 2, C), 5.0, dtype=torch.bfloat16, device=DEV)
        rows = torch.cat([p[s], torch.full((3, 2, 2 * C), 9.0, device=DEV)], dim=1).contiguous()
        K.gate_scan_prep(Partials(rows), 2 * C, ctx, state, scan, torch.empty(n + 2, 2 * C, device=DEV), out, err, torch.bfloat16)
        assert (out[n:] == 5.0).all()
        got.append(_np(out[:n]))
    for e in range(n):
        u, _ = pm.short_convolution(x[:, e, C:], conv_w, conv_b)
        o, _ = pm.linear_recurrence(u, pm.sigmoid(pm.block_product(u, _np(mats[0]), rb.reshape(parts, c))),
                                    pm.sigmoid(pm.block_product(u, _np(mats[1]), ib.reshape(parts, c))), lam)
        want = o * pm.gelu_tanh(x[:, e, :C])
        assert np.abs(np.stack(got)[:, e] - want).max() < 1e-2 * max(1.0, np.abs(want).max()), e
    assert (state[n] == 1e3).all() and int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [0, 1, 5, 64, 100])
@pytest.mark.parametrize("d, nq, nkv, ps, splits", [(128, 6, 2, 64, 1), (128, 4, 4, 16, 5), (128, 5, 1, 32, 12), (96, 6, 3, 16, 1), (64, 8, 2, 8, 3),
                                                    (16, 3, 3, 32, 40)])
def test_attention_with_gate_window_and_sinks(K, dtype, window, d, nq, nkv, ps, splits):
    """A prompt portion deep in a request, single tokens and a short prompt, with planted keys: the oldest that a
    window still shows, the one just outside it (which must change nothing), the newest, and without a window the
    first of all.  Pages that a window has passed are gone (-1), and what stands in their storage is large.  Sinks
    from negligible to larger than any score; a gate from a product whole and as partial sums."""
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(d + nq + window)
    scale = 0.2
    lens, q_lens = [700, 3 * ps + 1, 2 * ps, 45, 300], [37, 1, 1, 45, 1]
    sinks = np.linspace(-3.0, 6.0, nq)
    sinks[-1] = 60.0
    ks, vs, tabs = [], [], -np.ones((len(lens), max(-(-n // ps) for n in lens)), dtype=np.int32)
    n_pages = sum(-(-n // ps) for n in lens) + 2
    order = rng.permutation(n_pages)
    k_pool, v_pool = ((torch.randn(n_pages, nkv, ps, d, device=DEV) * 30).to(dtype) for _ in range(2))
    nxt = 0
    for e, n in enumerate(lens):
        k, v = (_dev(rng.standard_normal((n, nkv, d)) * 0.5, dtype) for _ in range(2))
        first = max(0, n - q_lens[e] + 1 - window) // ps if window else 0
        for b in range(-(-n // ps)):
            page = int(order[nxt]); nxt += 1
            if b >= first:
                tabs[e, b] = page
                rows = slice(b * ps, min(n, (b + 1) * ps))
                k_pool[page, :, :rows.stop - rows.start] = k[rows].transpose(0, 1)
                v_pool[page, :, :rows.stop - rows.start] = v[rows].transpose(0, 1)
        ks.append(_np(k)); vs.append(_np(v))
    qs, pos, ent, cu = [], [], [], [0]
    for e, (n, ql) in enumerate(zip(lens, q_lens)):
        q = rng.standard_normal((ql, nq, d)) * 0.5
        for t in {0, ql // 2, ql - 1}:
            p = n - ql + t
            lo = max(0, p - window + 1) if window else 0
            for h, key in ((0, lo), (1, lo - 1), (2, p), (nq - 1, lo)):
                if key >= 0:
                    kk = ks[e][key, h // (nq // nkv)]
                    q[t, h] = kk * 40.0 / max(1e-6, (kk ** 2).sum() * scale)
        qs.append(q)
        pos += list(range(n - ql, n)); ent += [e] * ql; cu.append(cu[-1] + ql)
    N = len(pos)
    q_all = _dev(np.concatenate(qs).reshape(N, -1), dtype)
    gate_off, gate_cols = 6, 6 + nq * d + 2
    gparts = _dev(rng.standard_normal((3, N, gate_cols)))
    gate = gparts.sum(0).to(dtype)
    want = np.concatenate([pm.sink_window_attention(_np(q_all)[cu[e]:cu[e + 1]].reshape(-1, nq, d), ks[e], vs[e], scale, window, sinks,
                                                    lens[e] - q_lens[e]) for e in range(len(lens))])
    want = want.reshape(N, -1) * pm.sigmoid(_np(gate)[:, gate_off:gate_off + nq * d])
    err, sk, table = _err(), _dev(sinks), _i32(tabs)
    tol = 3e-5 if dtype == torch.float32 else 2.5e-2
    for form in ("whole", "parts"):
        g = gate if form == "whole" else Partials(gparts)
        out = torch.full((N, nq * d), 5.0, dtype=dtype, device=DEV)
        if dtype == torch.float32:
            K.paged_attention_simt(q_all, out, k_pool, v_pool, _i32(pos), _i32(ent), table, ps, nq, nkv, d, window, scale, err, sinks=sk)
            K.gate_mul(out, g, gate_cols, gate_off)
        else:
            part_o, part_ml = torch.empty(len(lens) * nq * splits * d, device=DEV), torch.empty(len(lens) * nq * splits * 2, device=DEV)
            tiles = sum(-(-n // 64) for n in q_lens if n != 1)
            K.paged_prefill_attention(q_all, out, k_pool, v_pool, _i32(cu), _i32(lens), table, ps, tiles, nq, nkv, d, window, scale, err,
                                      skip_single=True, sinks=sk, gate=(g, gate_cols, gate_off))
            single = [cu[e] for e in range(len(lens)) if q_lens[e] == 1]
            assert (out[single] == 5.0).all()
            K.paged_decode_attention(q_all, out, k_pool, v_pool, _i32(cu), _i32(lens), table, ps, nq, nkv, d, window, scale, splits, part_o,
                                     part_ml, err, sinks=sk, gate=(g, gate_cols, gate_off))
            both = torch.full_like(out, 5.0)                # every entry through the kernel for portions
            K.paged_prefill_attention(q_all, both, k_pool, v_pool, _i32(cu), _i32(lens), table, ps, tiles + 3, nq, nkv, d, window, scale, err,
                                      sinks=sk, gate=(g, gate_cols, gate_off))
            assert np.abs(_np(both) - want).max() < tol * max(1.0, np.abs(want).max()), form
            if K.prefill_attention_tc_supports(d, nq, nkv, ps):          # the same on tcgen05, every entry and portions alone
                for skip in (False, True):
                    both.fill_(5.0)
                    K.prefill_attention_tc(q_all, both, k_pool, v_pool, _i32(cu), _i32(lens), table, ps, len(lens) + 1, nq, nkv, d, window,
                                           scale, err, skip_single=skip, sinks=sk, gate=(g, gate_cols, gate_off))
                    rows = [i for i in range(N) if not skip or i not in single]
                    assert np.abs(_np(both)[rows] - want[rows]).max() < tol * max(1.0, np.abs(want).max()), (form, skip)
                    assert not skip or (both[single] == 5.0).all()
        bad = np.abs(_np(out) - want).max(axis=1) >= tol * max(1.0, np.abs(want).max())
        assert not bad.any(), (form, np.nonzero(bad)[0][:5])
    assert int(err.item()) == 0


@pytest.mark.parametrize("window", [0, 200])
def test_long_prompts_two_heads_a_block(K, window):
    """As many tiles as make the tcgen05 kernel take two heads at a time: sinks, gate and window against the kernel of
    64-row tiles."""
    torch.manual_seed(window)
    T, nq, nkv, d, ps = 4096, 16, 4, 128, 64
    q, gate = torch.randn(T, nq * d, device=DEV).bfloat16(), torch.randn(T, nq * d + 8, device=DEV).bfloat16()
    kp, vp = (torch.randn(T // ps, nkv, ps, d, device=DEV).bfloat16() for _ in range(2))
    table, cu, kvl, err = _i32([torch.randperm(T // ps).tolist()]), _i32([0, T]), _i32([T]), _err()
    sinks = torch.linspace(-2, 9, nq, device=DEV)
    a, b = torch.empty_like(q), torch.empty_like(q)
    g = (gate, nq * d + 8, 8)
    K.prefill_attention_tc(q, a, kp, vp, cu, kvl, table, ps, T // 128, nq, nkv, d, window, d ** -0.5, err, sinks=sinks, gate=g)
    K.paged_prefill_attention(q, b, kp, vp, cu, kvl, table, ps, T // 64, nq, nkv, d, window, d ** -0.5, err, sinks=sinks, gate=g)
    assert float((a.float() - b.float()).abs().max()) < 2e-2 * float(b.float().abs().max()) and int(err.item()) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, d, m, rot, window", [(4, 2, 128, 128, (64, 1e4, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}), 20),
                                                     (6, 3, 24, 40, (24, 90.0, None), 9), (4, 1, 50, 31, (6, 100.0, None), 0),
                                                     (2, 2, 64, 64, None, 1), (3, 3, 15, 16, (4, 50.0, None), 33),
                                                     (2, 1, 264, 17, (128, 1e3, None), 10)])
def test_attention_part(dtype, H, G, d, m, rot, window):
    """The mixer part at heads stored wider than their keys and values: a whole sequence, the same in two portions, and
    its last tokens one by one (bfloat16: the kernel that prepares the new token itself)."""
    from test_gpu_parts import build, make_ctx, np64, runtime, whole
    from crane_b200.config import PartSpec
    from crane_b200.config.mufalix import stored_head_size
    from crane_b200.parts import LayerCache
    h, T, ps, eps = 72, 45, 16, 1e-3
    rt = runtime(dtype)
    rng = np.random.default_rng(d + m)
    D = stored_head_size(d, m)
    position = None if rot is None else PartSpec("position", "wavelength_rope", {"dims": rot[0], "base": rot[1], "scaling": rot[2],
                                                                                 "max_positions": 4096})
    names = {"q": "q", "k": "k", "v": "v", "o": "o", "q_bias": "q.b", "k_bias": "k.b", "v_bias": "v.b", "o_bias": "o.b",
             "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g", "sink": "sink"}
    spec = PartSpec("mixer", "gqa_attention", {
        "hidden_size": h, "num_heads": H, "num_kv_heads": G, "head_dim": D, "key_dim": d, "value_dim": m, "bias": True, "qk_norm": True,
        "qk_norm_eps": eps, "qk_norm_order": "before_rope", "rotary_dim": rot[0] if rot else None, "position": position, "window": window,
        "scale": 1.3 * d ** -0.5, "sink": True, "gate": True, "names": names}, "a.")
    from crane_b200.parts import part_class
    shapes = {n: s.shape for n, s in part_class(spec).manifest(spec).items()}
    t = {n: torch.from_numpy(rng.standard_normal(s) * (0.12 if len(s) == 2 else 0.5) + (1.0 if "norm" in n else 0.0)).float()
         for n, s in shapes.items()}
    t["a.q"] *= 0.3                                            # small rows, so that eps counts
    t["a.q.b"] *= 0.02
    t["a.sink"] = torch.linspace(-2.0, 4.0, H)
    if dtype == torch.bfloat16:
        t = {k: (x.bfloat16().float() if x.dim() == 2 else x) for k, x in t.items()}
    w = {k: np64(x) for k, x in t.items()}
    part = build(spec, dict(t), rt)
    x = _dev(rng.standard_normal((T, h)), dtype)
    cfg = {"heads": H, "kv_heads": G, "dim": d, "vdim": m, "scale": 1.3 * d ** -0.5}
    if window:
        cfg["mask"] = {"size": window}
    if rot:
        cfg["rot"] = {"dims": rot[0], "base": rot[1], "scaling": rot[2]}
    want, _ = pm.attention_side(_np(x), w, "a.", cfg, eps)
    need = part.cache_need()
    assert need.head_dim == D

    def cache():
        return LayerCache(need, 0, torch.full((6, G, ps, D), 30.0, device=DEV, dtype=dtype),
                          torch.full((6, G, ps, D), 30.0, device=DEV, dtype=dtype), ps)
    tol = 2e-5 if dtype == torch.float32 else 2.5e-2
    rows = [[4, 1, 5, 2]]
    for cuts in ([T], [23, 17, 5], [23, 17] + [1] * 5, [1] * T):
        c, outs, pos = cache(), [], 0
        for n in cuts:
            outs.append(whole(part.forward(x[pos:pos + n], make_ctx(rt, [(pos, n)], ps, 6, 4, rows), c, rt), dtype).clone())
            pos += n
        got = _np(torch.cat(outs))
        assert np.abs(got - want).max() < tol * np.abs(want).max(), (cuts[:3], np.abs(got - want).max(axis=1).argmax())
    rt.check_errors()


@pytest.mark.parametrize("d, rot, norm", [(128, 64, True), (96, 32, True), (64, 64, True), (200, 48, True), (256, 256, True), (128, 0, True),
                                          (24, 16, True), (128, 32, False), (8, 0, True)])
def test_norm_before_a_partial_rotation(K, d, rot, norm):
    """Whole bfloat16 rows of many tokens (16-byte loads, the partner by shuffle) against NumPy, with rows of no entry,
    a missing page and pages in no order."""
    rng = np.random.default_rng(d + rot)
    n, H, G, ps, eps, off = 70, 3, 1, 8, 1e-3, 0.5
    cols = (H + 2 * G) * d + 16
    x = _dev(rng.standard_normal((n, cols)) * 0.05, torch.bfloat16)
    pos = rng.permutation(80)[:n]
    table = np.array([rng.permutation(12)[:10]], dtype=np.int32)
    table[0, 9] = -1
    ent = np.zeros(n, dtype=np.int32)
    ent[5] = -1
    f = pm.rotary_frequencies(rot, 300.0)
    ang = np.arange(80)[:, None] * f[None]
    cos, sin = (_dev(np.cos(ang)), _dev(np.sin(ang))) if rot else (None, None)
    qw, kw = (rng.standard_normal(d), rng.standard_normal(d)) if norm else (None, None)
    q = torch.full((n, H * d), 5.0, dtype=torch.bfloat16, device=DEV)
    kp, vp = (torch.full((12, G, ps, d), 5.0, dtype=torch.bfloat16, device=DEV) for _ in range(2))
    err = _err()
    K.rope_norm_cache(x, cols, torch.bfloat16, _i32(pos), _i32(ent), _i32(table), cos, sin, None if qw is None else _dev(qw),
                      None if kw is None else _dev(kw), eps, q, kp, vp, ps, H, G, d, True, rot > 0, err, rope=(rot or d, False, True, off))
    xn = _np(x)

    def heads(a, w):
        y = a.reshape(n, -1, d)
        return pm.rotate_half(pm.over_rms(y, eps) * (off + w) if w is not None else y, pos, f)
    want_q, want_k = heads(xn[:, :H * d], qw), heads(xn[:, H * d:(H + G) * d], kw)
    assert np.abs(_np(q).reshape(n, H, d) - want_q).max() < 1e-2 * max(1.0, np.abs(want_q).max())
    for t in range(n):
        page = table[0, pos[t] // ps]
        if ent[t] < 0 or page < 0:
            continue
        k, v = _np(kp)[page, :, pos[t] % ps], _np(vp)[page, :, pos[t] % ps]
        assert np.abs(k - want_k[t]).max() < 1e-2 * max(1.0, np.abs(want_k).max()), t
        assert np.abs(v - xn[t, (H + G) * d:(H + 2 * G) * d].reshape(G, d)).max() == 0
    used = {int(p) for p in table[0] if p >= 0}
    assert all((kp[p] == 5.0).all() for p in range(12) if p not in used)
    assert int(err.item()) == (2 if (pos // ps == 9).any() else 0)


@pytest.mark.parametrize("experts, top, scale", [(3, 3, 1.0), (12, 1, 2.5), (6, 2, 0.7), (64, 6, 1.0), (40, 8, 1.6)])
def test_route_by_corrected_scores(K, experts, top, scale):
    """The correction chooses and the score weighs; the weights are over the chosen scores' sum."""
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(experts)
    n = 29
    z = (rng.standard_normal((n, experts)) * 3).astype(np.float32)
    z[1] = 0.25
    z[2] = -30.0
    corr = rng.standard_normal(experts).astype(np.float32) * 0.5
    corr[0] = 0.8
    for c in (corr, None):
        route, again = (torch.full((n, experts), 5.0, device=DEV) for _ in range(2))
        cd = None if c is None else _dev(c)
        K.route_grouped(_dev(z), cd, route, experts, top, 1, 1, False, sigmoid=True, renorm=True, scale=scale)
        K.route_grouped(Partials(torch.stack([_dev(z), torch.zeros(n, experts, device=DEV)])), cd, again, experts, top, 1, 1, False,
                        sigmoid=True, renorm=True, scale=scale)
        assert torch.equal(route, again)
        got = _np(route)
        for t in range(n):
            idx, w = pm.choose_experts(z[t].astype(np.float64), np.zeros(experts) if c is None else c.astype(np.float64), top, scale)
            want = np.zeros(experts)
            want[idx] = w
            assert np.abs(got[t] - want).max() < 2e-6 * scale and set(np.nonzero(got[t])[0]) == set(idx), t


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, hidden", [(1, 48), (9, 7), (70, 256), (300, 66)])
def test_pass_projection(dtype, n, hidden):
    """The stream, what is pending and the kept embedding output, one product, its result the stream in 32-bit."""
    from test_gpu_parts import build, runtime
    from crane_b200.config import PartSpec
    from crane_b200.kernels import Partials
    rng = np.random.default_rng(n)
    rt = runtime(dtype)
    w = (rng.standard_normal((hidden, 2 * hidden)) * 0.1)
    w = _np(_dev(w, dtype))
    part = build(PartSpec("entry", "pass_projection", {"size": hidden, "tensor": "w"}), {"w": torch.from_numpy(w).float()}, rt)
    x0 = _dev(rng.standard_normal((n, hidden)))
    rt.ws.get("embedding_output", n, hidden, torch.float32).copy_(x0)
    delta = _dev(rng.standard_normal((2, n, hidden)))
    for pending in (None, delta.sum(0).to(dtype), Partials(delta)):
        x = _dev(rng.standard_normal((n, hidden)))
        full = _np(x) + (0.0 if pending is None else _np(delta.sum(0).to(dtype)))
        want = np.concatenate([full, _np(x0)], axis=1) @ w.T
        assert part.forward(x, pending, None, rt) is None
        assert np.abs(_np(x) - want).max() < (2e-5 if dtype == torch.float32 else 1e-2) * np.abs(want).max()
    rt.check_errors()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_embedding_scale_and_copies(K, dtype):
    rng = np.random.default_rng(1)
    table = _dev(rng.standard_normal((11, 37)), dtype)
    toks = _i32([3, 0, 10, -2, 4])
    x, keep, raw = torch.empty(5, 37, device=DEV), torch.empty(5, 37, device=DEV), torch.empty(5, 37, dtype=dtype, device=DEV)
    err = _err()
    K.embed_gather(toks, table, x, err, _i32([7]), raw, 2.3, keep)
    want = (table[[3, 0, 10, 7, 4]].float() * 2.3)
    assert torch.equal(x, want) and torch.equal(keep, want) and torch.equal(raw, want.to(dtype)) and int(err.item()) == 0


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
    cfg, w = pm.load_folder(folder)
    m = _load(folder, "fp32", page_size=tm.TINY[name]["page_size"], num_pages=24, max_concurrent=3,
              max_batched_tokens=64, max_seq_len=192)
    rng = np.random.default_rng(3)
    for n in (1, 5, 17):
        prompt = rng.integers(0, cfg["vocab"], n).tolist()
        assert m.generate(prompt, _greedy(8)) == pm.greedy_generate(cfg, w, prompt, 8)
    m.runner.table.check()
    assert m.runner.table.live() == 0


@pytest.mark.parametrize("name", ["FA", "FL"])
def test_greedy_batch_bfloat16_through_the_scheduler(name, model_folders):
    """Six prompts, three slots, portions of at most 16 tokens: requests wait, slots and pages are used
    again, and decode steps replay the batch-size buckets' graphs with the recurrent states in them."""
    folder = model_folders(name, "bfloat16")
    cfg, w = pm.load_folder(folder)
    m = _load(folder, "bf16", page_size=16, num_pages=40, max_concurrent=3, max_batched_tokens=48, chunk_size=16,
              max_seq_len=256)
    rng = np.random.default_rng(4)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (12, 3, 40, 1, 25, 7)]
    outs = m.generate_batch(prompts, _greedy(20))
    ok = 0
    for prompt, toks in zip(prompts, outs):
        assert len(toks) == len(prompt) + 20 and toks[:len(prompt)] == prompt
        logits = pm.logits_all(cfg, w, toks[:-1])
        for i in range(len(prompt), len(toks)):
            row = logits[i - 1]
            # (a token that another rounding would not have chosen does not end the comparison: every later one is
            # checked against the plain logits of the sequence as it was generated)
            ok += bool(row[toks[i]] >= row.max() - 3e-2 * np.abs(row).max())
    assert ok >= 0.95 * 20 * len(prompts), ok
    m.runner.table.check()
    assert m.runner.table.live() == 0
    assert m.runner.graph_replays > 0 and m.runner._pad_with_copies       # (the batch-size buckets)


def test_decode_batches_of_changing_size_without_the_decode_kernel(model_folders):
    """Heads that the decode kernel does not take: single tokens go through the kernel for portions, also in the
    batch-size buckets' graphs, which are recorded with fewer requests than later steps have."""
    from crane_b200.config import EngineConfig
    from crane_b200.engine import ModelRunner, StepEntry
    folder = model_folders("FG", "bfloat16")
    cfg, w = pm.load_folder(folder)
    runner = ModelRunner(folder, EngineConfig(dtype="bfloat16", page_size=16, num_pages=24, max_concurrent=4, max_batched_tokens=64,
                                              max_seq_len=128))
    rng = np.random.default_rng(2)
    toks = [rng.integers(0, cfg["vocab"], 40).tolist() for _ in range(4)]
    want = [pm.logits_all(cfg, w, t) for t in toks]
    done = [9, 14, 3, 6]
    for r in range(4):
        runner.step([StepEntry(r, toks[r][:done[r]], [])])
    for live in [(0, 1, 2)] * 3 + [(0, 1, 2, 3)] * 4 + [(1, 2, 3)] * 2 + [(2,)] * 2 + [(0, 1, 2, 3)] * 3:
        got = runner.step([StepEntry(r, [toks[r][done[r]]], [0]) for r in live]).cpu().numpy()
        for i, r in enumerate(live):
            row = want[r][done[r]]
            assert np.sqrt(((got[i] - row) ** 2).mean()) < 6e-2 * np.sqrt((row ** 2).mean()), (live, r)
            done[r] += 1
    runner.rt.check_errors()
    assert runner.graph_replays > 0 and runner._pad_with_copies


def test_command_line(model_folders):
    """bin/crane picks the model class from config.json."""
    import os
    import subprocess
    import sys
    folder = model_folders("FA", "float32")
    cfg, w = pm.load_folder(folder)
    crane = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "crane")
    cmd = [sys.executable, crane, "-m", folder, "--dtype", "fp32", "--prompt-ids", "5,6,7", "--max-new-tokens", "6",
           "--eos-token-id", "-1", "--page-size", "16", "--num-pages", "8", "-c", "2", "--max-batched-tokens", "32",
           "--max-seq-len", "64"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-3000:]
    assert p.stdout.strip().splitlines()[-1] == ",".join(map(str, pm.greedy_generate(cfg, w, [5, 6, 7], 6)[3:]))
