"""Mufalix on the host: configuration errors, the manifest, the schedule of repeated layers, and the plain
implementation's own mechanisms against hand arithmetic and against their continuation from a carried state."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_mufalix as pm
import tiny_mufalix as tm
from crane_b200.config import ConfigError, resolve
from crane_b200.config.mufalix import stored_head_size
from crane_b200.parts import model_manifest


def _spec(config):
    arch = resolve(config)
    return arch, arch.build_spec(arch.config_from_dict(config))


def test_registered_by_its_name():
    arch, spec = _spec(tm.FA)
    assert arch.name == "Mufalix" and spec.architecture == "Mufalix"
    assert [l.block for l in spec.layers] == ["prenorm_residual"] * 4
    assert [l.parts["mixer"].name for l in spec.layers] == ["parallel_pair", "exponential_gates", "parallel_pair", "exponential_gates"]
    assert ["ffn" in l.parts for l in spec.layers] == [True, True, False, True] and "norm2" not in spec.layers[2].parts
    left = spec.layers[0].parts["mixer"].params["left"].params
    assert (left["head_dim"], left["key_dim"], left["value_dim"], left["window"], left["rotary_dim"]) == (32, 14, 24, 11, 8)
    assert left["sink"] and left["gate"] and left["bias"] and left["qk_norm_order"] == "before_rope"
    moe = spec.layers[0].parts["ffn"].params
    assert (moe["scores"], moe["route_scale"], moe["top"], moe["act"]) == ("sigmoid", 0.8, 2, "relu2")
    assert spec.embed.params["scale"] == 1.7 and spec.embed.params["keep_copy"]
    b = _spec(tm.FB)[1]
    assert b.embed.params["scale"] == 1.0
    assert b.layers[0].parts["mixer"].params["left"].params["position"] is None
    c = _spec(tm.FC)[1]
    assert c.entry is None and not c.embed.params["keep_copy"]


@pytest.mark.parametrize("config, runs", [
    (tm.FA, [(0, None), (1, {}), (2, None), (1, {}), (2, None), (3, None)]),
    (tm.FB, [(0, {}), (0, {}), (0, {}), (1, None), (2, None)]),
    (tm.FC, [(0, None), (1, None), (2, None)]),
    (tm.FD, [(0, {}), (1, None), (2, None)] * 2)])
def test_schedule(config, runs):
    spec = _spec(config)[1]
    assert [(s.layer, s.enter) for s in spec.schedule] == runs and all(s.cache_of is None for s in spec.schedule)
    assert [i for i, _ in pm.layer_runs(config)] == [i for i, _ in runs]


def test_manifest_names_and_shapes():
    m = model_manifest(_spec(tm.FA)[1])
    assert m["embed"].shape == (157, 72) and m["head"].shape == (157, 72) and m["final.norm"].shape == (72,)
    assert m["loop.in"].shape == (72, 144) and "l2.norm2" not in m
    p = "l0.mix.left."
    assert m[p + "q"].shape == (56, 72) and m[p + "k"].shape == (28, 72) and m[p + "v"].shape == (48, 72)
    assert m[p + "q.b"].shape == (56,) and m[p + "v.b"].shape == (48,) and m[p + "g"].shape == (96, 72)
    assert m[p + "q.norm"].shape == (14,) and m[p + "sink"].shape == (4,)
    assert m[p + "o"].shape == (72, 96) and m[p + "o.b"].shape == (72,) and p + "g.b" not in m
    p = "l0.mix.right."
    assert m[p + "y"].shape == (40, 72) and m[p + "conv"].shape == (40, 3) and m[p + "ra"].shape == (4, 10, 10)
    assert m[p + "ri.b"].shape == (4, 10) and m[p + "lam"].shape == (40,) and m[p + "o"].shape == (72, 40)
    assert m["l0.mix.left.out"].shape == (72,) and m["l0.mix.right.out"].shape == (72,)
    assert m["l1.mix.q"].shape == (48, 72) and m["l1.mix.v"].shape == (24, 72) and m["l1.mix.i"].shape == (3, 72)
    assert m["l1.mix.f.b"].shape == (3,) and m["l1.mix.norm"].shape == (24,)
    assert m["l1.mlp.router"].shape == (4, 72) and m["l1.mlp.correction"].shape == (4,) and m["l1.mlp.e3.down"].shape == (72, 40)
    assert model_manifest(_spec(tm.FB)[1])["l1.mix.o"].shape == (68, 24)
    assert "loop.in" not in model_manifest(_spec(tm.FC)[1])


def test_stored_head_sizes():
    assert [stored_head_size(*s) for s in ((16, 16), (14, 24), (90, 64), (64, 97), (257, 3), (300, 301))] == [16, 32, 96, 112, 258, 302]


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="attention"), "no mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "router.top"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("dim"), "'dim'"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=16), "dims must be even and at most dim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=5), "dims must be even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("low"), "'low'"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=-1), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(blocks=3), "multiple of blocks"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["norm"].update(eps=0.0), "norm.eps"),
    (lambda c: c.pop("vocab"), "'vocab'")])
def test_configuration_errors(edit, text):
    cfg = copy.deepcopy(tm.FA)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        _spec(cfg)


# ------------------------------------------------------------------ the plain mechanisms
def test_frequencies_by_wavelength():
    """Wavelengths on both sides of both limits; the mix at one in between, by hand; the part's tables."""
    from crane_b200.config import PartSpec
    from crane_b200.parts import build_part
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 64}
    plain = pm.rotary_frequencies(8, 100.0)
    f = pm.rotary_frequencies(8, 100.0, sc)
    lengths = 2 * math.pi / plain                               # 6.3, 19.9, 62.8, 198.7
    assert lengths[0] < 16 < lengths[1] < lengths[2] < 64 < lengths[3]
    assert f[0] == plain[0] and f[3] == plain[3] / 8
    for i in (1, 2):
        s = (64 / lengths[i] - 1.0) / 3.0
        assert 0 < s < 1 and abs(f[i] - (plain[i] * (s + (1 - s) / 8))) < 1e-15
    for dims, base, scaling in ((8, 100.0, sc), (24, 5e4, None), (64, 1e4, {"factor": 4.0, "low": 0.5, "high": 0.75, "original": 900}),
                                (12, 10.0, {"factor": 2.0, "low": 2.0, "high": 2.0, "original": 32})):
        part = build_part(PartSpec("position", "wavelength_rope", {"dims": dims, "base": base, "scaling": scaling,
                                                                   "max_positions": 1000}))
        if scaling is None or scaling["low"] != scaling["high"]:
            assert np.allclose(part.frequencies(), pm.rotary_frequencies(dims, base, scaling), rtol=1e-14)

        class Rt:
            device = torch.device("cpu")
        cos, sin = part.tables(Rt(), 300)
        a = np.arange(300)[:, None] * part.frequencies()[None]
        assert cos.shape == (300, dims // 2) and np.abs(cos.numpy() - np.cos(a)).max() < 1e-7
        assert np.abs(sin.numpy() - np.sin(a)).max() < 1e-7


def test_rotation_pairs_halves_of_the_leading_part():
    x = np.zeros((1, 1, 6))
    x[0, 0] = [1.0, 2.0, 3.0, 4.0, 5.0, 6.0]
    f = np.array([0.5, 0.25])
    y = pm.rotate_half(x, [3], f)[0, 0]
    a, b = 1.5, 0.75
    assert np.allclose(y, [math.cos(a) - 3 * math.sin(a), 2 * math.cos(b) - 4 * math.sin(b), 3 * math.cos(a) + math.sin(a),
                           4 * math.cos(b) + 2 * math.sin(b), 5.0, 6.0])


def test_window_and_sink_by_hand():
    q, k = np.zeros((4, 2, 1)), np.zeros((4, 1, 1))
    v = np.arange(1.0, 5.0).reshape(4, 1, 1)
    o = pm.sink_window_attention(q, k, v, 1.0, 2, np.array([0.0, math.log(3.0)]))
    assert np.allclose(o[0, :, 0], [1 / 2, 1 / 4])                       # itself and the sink
    assert np.allclose(o[3, :, 0], [(3 + 4) / 3, (3 + 4) / 5])           # two tokens and the sink
    o = pm.sink_window_attention(q[3:], k, v, 1.0, 0, np.array([0.0, 0.0]), first_query=3)
    assert np.allclose(o[0, :, 0], 10 / 5)
    q[:, 0], k[0] = 10.0, 10.0                                           # a far key stands out for head 0
    far = pm.sink_window_attention(q, k, v, 1.0, 4, np.zeros(2))[3, 0, 0]
    gone = pm.sink_window_attention(q, k, v, 1.0, 3, np.zeros(2))[3, 0, 0]
    assert abs(far - 1.0) < 1e-9 and abs(gone - (2 + 3 + 4) / 4) < 1e-9


def test_convolution_and_recurrence_by_hand():
    x = np.array([[1.0], [2.0], [4.0]])
    y, kept = pm.short_convolution(x, np.array([[0.5, 10.0, 100.0]]), np.array([7.0]))
    assert np.allclose(y[:, 0], [107.0, 217.0, 427.5]) and np.allclose(kept[:, 0], [2.0, 4.0])
    y2, _ = pm.short_convolution(x[2:], np.array([[0.5, 10.0, 100.0]]), np.array([7.0]), np.array([[1.0], [2.0]]))
    assert np.allclose(y2[0], y[2])
    lam = math.log(math.e - 1.0)                                         # softplus(lam) = 1
    r, i = np.array([[0.125], [0.25]]), np.array([[1.0], [0.5]])
    o, S = pm.linear_recurrence(np.array([[3.0], [5.0]]), r, i, np.array([lam]))
    s1 = math.sqrt(1 - math.exp(-2.0)) * 3.0                             # the first token has no special case
    s2 = math.exp(-2.0) * s1 + math.sqrt(1 - math.exp(-4.0)) * 2.5
    assert np.allclose(o[:, 0], [s1, s2]) and np.allclose(S, [s2])
    u = np.arange(1.0, 5.0)[None]
    mats = np.array([[[1.0, 2.0], [3.0, 4.0]], [[0.0, 1.0], [1.0, 0.0]]])
    assert np.allclose(pm.block_product(u, mats, np.array([[0.0, 1.0], [2.0, 3.0]]))[0], [5.0, 12.0, 6.0, 6.0])


def test_stabilised_scan_by_hand_and_without_its_maximum():
    """One head and one number: the maximum starts at 0, so a small first input gate leaves the floor exp(0)."""
    q = k = v = np.ones((1, 1, 1))
    o, (S, N, M) = pm.stabilised_scan(q, k, 5 * v, np.array([[-2.0]]), np.array([[-3.0]]))
    assert M[0] == -2.0 and np.allclose(S, 5.0) and np.allclose(N, 1.0)
    assert np.allclose(o, 5.0 / (math.exp(2.0) + 1e-6))
    o, (_, _, M) = pm.stabilised_scan(q, k, 5 * v, np.array([[-2.0]]), np.array([[-1.0]]))
    assert M[0] == -1.0 and np.allclose(o, 5.0 * math.exp(-1.0) / (math.exp(1.0) + 1e-6))
    # without the floor and the constant it is the plain recurrence with gates exp(i) and exp(f)
    rng = np.random.default_rng(0)
    n, H, d, m = 20, 2, 5, 3
    q, k, v = rng.standard_normal((n, H, d)), np.abs(rng.standard_normal((n, H, d))), rng.standard_normal((n, H, m))
    q = np.abs(q) + 1.0
    li, lf = rng.standard_normal((n, H)) + 3.0, -rng.random((n, H))
    o, _ = pm.stabilised_scan(q, k, v, li, lf)
    S, N = np.zeros((H, d, m)), np.zeros((H, d))
    for t in range(n):
        S = np.exp(lf[t])[:, None, None] * S + np.exp(li[t])[:, None, None] * k[t][:, :, None] * v[t][:, None]
        N = np.exp(lf[t])[:, None] * N + np.exp(li[t])[:, None] * k[t]
        want = (S * q[t][..., None]).sum(1) / np.abs((N * q[t]).sum(-1))[:, None]
        assert np.abs(o[t] - want).max() < 1e-4 * np.abs(want).max()


def test_choice_and_weights_of_experts():
    z = np.array([0.0, 2.0, -1.0, 0.5])
    s = 1 / (1 + np.exp(-z))
    idx, w = pm.choose_experts(z, np.array([0.0, -0.6, 0.7, 0.0]), 2, 1.5)
    assert idx == [2, 3] and np.allclose(w, s[[2, 3]] / (s[2] + s[3]) * 1.5)       # the correction chooses, the score weighs
    assert pm.choose_experts(np.zeros(4), np.zeros(4), 3, 1.0)[0] == [0, 1, 2]     # ties to the lower index


@pytest.mark.parametrize("name", ["FA", "FB", "FC", "FD"])
def test_plain_model_cut_anywhere(name, model_folders):
    cfg, w = pm.load_folder(model_folders(name, "float32"))
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 23).tolist()
    want, streams, _ = pm.forward(cfg, w, toks)
    assert streams.shape[0] == len(pm.layer_runs(cfg))
    state, pos = None, 0
    for n in (4, 1, 2, 9, 1, 6):
        got, _, state = pm.forward(cfg, w, toks[pos:pos + n], state, start=pos)
        assert np.abs(got - want[pos:pos + n]).max() < 1e-9
        pos += n


def test_a_pass_reads_the_embedding_output_again():
    """One pass more changes the result, and a pass's product sees [x; x0] with x first."""
    cfg = copy.deepcopy(tm.FB)
    rng = np.random.default_rng(2)
    from crane_b200.weights.random_init import random_tensors
    w = {k: v.double().numpy() for k, v in random_tensors(model_manifest(_spec(cfg)[1]), 1, torch.float32, std=0.1).items()}
    toks = rng.integers(0, cfg["vocab"], 5).tolist()
    three = pm.logits_all(cfg, w, toks)
    cfg["loop"]["times"] = 2
    assert np.abs(pm.logits_all(cfg, w, toks) - three).max() > 1e-3
    W = cfg["width"]
    w["loop.in"] = np.concatenate([np.zeros((W, W)), np.eye(W)], axis=1)        # every pass begins at x0
    two = pm.logits_all(cfg, w, toks)
    cfg["loop"]["times"] = 1
    assert np.abs(pm.logits_all(cfg, w, toks) - two).max() < 1e-12
