"""Pogarax on the host: configuration errors, the manifest, what a shared cache keeps, and the plain
implementation's own mechanisms against hand arithmetic and against their continuation from a
carried state."""
import copy
import math

import numpy as np
import pytest

import plain_pogarax as pp
import tiny_pogarax as tp
from crane_b200.config import ConfigError, resolve
from crane_b200.parts import model_manifest


def _spec(config):
    arch = resolve(config)
    return arch, arch.build_spec(arch.config_from_dict(config))


def test_registered_by_its_name():
    arch, spec = _spec(tp.PA)
    assert arch.name == "Pogarax" and spec.architecture == "Pogarax"
    assert [l.block for l in spec.layers] == ["output_norm_residual"] * 5
    assert [l.parts["mixer"].name for l in spec.layers] == ["wkv_time_mix", "latent_attention", "gated_delta",
                                                            "latent_attention", "gated_delta"]
    assert [l.parts["ffn"].name if "ffn" in l.parts else None for l in spec.layers] == [
        "swiglu", "grouped_experts", "grouped_experts", None, "swiglu"]
    assert "norm2" not in spec.layers[3].parts
    assert [s.cache_of for s in spec.schedule] == [None, None, None, 1, None]
    assert all(l.parts["norm1"].params["gain"] == 0.45 for l in spec.layers) and "gain" not in spec.final_norm.params
    moe = spec.layers[2].parts["ffn"].params
    assert (moe["scores"], moe["weight_on"], moe["top"], moe["experts"]) == ("sigmoid", "input", 1, 4)
    assert _spec(tp.PB)[1].layers[0].parts["norm1"].params["gain"] == 1.0


def test_manifest_names_and_shapes():
    m = model_manifest(_spec(tp.PA)[1])
    assert m["embed"].shape == (199, 104) and m["head"].shape == (199, 104) and m["final.norm"].shape == (104,)
    assert m["l0.norm1"].shape == (104,) and m["l0.norm2"].shape == (104,) and "l3.norm2" not in m
    assert m["l0.mix.mu.w"].shape == (104,) and m["l0.mix.r"].shape == (48, 104) and m["l0.mix.w1"].shape == (5, 104)
    assert m["l0.mix.w2"].shape == (48, 5) and m["l0.mix.u"].shape == (3, 16) and m["l0.mix.norm"].shape == (48,)
    assert m["l0.mix.w0"].shape == (48,) and m["l0.mix.o"].shape == (104, 48) and m["l0.mlp.gate"].shape == (72, 104)
    assert m["l1.mix.dq"].shape == (56, 104) and m["l1.mix.dq.norm"].shape == (56,) and m["l1.mix.uq"].shape == (160, 56)
    assert m["l1.mix.dkv"].shape == (48, 104) and m["l1.mix.dkv.norm"].shape == (40,) and m["l1.mix.sink"].shape == (5,)
    assert m["l1.mix.uk"].shape == (120, 40) and m["l1.mix.uv"].shape == (100, 40) and m["l1.mix.o"].shape == (104, 100)
    assert m["l1.mlp.router"].shape == (5, 104) and m["l1.mlp.e4.down"].shape == (104, 24)
    assert m["l2.mix.q"].shape == (32, 104) and m["l2.mix.v"].shape == (96, 104) and m["l2.mix.q.conv"].shape == (32, 3)
    assert m["l2.mix.a1"].shape == (6, 104) and m["l2.mix.a2"].shape == (64, 6) and m["l2.mix.dt_bias"].shape == (64,)
    assert m["l2.mix.A_log"].shape == (4,) and m["l2.mix.g1"].shape == (9, 104) and m["l2.mix.g2"].shape == (96, 9)
    assert m["l2.mix.b"].shape == (4, 104) and m["l2.mix.norm"].shape == (24,) and "l2.mix.a" not in m and "l2.mix.g" not in m
    assert "l3.mix.dkv" not in m and "l3.mix.dkv.norm" not in m and m["l3.mix.uk"].shape == (48, 40)
    assert m["l4.mix.q"].shape == (72, 104)                       # no kv_heads entry: as many as heads


def test_inner_sizes_of_a_stored_model_are_read_from_its_tensors():
    cfg = copy.deepcopy(tp.PA)
    del cfg["layers"][0]["mixer"]["decay_rank"], cfg["layers"][2]["mixer"]["decay_rank"], cfg["layers"][2]["mixer"]["gate_rank"]
    m = model_manifest(_spec(cfg)[1])
    assert m["l0.mix.w1"].shape == (-1, 104) and m["l0.mix.w2"].shape == (48, -1)
    assert m["l2.mix.a1"].shape == (-1, 104) and m["l2.mix.g2"].shape == (96, -1)


def test_a_shared_cache_keeps_what_its_widest_reader_looks_back_at():
    kept = lambda c: [l.parts["mixer"].params["cache_window"] for l in _spec(c)[1].layers
                      if l.parts["mixer"].name == "latent_attention" and l.parts["mixer"].params["own_kv"]]
    assert kept(tp.PA) == [24]                                   # the owner's 24, the reader's 10
    assert kept(tp.PB) == [33, 0]                                # a reader's 33; an owner that sees everything
    assert kept(tp.PL) == [0]                                    # a reader without a window
    assert kept(tp.PD) == [17, 500]


@pytest.mark.parametrize("edit, text", [
    (lambda c: c["layers"][0].update(type="attention"), "no mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "feed-forward kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "router.top"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=0.0), "base"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][2]["mixer"].update(conv=17), "taps"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "latent"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "earlier layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=48), "must be equal"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=99.0), "must be equal"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=-2), "mask.size"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_configuration_errors(edit, text):
    cfg = copy.deepcopy(tp.PA)
    edit(cfg)
    with pytest.raises(ConfigError, match=text):
        _spec(cfg)


# ------------------------------------------------------------------ mechanisms by hand
def test_channel_delta_scan_by_hand():
    k = np.array([[[1.0, 0.0]], [[0.6, 0.8]]])
    q = np.array([[[1.0, 0.0]], [[1.0, 2.0]]])
    v = np.array([[[2.0]], [[10.0]]])
    beta, decay = np.array([[1.0], [0.5]]), np.array([[[0.3, 0.3]], [[0.5, 0.25]]])
    o, S = pp.channel_delta_scan(q, k, v, beta, decay)
    # token 1: u = 2, S = [2, 0]; o = 2.  token 2: S <- [1, 0]; S^T k = .6; u = .5 (10 - .6) = 4.7;
    # S = [1 + .6 * 4.7, .8 * 4.7] = [3.82, 3.76]; o = 3.82 + 2 * 3.76
    assert np.allclose(o[:, 0, 0], [2.0, 3.82 + 7.52]) and np.allclose(S[0, :, 0], [3.82, 3.76])
    # the decay acts on the rows of the key channels, so another order of channels is another result
    o2, _ = pp.channel_delta_scan(q, k, v, beta, decay[..., ::-1])
    assert not np.allclose(o2[1], o[1])
    # two heads on one query/key head, each with a decay of its own
    o3, _ = pp.channel_delta_scan(q, k, np.concatenate([v, v], 1), np.repeat(beta, 2, 1),
                                  np.concatenate([decay, decay[..., ::-1]], 1))
    assert np.allclose(o3[:, 0], o[:, 0]) and np.allclose(o3[:, 1], o2[:, 0])


def test_channel_decay_by_hand():
    w = {"a1": np.array([[1.0, 0.0]]), "a2": np.array([[1.0], [2.0], [0.0], [-1.0]]), "dt_bias": np.array([0.0, 0.1, 0.2, 0.3]),
         "A_log": np.array([0.0, math.log(2.0)])}
    g = pp.channel_decay(np.array([[3.0, 9.0]]), w, "", 2, 2)
    sp = lambda z: math.log1p(math.exp(z))
    assert np.allclose(g[0], [[math.exp(-sp(3.0)), math.exp(-sp(6.1))], [math.exp(-2 * sp(0.2)), math.exp(-2 * sp(-2.7))]])


def test_bonus_scan_by_hand():
    r = np.array([[[1.0, 2.0]], [[1.0, 1.0]]])
    k = np.array([[[3.0, 0.0]], [[1.0, 1.0]]])
    v = np.array([[[2.0]], [[10.0]]])
    decay, u = np.array([[[0.5, 0.5]], [[0.5, 0.25]]]), np.array([[7.0, 1.0]])
    o, S = pp.bonus_scan(r, k, v, decay, u)
    # token 1: S = 0; o = 7 * 3 * 2 = 42 (the write itself scaled by u); S = [6, 0] (not scaled)
    # token 2: o = 6 + (7 + 1) * 10 = 86; S = [.5 * 6 + 10, 10]
    assert np.allclose(o[:, 0, 0], [42.0, 86.0]) and np.allclose(S[0, :, 0], [13.0, 10.0])
    o2, S2 = pp.bonus_scan(r[1:], k[1:], v[1:], decay[1:], u, pp.bonus_scan(r[:1], k[:1], v[:1], decay[:1], u)[1])
    assert np.allclose(o2[0], o[1]) and np.allclose(S2, S)


def test_token_mix_by_hand():
    h = np.array([[1.0, 2.0], [5.0, 6.0]])
    mu = np.array([0.25, 1.0])
    assert np.allclose(pp.token_mix(h, mu), [[0.75, 0.0], [4.0, 2.0]])              # zeros before the first token
    assert np.allclose(pp.token_mix(h[1:], mu, h[0]), [[4.0, 2.0]])


def test_rotation_pairs_neighbours_and_yarn_by_hand():
    x = np.arange(1.0, 5.0).reshape(1, 4)
    y = pp.rotate_pairs(x, [3], {"dims": 4, "base": 100.0})
    a0, a1 = 3.0, 0.3
    assert np.allclose(y[0], [math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + math.sin(a0),
                              3 * math.cos(a1) - 4 * math.sin(a1), 4 * math.cos(a1) + 3 * math.sin(a1)])
    f, mult = pp.yarn(16, 200.0, {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 1.0})
    dim_of = lambda t: 16 * math.log(64 / (2 * math.pi * t)) / (2 * math.log(200.0))
    lo, hi = max(math.floor(dim_of(8.0)), 0), min(math.ceil(dim_of(1.0)), 15)
    assert (lo, hi) == (0, 4) and abs(mult - (0.1 * math.log(8.0) + 1)) < 1e-12
    for i in range(8):
        ramp = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        base = 200.0 ** (-2 * i / 16)
        assert abs(f[i] - (base / 8 * ramp + base * (1 - ramp))) < 1e-15


def test_sink_and_window_by_hand():
    s = np.array([1.0, 2.0, -np.inf])
    p = pp.sink_softmax(s, 0.5)
    z = math.e + math.e ** 2 + math.exp(0.5)
    assert np.allclose(p, [math.e / z, math.e ** 2 / z, 0.0])
    assert np.allclose(pp.sink_softmax(s, 900.0), 0.0)             # a sink that takes everything
    assert pp.visible(5, range(8), 3).tolist() == [False, False, False, True, True, True, False, False]
    assert pp.visible(5, range(8), 0).tolist() == [True] * 6 + [False] * 2
    assert pp.visible(5, range(8), 1).tolist() == [False] * 5 + [True, False, False]


def test_the_weight_scales_an_experts_input():
    rng = np.random.default_rng(0)
    w = {f"e{e}.{n}": rng.standard_normal(s) for e in range(3) for n, s in (("gate", (4, 6)), ("up", (4, 6)), ("down", (6, 4)))}
    w["router"] = rng.standard_normal((3, 6))
    h = rng.standard_normal((1, 6))
    z = w["router"] @ h[0]
    best = int(np.argmax(z))
    s = 1 / (1 + math.exp(-z[best]))
    out = pp.experts(h, w, "", {"router": {"top": 1}})
    g, u = w[f"e{best}.gate"] @ (s * h[0]), w[f"e{best}.up"] @ (s * h[0])
    assert np.allclose(out[0], w[f"e{best}.down"] @ (g / (1 + np.exp(-g)) * u))
    assert not np.allclose(out[0], s * pp.gated(h, w, f"e{best}.")[0])
    idx, wt = pp.choose_experts(np.array([0.1, 3.0, -1.0, 3.0]), 3)
    assert idx == [1, 3, 0] and np.allclose(wt, pp.sigmoid(np.array([3.0, 3.0, 0.1])))      # not renormalised


def test_only_the_result_is_normed():
    x, y = np.array([[3.0, 4.0]]), np.array([[30.0, 40.0]])
    r = math.sqrt(1250.0 + 0.5)
    assert np.allclose(pp.joined(x, y, np.array([1.0, 2.0]), 0.5, 0.25), [[3 + 0.25 * 30 / r, 4 + 0.25 * 80 / r]])


# ------------------------------------------------------------------ the whole model
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    from crane_b200.weights.random_init import write_model_folder
    made = {}

    def get(name):
        if name not in made:
            spec = tp.TINY[name]
            d = tmp_path_factory.mktemp(name)
            write_model_folder(str(d), spec["config"], spec["seed"], "float32", std=spec["std"], norm_std=spec["norm_std"])
            made[name] = pp.load_folder(str(d))
        return made[name]
    return get


@pytest.mark.parametrize("name", ["PA", "PB", "PC", "PD"])
def test_cut_anywhere_the_logits_stay(name, folders):
    cfg, w = folders(name)
    rng = np.random.default_rng(1)
    toks = rng.integers(0, cfg["vocab"], 41).tolist()
    whole, streams, _ = pp.forward(cfg, w, toks)
    assert whole.shape == (41, cfg["vocab"]) and streams.shape == (len(cfg["layers"]), 41, cfg["width"])
    got, state, pos = [], None, 0
    for n in (1, 2, 17, 1, 20):
        part, _, state = pp.forward(cfg, w, toks[pos:pos + n], state, start=pos)
        got.append(part)
        pos += n
    assert np.abs(np.concatenate(got) - whole).max() < 1e-10
    # causal: what comes later changes nothing before it
    other = toks[:10] + rng.integers(0, cfg["vocab"], 31).tolist()
    assert np.abs(pp.logits_all(cfg, w, other)[:10] - whole[:10]).max() < 1e-12


def test_a_token_outside_every_window_is_forgotten(folders):
    """PD with a window of 17 in its middle layer: that layer looks 16 positions back, and the last one reads
    rows of the first layer, which hold one token each, so nothing is older than 16 positions."""
    cfg, w = folders("PD")
    cfg = copy.deepcopy(cfg)
    cfg["layers"][1]["mixer"]["mask"]["size"] = 17
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 50).tolist()
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    a, b = pp.logits_all(cfg, w, toks), pp.logits_all(cfg, w, other)
    assert np.abs(a[17:] - b[17:]).max() < 1e-12 and np.abs(a[16] - b[16]).max() > 1e-6
