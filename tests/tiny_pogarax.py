"""Tiny Pogarax configurations for tests.  They differ from one another in every size, and each sets apart
what a model may happen to make equal or 1: query/key heads and heads, key and value widths, the
inner sizes of the low-rank products, the queries' and the keys' latent, windows of a cache's owner and
of the layers that read it, the experts chosen and there, the residual multiplier."""
import copy


def _delta(heads, kv_heads, dim, vdim, conv, ra, rg):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ra, "gate_rank": rg}
    if kv_heads:
        m["kv_heads"] = kv_heads
    return {"type": "channel_delta", "mixer": m}


def _wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def _latent(heads, dim, rot, vdim, r, rq, scale, base, window, scaling=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": r, "q_rank": rq, "scale": scale,
         "rot": {"dims": rot, "base": base}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def _dense(layer, ff):
    return dict(layer, mlp={"kind": "dense", "ff": ff})


def _moe(layer, experts, top, ff):
    return dict(layer, mlp={"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}})


def _none(layer):
    return dict(layer, mlp=None)


YARN = (4.0, 256, 16.0, 1.0)

# all three mixers; two query/key heads for four heads; a reader that looks back less than the cache's owner
PA = {
    "architecture": "Pogarax", "vocab": 199, "width": 104, "norm": {"eps": 1e-6}, "residual_mult": 0.45,
    "layers": [
        _dense(_wkv(3, 16, 5), 72),
        _moe(_latent(5, 24, 8, 20, 40, 56, 0.21, 5000.0, 24, YARN), 5, 2, 24),
        _moe(_delta(4, 2, 16, 24, 3, 6, 9), 4, 1, 40),
        _none(_latent(3, 16, 8, 32, 40, 24, 0.3, 5000.0, 10, YARN, kv_from=1)),
        _dense(_delta(3, None, 24, 16, 5, 7, 2), 48),
    ],
}

# a reader that looks back further than the owner, and one without a window; one query/key head for five; a
# convolution of one tap; all experts chosen; no YaRN; a width off the multiples of 8; no residual multiplier
PB = {
    "architecture": "Pogarax", "vocab": 127, "width": 68, "norm": {"eps": 1e-5},
    "layers": [
        _dense(_latent(2, 12, 12, 8, 24, 17, 0.4, 300.0, 9), 36),
        _moe(_delta(5, 1, 16, 8, 1, 3, 4), 3, 3, 20),
        _none(_latent(4, 8, 12, 16, 24, 30, 0.35, 300.0, 33, kv_from=0)),
        _moe(_wkv(2, 24, 11), 7, 3, 12),
        _dense(_latent(3, 20, 4, 12, 32, 20, 0.25, 90.0, 0), 28),
        _none(_latent(1, 16, 4, 24, 32, 12, 0.3, 90.0, 5, kv_from=4)),
    ],
}

# recurrences only (no layer asks for pages); heads of 8 and of 40 (rows past the lanes' own); a decay's inner size
# above the heads' width
PC = {
    "architecture": "Pogarax", "vocab": 89, "width": 56, "norm": {"eps": 1e-5}, "residual_mult": 1.7,
    "layers": [
        _moe(_wkv(1, 40, 44), 6, 2, 16),
        _none(_delta(2, 2, 40, 12, 2, 4, 4)),
        _dense(_wkv(5, 8, 3), 24),
        _moe(_delta(6, 3, 8, 8, 4, 2, 5), 4, 2, 8),
    ],
}

# latent attention only; a window of one (a token sees itself and the sink) beside one longer than any prompt;
# the YaRN ramp inside the rotated part
PD = {
    "architecture": "Pogarax", "vocab": 75, "width": 48, "norm": {"eps": 1e-6}, "residual_mult": 0.8,
    "layers": [
        _dense(_latent(3, 16, 16, 16, 16, 24, 0.3, 200.0, 1, (8.0, 64, 8.0, 1.0)), 40),
        _moe(_latent(7, 8, 16, 8, 48, 16, 0.28, 900.0, 500, (2.0, 128, 4.0, 2.0)), 9, 4, 8),
        _none(_latent(2, 24, 16, 12, 16, 40, 0.22, 200.0, 17, (8.0, 64, 8.0, 1.0), kv_from=0)),
    ],
}

# layer sizes at which the tensor-core kernels are taken (grouped products among them)
PL = {
    "architecture": "Pogarax", "vocab": 512, "width": 512, "norm": {"eps": 1e-5}, "residual_mult": 0.6,
    "layers": [
        _moe(_wkv(8, 64, 32), 8, 2, 128),
        _dense(_delta(8, 4, 64, 64, 4, 32, 48), 1024),
        _dense(_latent(8, 96, 32, 64, 128, 256, 0.09, 10000.0, 100, YARN), 768),
        _moe(_delta(4, 4, 128, 64, 3, 64, 24), 6, 1, 256),
        _none(_latent(16, 64, 32, 128, 128, 192, 0.1, 10000.0, 0, YARN, kv_from=2)),
        _dense(_wkv(3, 128, 20), 512),
    ],
}


def all_chosen(config):
    """The same with every expert of every layer chosen: no choice that rounding could flip, so whole-model logits
    can be compared closely in bfloat16."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


TINY = {
    "PA": {"config": PA, "seed": 51, "std": 0.1, "norm_std": 0.05, "page_size": 16},
    "PB": {"config": PB, "seed": 52, "std": 0.12, "norm_std": 0.05, "page_size": 8},
    "PC": {"config": PC, "seed": 53, "std": 0.12, "norm_std": 0.05, "page_size": 16},
    "PD": {"config": PD, "seed": 54, "std": 0.14, "norm_std": 0.05, "page_size": 32},
    "PL": {"config": PL, "seed": 55, "std": 0.04, "norm_std": 0.05, "page_size": 64},
}
for _name in list(TINY):
    TINY[_name + "-all"] = dict(TINY[_name], config=all_chosen(TINY[_name]["config"]), seed=TINY[_name]["seed"] + 10)
