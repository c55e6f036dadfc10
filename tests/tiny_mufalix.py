"""Tiny Mufalix configurations for tests.  They differ from one another in every size, and each sets apart
what a model may happen to make equal or 1: key and value widths, query and key/value heads, rotated and head
width, the recurrence's parts and taps, where the repeated layers begin and end and how often they run, the
experts chosen and there, the embedding's and the router's constants."""
import copy


def _attention(heads, kv_heads, dim, vdim, scale, window, rot=None):
    m = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads:
        m["kv_heads"] = kv_heads
    if vdim:
        m["vdim"] = vdim
    if window:
        m["mask"] = {"size": window}
    if rot:
        dims, base, scaling = rot
        m["rot"] = {"dims": dims, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _parallel(left, width, blocks, conv):
    return {"type": "parallel", "mixer": {"left": left, "right": {"width": width, "blocks": blocks, "conv": conv}}}


def _mlstm(heads, dim, vdim, cap):
    m = {"heads": heads, "dim": dim, "gate_cap": cap}
    if vdim:
        m["vdim"] = vdim
    return {"type": "mlstm", "mixer": m}


def _moe(layer, experts, top, scale, ff):
    return dict(layer, mlp={"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}})


def _none(layer):
    return dict(layer, mlp=None)


LLAMA = (8.0, 1.0, 4.0, 64)

# both mixers in the repeated range, layers before and behind it; keys narrower than values, both narrower than the
# head they are stored at; frequencies kept, mixed and divided; parts of 10 channels; a layer without feed-forward
FA = {
    "architecture": "Mufalix", "vocab": 157, "width": 72, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.7},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        _moe(_parallel(_attention(4, 2, 14, 24, 0.31, 11, (8, 100.0, LLAMA)), 40, 4, 3), 5, 2, 0.8, 24),
        _moe(_mlstm(3, 16, 8, 5.0), 4, 1, 2.5, 40),
        _none(_parallel(_attention(3, None, 20, 12, 0.2, 7, (20, 50.0, None)), 48, 3, 4)),
        _moe(_mlstm(2, 24, 40, 15.0), 6, 3, 1.0, 16),
    ],
}

# the range begins with the first layer; one key/value head for five, no rotation, no window; one part and one tap;
# all experts chosen; a width off the multiples of 8; no scale of the embedding
FB = {
    "architecture": "Mufalix", "vocab": 101, "width": 68, "norm": {"eps": 1e-5}, "loop": {"start": 0, "stop": 1, "times": 3},
    "layers": [
        _moe(_parallel(_attention(5, 1, 16, None, 0.4, 0), 24, 1, 1), 3, 3, 1.3, 20),
        _moe(_mlstm(1, 8, 24, 2.0), 7, 4, 1.0, 12),
        _moe(_parallel(_attention(2, 2, 32, 8, 0.18, 33, (4, 1000.0, (2.0, 2.0, 3.0, 128))), 36, 2, 2), 4, 2, 0.6, 28),
    ],
}

# recurrences only (no layer asks for pages), nothing repeated; heads of 40 (rows past the lanes' own) and of 8
FC = {
    "architecture": "Mufalix", "vocab": 83, "width": 56, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.0},
    "layers": [
        _moe(_mlstm(2, 40, 12, 4.0), 6, 2, 1.1, 16),
        _none(_mlstm(5, 8, 16, 30.0)),
        _moe(_mlstm(1, 20, 36, 8.0), 4, 2, 0.9, 8),
    ],
}

# pairs only, all of them repeated; a window of one (a token sees itself and the sink) beside one longer than any
# prompt; heads of odd widths; more taps than the sliding form takes
FD = {
    "architecture": "Mufalix", "vocab": 75, "width": 48, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.9},
    "loop": {"start": 0, "stop": 3, "times": 2},
    "layers": [
        _moe(_parallel(_attention(3, 3, 17, 9, 0.33, 1, (2, 20.0, None)), 32, 2, 6), 9, 4, 1.7, 8),
        _none(_parallel(_attention(6, 2, 16, 16, 0.25, 500, (16, 900.0, (4.0, 1.0, 2.0, 256))), 45, 5, 5)),
        _moe(_parallel(_attention(2, 1, 48, 30, 0.15, 17, (12, 200.0, (16.0, 0.5, 8.0, 32))), 16, 1, 2), 2, 1, 1.0, 16),
    ],
}

# layer sizes at which the tensor-core kernels are taken: heads stored at 128 (tiles by TMA, slices merged in a
# cluster) and at 96, parts of 256, 64 and 416 channels (the last beyond the tensor-core kernel)
FL = {
    "architecture": "Mufalix", "vocab": 512, "width": 512, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.2},
    "loop": {"start": 1, "stop": 2, "times": 2},
    "layers": [
        _moe(_parallel(_attention(8, 2, 128, 128, 0.09, 100, (64, 10000.0, (8.0, 1.0, 4.0, 256))), 512, 2, 4), 8, 2, 1.4, 128),
        _moe(_mlstm(4, 64, 128, 15.0), 6, 3, 1.0, 128),
        _moe(_parallel(_attention(6, 3, 64, 90, 0.12, 0, (32, 10000.0, None)), 640, 10, 3), 4, 4, 0.7, 256),
        _moe(_mlstm(2, 128, 64, 10.0), 5, 1, 1.0, 192),
        _none(_parallel(_attention(4, 4, 112, 128, 0.1, 64, None), 832, 2, 4)),
    ],
}


# more query heads per key/value head than the decode kernel's tile has rows
FG = {
    "architecture": "Mufalix", "vocab": 120, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.5},
    "layers": [
        _none(_parallel(_attention(20, 1, 16, 16, 0.3, 12, (8, 100.0, None)), 32, 2, 3)),
        _moe(_mlstm(2, 16, 16, 6.0), 3, 3, 1.2, 16),
        _none(_parallel(_attention(34, 2, 32, 24, 0.2, 0, None), 48, 1, 4)),
    ],
}


def all_chosen(config):
    """The same with every expert of every layer chosen: no choice that rounding could flip, so whole-model logits
    can be compared closely in bfloat16."""
    out = copy.deepcopy(config)
    for layer in out["layers"]:
        if layer["mlp"] is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return out


TINY = {
    "FA": {"config": FA, "seed": 61, "std": 0.12, "norm_std": 0.05, "page_size": 16},
    "FB": {"config": FB, "seed": 62, "std": 0.12, "norm_std": 0.05, "page_size": 8},
    "FC": {"config": FC, "seed": 63, "std": 0.14, "norm_std": 0.05, "page_size": 16},
    "FD": {"config": FD, "seed": 64, "std": 0.15, "norm_std": 0.05, "page_size": 32},
    "FL": {"config": FL, "seed": 65, "std": 0.045, "norm_std": 0.05, "page_size": 64},
    "FG": {"config": FG, "seed": 66, "std": 0.12, "norm_std": 0.05, "page_size": 16},
}
for _name in list(TINY):
    TINY[_name + "-all"] = dict(TINY[_name], config=all_chosen(TINY[_name]["config"]), seed=TINY[_name]["seed"] + 10)
