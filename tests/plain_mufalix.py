"""A plain, slow restatement of Mufalix in NumPy float64, one function per mechanism, written from the
design's equations and sharing nothing with the engine.

Notation: n tokens, W width, H heads, G key/value heads, d key size, m value size, E experts, C channels of
the gated linear recurrence.  Weights are dictionaries name -> float64 array.  Every matrix is stored
[out, in] and applied as ``x @ M.T`` to rows x.  Functions with a memory take and return it, so a sequence can
be run in one call or continued from where another call stopped.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional

import numpy as np
import torch

from crane_b200.weights.safetensors_io import TensorSource, model_files


def load_folder(folder: str):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    src = TensorSource(model_files(folder))
    w = {}
    for name in src.names():
        t = src.tensor(name)
        w[name] = t.to(torch.float64).numpy() if t.dtype.is_floating_point else t.numpy()
    return cfg, w


# ------------------------------------------------------------------ small functions
def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.logaddexp(0.0, z)


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def over_rms(x, eps):
    """x over the root of its mean square, eps under the root."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return over_rms(x, eps) * w


# ------------------------------------------------------------------ positions
def rotary_frequencies(dims: int, base: float, scaling=None):
    """f_i = base^(-2 i / dims); with ``scaling`` (factor, low, high, original) by wavelength l = 2 pi / f:
    f where l < original / high, f / factor where l > original / low, in between the mix
    (1 - s) f / factor + s f with s = (original / l - low) / (high - low)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wavelength = 2.0 * math.pi / f
            if wavelength < original / high:
                pass
            elif wavelength > original / low:
                f = f / factor
            else:
                s = (original / wavelength - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return np.array(out)


def rotate_half(x, positions, freq):
    """x [n, heads, d]: of the leading 2 len(freq) elements of every head, element i turns with element
    i + len(freq) by the angle p freq_i; the others stay."""
    half = len(freq)
    out = x.copy()
    if half == 0:
        return out
    a = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


# ------------------------------------------------------------------ attention with a sink and a window
def sink_window_attention(q, k, v, scale: float, window: int, sink, first_query: int = 0):
    """q [n, H, d] at positions first_query .. first_query + n - 1; k [N, G, d], v [N, G, m] at positions
    0 .. N - 1.  Position i sees j with 0 <= i - j < window (0: every j <= i); the softmax's denominator also
    holds exp(sink_h).  Returns [n, H, m]."""
    n, H, _ = q.shape
    N, G, m = v.shape
    i, j = first_query + np.arange(n)[:, None], np.arange(N)[None, :]
    seen = (j <= i) & ((i - j < window) if window else True)
    out = np.zeros((n, H, m))
    for h in range(H):
        g = h // (H // G)
        s = np.where(seen, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = np.maximum(s.max(axis=1, keepdims=True), sink[h])
        e = np.exp(s - top)
        out[:, h] = (e / (e.sum(axis=1, keepdims=True) + np.exp(sink[h] - top))) @ v[:, g]
    return out


def attention_side(h, w, p: str, a: dict, eps: float, memory=None, start: int = 0):
    """``memory``: (keys, values) of positions 0 .. start - 1 or None."""
    H, d = int(a["heads"]), int(a["dim"])
    G, m = int(a.get("kv_heads") or H), int(a.get("vdim") or d)
    n = h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(n, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(n, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(n, G, m)
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    rot = a.get("rot")
    if rot:
        freq = rotary_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
        positions = start + np.arange(n)
        q, k = rotate_half(q, positions, freq), rotate_half(k, positions, freq)
    if memory is not None:
        k, v = np.concatenate([memory[0], k]), np.concatenate([memory[1], v])
    o = sink_window_attention(q, k, v, float(a["scale"]), int((a.get("mask") or {}).get("size") or 0), w[p + "sink"], start)
    o = o.reshape(n, H * m) * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T + w[p + "o.b"], (k, v)


# ------------------------------------------------------------------ the gated linear recurrence
def short_convolution(x, taps_w, bias, before=None):
    """y_t[c] = bias[c] + sum_j w[c, j] x_(t - (T - 1) + j)[c], zeros before the start.  ``before`` [T - 1, C]: the
    inputs just before x.  Returns (y [n, C], the last T - 1 inputs)."""
    n, C = x.shape
    T = taps_w.shape[1]
    past = np.zeros((T - 1, C)) if before is None else before
    ext = np.concatenate([past, x], axis=0)
    y = np.zeros((n, C))
    for t in range(n):
        y[t] = (ext[t:t + T] * taps_w.T).sum(axis=0) + bias
    return y, ext[ext.shape[0] - (T - 1):].copy()


def block_product(u, mats, bias):
    """u [n, B c], mats [B, c, c] ([out, in] each), bias [B, c]: part b of the row through matrix b."""
    B, c, _ = mats.shape
    return np.concatenate([u[:, b * c:(b + 1) * c] @ mats[b].T + bias[b] for b in range(B)], axis=1)


def linear_recurrence(u, r, i, lam, state=None):
    """Per channel: log a = -8 r softplus(lam); S_t = a S_(t-1) + sqrt(1 - a^2) i u.  All [n, C]; ``state`` [C]."""
    S = np.zeros(u.shape[1]) if state is None else state.copy()
    out = np.zeros(u.shape)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * softplus(lam)
        S = np.exp(log_a) * S + np.sqrt(-np.expm1(2.0 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def recurrent_side(h, w, p: str, state=None):
    """``state``: (S [C], the convolution's last inputs) or None."""
    S, kept = state if state is not None else (None, None)
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u, kept = short_convolution(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"], kept)
    r = sigmoid(block_product(u, w[p + "ra"], w[p + "ra.b"]))
    i = sigmoid(block_product(u, w[p + "ri"], w[p + "ri.b"]))
    o, S = linear_recurrence(u, r, i, w[p + "lam"], S)
    return (o * y) @ w[p + "o"].T, (S, kept)


def parallel_mixer(h, w, p: str, a: dict, eps: float, memory=None, start: int = 0):
    """Both sides on the same input; half the sum of their results, each normed over the width first."""
    ml, mr = memory if memory is not None else (None, None)
    x, ml = attention_side(h, w, p + "left.", a["left"], eps, ml, start)
    y, mr = recurrent_side(h, w, p + "right.", mr)
    return 0.5 * (rms_norm(x, w[p + "left.out"], eps) + rms_norm(y, w[p + "right.out"], eps)), (ml, mr)


# ------------------------------------------------------------------ a matrix memory with exponential gates
def stabilised_scan(q, k, v, log_i, log_f, state=None):
    """q, k [n, H, d], v [n, H, m], gates [n, H].  With a running maximum M (0 at first):
    M' = max(f + M, i); S <- exp(f + M - M') S + exp(i - M') k v^T; N likewise with k alone;
    o = S^T q / (max(|N . q|, exp(-M')) + 1e-6).  ``state``: (S [H, d, m], N [H, d], M [H])."""
    n, H, d = q.shape
    m = v.shape[2]
    if state is None:
        S, N, M = np.zeros((H, d, m)), np.zeros((H, d)), np.zeros(H)
    else:
        S, N, M = (a.copy() for a in state)
    out = np.zeros((n, H, m))
    for t in range(n):
        new = np.maximum(log_f[t] + M, log_i[t])
        keep, add = np.exp(log_f[t] + M - new), np.exp(log_i[t] - new)
        M = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        N = keep[:, None] * N + add[:, None] * k[t]
        den = np.maximum(np.abs((N * q[t]).sum(-1)), np.exp(-M)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(axis=1) / den[:, None]
    return out, (S, N, M)


def mlstm_mixer(h, w, p: str, a: dict, eps: float, state=None):
    H, d = int(a["heads"]), int(a["dim"])
    m = int(a.get("vdim") or d)
    cap = float(a["gate_cap"])
    n = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(n, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, H, d)
    v = (h @ w[p + "v"].T).reshape(n, H, m)
    log_i = cap * np.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    log_f = log_sigmoid(cap * np.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, state = stabilised_scan(q, k, v, log_i, log_f, state)
    o = over_rms(o, eps).reshape(n, H * m) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T, state


# ------------------------------------------------------------------ feed-forward
def choose_experts(z, correction, top: int, scale: float):
    """One token's router logits z [E]: scores s = sigmoid(z); the ``top`` largest of s + correction are chosen
    (ties to the lower index); weights are their s over the sum of those (+ 1e-20), times ``scale``."""
    s = sigmoid(z)
    order = sorted(range(len(z)), key=lambda e: (-(s[e] + correction[e]), e))[:top]
    return order, s[order] / (s[order].sum() + 1e-20) * scale


def moe(h, w, p: str, mlp: dict):
    top, scale = int(mlp["router"]["top"]), float(mlp["router"]["scale"])
    z = h @ w[p + "router"].T
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, a in zip(*choose_experts(z[t], w[p + "correction"], top, scale)):
            out[t] += a * (squared_relu(h[t] @ w[f"{p}e{e}.up"].T) @ w[f"{p}e{e}.down"].T)
    return out


# ------------------------------------------------------------------ the model
def layer_runs(cfg: dict):
    """(layer, whether a pass of the repeated range begins with this run) in the order of running."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    passes = [(i, i == a) for _ in range(int(loop["times"])) for i in range(a, b)]
    return [(i, False) for i in range(a)] + passes + [(i, False) for i in range(b, n)]


def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, state: Optional[list] = None, start: int = 0):
    """One sequence's tokens at positions start .. start + n - 1, continued from ``state`` (a list per layer run;
    None: the start).  Returns (logits [n, V], the stream after every run [runs, n, W], state)."""
    eps = float(cfg["norm"]["eps"])
    runs = layer_runs(cfg)
    x = w["embed"][np.asarray(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    x0 = x.copy()
    state = [None] * len(runs) if state is None else list(state)
    streams = []
    for place, (i, enters) in enumerate(runs):
        layer, p = cfg["layers"][i], f"l{i}."
        if enters:
            x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "parallel":
            y, state[place] = parallel_mixer(h, w, p + "mix.", layer["mixer"], eps, state[place], start)
        elif layer["type"] == "mlstm":
            y, state[place] = mlstm_mixer(h, w, p + "mix.", layer["mixer"], eps, state[place])
        else:
            raise ValueError(f"no mixer '{layer['type']}'")
        x = x + y
        if layer.get("mlp") is not None:
            x = x + moe(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        streams.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T, np.stack(streams), state


def logits_all(cfg: dict, w: Dict[str, np.ndarray], tokens) -> np.ndarray:
    """Logits at every position of one sequence, [n, V]."""
    return forward(cfg, w, list(tokens))[0]


def greedy_generate(cfg: dict, w: Dict[str, np.ndarray], prompt: List[int], new_tokens: int) -> List[int]:
    """The prompt and ``new_tokens`` more, each the largest logit's index (ties to the lower index);
    the prompt in one call, then token by token from the carried state."""
    toks = list(prompt)
    logits, _, state = forward(cfg, w, toks)
    for _ in range(new_tokens):
        toks.append(int(np.argmax(logits[-1])))
        logits, _, state = forward(cfg, w, toks[-1:], state, start=len(toks) - 1)
    return toks
