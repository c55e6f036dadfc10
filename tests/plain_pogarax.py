"""A plain, slow restatement of Pogarax in NumPy float64, one function per mechanism, written from the
design's equations and sharing nothing with the engine.

Notation: n tokens, W width, H heads, G query/key heads, d key size, m value size, E experts.  Weights
are dictionaries name -> float64 array.  Every matrix is stored [out, in] and applied as ``x @ M.T`` to
rows x.  Functions with a memory take and return it, so a sequence can be run in one call or continued
from where another call stopped.
"""
from __future__ import annotations

import json
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
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    """x over the root of its mean square, eps under the root."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def unit_vector(x, eps=1e-6):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + eps)


def joined(x, y, w, eps, mult):
    """The stream after a sublayer's result y has joined it: only the result is normed."""
    return x + mult * (over_rms(y, eps) * w)


# ------------------------------------------------------------------ the delta rule with a decay per key channel
def short_convolution(x, taps_w, before=None):
    """y_t[c] = sum_j w[c, j] x_(t - (T - 1) + j)[c], zeros before the start.  x [n, C], taps_w [C, T],
    ``before`` [T - 1, C]: the inputs just before x (None: the start).  Returns (y, the last T - 1 inputs)."""
    n, C = x.shape
    T = taps_w.shape[1]
    ext = np.concatenate([np.zeros((T - 1, C)) if before is None else before, x], axis=0)
    y = np.stack([(ext[t:t + T] * taps_w.T).sum(axis=0) for t in range(n)])
    return y, ext[ext.shape[0] - (T - 1):].copy()


def channel_delta_scan(q, k, v, beta, decay, state=None):
    """Per head: S <- diag(decay_t) S; u = beta_t (v_t - S^T k_t); S <- S + k_t u^T; o_t = S^T q_t.
    q, k [n, G, d] (head h reads q/k head h // (H / G)), v [n, H, m], beta [n, H], decay [n, H, d];
    ``state`` [H, d, m] or None (zeros).  Returns (o [n, H, m], state)."""
    n, H, m = v.shape
    G, d = q.shape[1], q.shape[2]
    S = np.zeros((H, d, m)) if state is None else state.copy()
    o = np.zeros((n, H, m))
    for t in range(n):
        for h in range(H):
            kk, qq = k[t, h // (H // G)], q[t, h // (H // G)]
            S[h] = decay[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + np.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


def channel_decay(h, w, p: str, H: int, d: int):
    """exp(-exp(A_h) softplus(a2 (a1 h) + dt)) per head and key channel, [n, H, d]."""
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    return np.exp(-np.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(-1, H, d))


def channel_delta(h, w, p: str, mx: dict, eps: float, state=None):
    """``state``: (S, the last taps - 1 inputs of the q, k and v convolutions) or None."""
    H, G, d, m = mx["heads"], mx.get("kv_heads") or mx["heads"], mx["dim"], mx["vdim"]
    n = h.shape[0]
    S, cq, ck, cv = state if state is not None else (None, None, None, None)
    q, cq = short_convolution(h @ w[p + "q"].T, w[p + "q.conv"], cq)
    k, ck = short_convolution(h @ w[p + "k"].T, w[p + "k.conv"], ck)
    v, cv = short_convolution(h @ w[p + "v"].T, w[p + "v.conv"], cv)
    q = unit_vector(silu(q).reshape(n, G, d)) * d ** -0.5
    k = unit_vector(silu(k).reshape(n, G, d))
    v = silu(v).reshape(n, H, m)
    beta = sigmoid(h @ w[p + "b"].T)
    o, S = channel_delta_scan(q, k, v, beta, channel_decay(h, w, p, H, d), S)
    o = (over_rms(o, eps) * w[p + "norm"]).reshape(n, H * m)
    o = o * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return o @ w[p + "o"].T, (S, cq, ck, cv)


# ------------------------------------------------------------------ time mixing with a bonus for the current token
def token_mix(h, mu, before=None):
    """h_t + (h_(t-1) - h_t) mu; ``before`` [W]: the row just before h (None: zeros)."""
    prev = np.concatenate([(np.zeros_like(h[:1]) if before is None else before[None]), h[:-1]], axis=0)
    return h + (prev - h) * mu


def bonus_scan(r, k, v, decay, u, state=None):
    """Per head: o_t = (S + diag(u) k_t v_t^T)^T r_t, then S <- diag(decay_t) S + k_t v_t^T.
    r, k, v, decay [n, H, d], u [H, d]; ``state`` [H, d, d] or None.  Returns (o, state)."""
    n, H, d = r.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    o = np.zeros((n, H, v.shape[2]))
    for t in range(n):
        for h in range(H):
            kv = np.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h][:, None] * kv).T @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return o, S


def wkv(h, w, p: str, mx: dict, eps: float, state=None):
    """``state``: (S, the last row of h) or None."""
    H, d = mx["heads"], mx["dim"]
    n = h.shape[0]
    S, last = state if state is not None else (None, None)
    mix = {s: token_mix(h, w[p + "mu." + s], last) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].T).reshape(n, H, d) for s in "rkv")
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(n, H, d)
    o, S = bonus_scan(r, k, v, decay, w[p + "u"].reshape(H, d), S)
    o = over_rms(o, eps).reshape(n, H * d) * w[p + "norm"] * silu(mix["g"] @ w[p + "g"].T)
    return o @ w[p + "o"].T, (S, h[-1].copy())


# ------------------------------------------------------------------ latent attention
def yarn(dims: int, base: float, scaling: Optional[dict]):
    """(frequencies [dims / 2], the factor of cos and sin)."""
    i = np.arange(dims // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0
    def dim_of(turns):
        return dims * np.log(scaling["original"] / (2 * np.pi * turns)) / (2 * np.log(base))
    lo, hi = max(np.floor(dim_of(scaling["fast"])), 0), min(np.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * np.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, rot: Optional[dict]):
    """x [n, ..., e]: elements 2i and 2i + 1 of the leading rot.dims turned by the position's angle."""
    out = x.copy()
    if not rot or not rot["dims"]:
        return out
    dims = int(rot["dims"])
    f, mult = yarn(dims, rot["base"], rot.get("scaling"))
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a) * mult, np.sin(a) * mult
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def latent_rows(h, w, p: str, mx: dict, eps: float, positions):
    """What a layer keeps per position: (the normed latent [n, r], the rotated key part [n, e])."""
    r = int(mx["kv_rank"])
    y = h @ w[p + "dkv"].T
    return over_rms(y[:, :r], eps) * w[p + "dkv.norm"], rotate_pairs(y[:, r:], positions, mx["rot"])


def sink_softmax(s, sink):
    """exp(s_j) / (exp(sink) + sum_i exp(s_i)) along the last axis; -inf scores weigh nothing."""
    top = np.maximum(s.max(-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink - top))


def visible(i: int, j, window: int):
    """Whether position i sees position j: its own and the ``window`` - 1 before it (0: all before it)."""
    j = np.asarray(j)
    return (j <= i) & ((i - j < window) if window else True)


def latent_attention(h, w, p: str, mx: dict, eps: float, positions, c, kr):
    """h [n, W] at ``positions``; c [T, r], kr [T, e]: the kept rows of positions 0 .. T - 1 (T > the last
    of ``positions``), this layer's own or another layer's."""
    H, d, e, m = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    n, T = h.shape[0], c.shape[0]
    cq = over_rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(n, H, d + e)
    qr = rotate_pairs(q[..., d:], positions, mx["rot"])
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, m)
    window = int((mx.get("mask") or {}).get("size") or 0)
    o = np.zeros((n, H, m))
    for t in range(n):
        i = int(positions[t])
        see = visible(i, np.arange(T), window)
        for a in range(H):
            s = (k[:, a] @ q[t, a, :d] + kr @ qr[t, a]) * float(mx["scale"])
            o[t, a] = sink_softmax(np.where(see, s, -np.inf), w[p + "sink"][a]) @ v[:, a]
    return o.reshape(n, H * m) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forwards
def gated(h, w, p: str):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose_experts(z, top: int):
    """One token's router logits z [E]: the ``top`` largest scores sigmoid(z) and their indices."""
    s = sigmoid(z)
    order = sorted(range(z.shape[0]), key=lambda e: (-s[e], e))[:top]
    return order, s[order]


def experts(h, w, p: str, mlp: dict):
    """The weight scales an expert's INPUT: sum of expert(weight * h) over the chosen ones."""
    z = h @ w[p + "router"].T
    out = np.zeros((h.shape[0], w[p + "e0.down"].shape[0]))
    for t in range(h.shape[0]):
        for e, a in zip(*choose_experts(z[t], int(mlp["router"]["top"]))):
            out[t] += gated(a * h[t:t + 1], w, f"{p}e{e}.")[0]
    return out


def feed_forward(h, w, p: str, mlp: dict):
    return gated(h, w, p) if mlp["kind"] == "dense" else experts(h, w, p, mlp)


# ------------------------------------------------------------------ the model
def forward(cfg: dict, w: Dict[str, np.ndarray], tokens, state: Optional[list] = None, start: int = 0):
    """One sequence's tokens at positions start .. start + n - 1, continued from ``state`` (a list per layer;
    None: the start).  Returns (logits [n, V], the stream after every layer [L, n, W], state)."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    n = len(tokens)
    positions = np.arange(start, start + n)
    x = w["embed"][np.asarray(tokens)]
    state = [None] * len(cfg["layers"]) if state is None else list(state)
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        if layer["type"] == "channel_delta":
            y, state[i] = channel_delta(x, w, p + "mix.", mx, eps, state[i])
        elif layer["type"] == "wkv":
            y, state[i] = wkv(x, w, p + "mix.", mx, eps, state[i])
        elif layer["type"] == "latent_attention":
            if mx.get("kv_from") is None:
                rows = latent_rows(x, w, p + "mix.", mx, eps, positions)
                state[i] = rows if state[i] is None else tuple(np.concatenate(ab) for ab in zip(state[i], rows))
                kept = state[i]
            else:
                kept = state[mx["kv_from"]]
            y = latent_attention(x, w, p + "mix.", mx, eps, positions, *kept)
        else:
            raise ValueError(f"no mixer '{layer['type']}'")
        x = joined(x, y, w[p + "norm1"], eps, mult)
        if layer.get("mlp") is not None:
            x = joined(x, feed_forward(x, w, p + "mlp.", layer["mlp"]), w[p + "norm2"], eps, mult)
        streams.append(x)
    return (over_rms(x, eps) * w["final.norm"]) @ w["head"].T, np.stack(streams), state


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
