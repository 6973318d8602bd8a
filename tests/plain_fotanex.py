"""A plain, slow Fotanex in numpy float64: one function per mechanism, written from the design's equations.

It shares no code with the library: the tests compare the library's kernels, cache and step function with it.
A model is (config dict as in config.json, {tensor name: float64 array}); `forward` runs one whole sequence and
returns the logits of every position (and, if asked, the residual stream after every layer that was run).
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from plain_gptj import read_safetensors


def load_model(folder):
    """(config dict, {tensor name: float64 array}) of a model folder (the reader is `plain_gptj`'s, also test code)."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    w = {}
    for f in sorted(folder.glob("*.safetensors")):
        w.update(read_safetensors(f))
    return cfg, w


# ----------------------------------------------------------------------------- small pieces

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(z, 0.0)


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def tanh_norm(x, alpha, w, b):
    """The dynamic tanh: no statistics, tanh(alpha x) w + b."""
    return np.tanh(alpha * x) * w + b


def named_tanh_norm(x, w, name):
    return tanh_norm(x, float(w[name + ".alpha"]), w[name], w[name + ".b"])


def causal_conv(x, taps, bias):
    """x [T, C], taps [C, n]: out[t, c] = bias[c] + sum_j taps[c, n - 1 - j] x[t - j, c], x zero before the start."""
    T, n = x.shape[0], taps.shape[1]
    out = np.tile(bias, (T, 1)).astype(np.float64)
    for j in range(n):
        out[j:] += taps[:, n - 1 - j] * x[:max(T - j, 0)]
    return out


# ----------------------------------------------------------------------------- attention in chunks

def chunk_attention(m, w, p, h):
    """Grouped softmax attention without positions, inside chunks of positions, a sink in the denominator, one gate
    value per head."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    q = (h @ w[p + "q"].T).reshape(T, H, d)
    k = (h @ w[p + "k"].T).reshape(T, G, d)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    gate = sigmoid(h @ w[p + "g"].T)
    size = (m.get("mask") or {}).get("size", 0)
    pos = np.arange(T)
    i, j = pos[:, None], pos[None, :]
    visible = (j <= i) & ((i // size == j // size) if size else True)
    out = np.zeros((T, H, dv))
    for hh in range(H):
        g = hh // (H // G)
        s = np.where(visible, (q[:, hh] @ k[:, g].T) * m["scale"], -np.inf)
        sink = float(w[p + "sink"][hh])
        top = np.maximum(s.max(-1, keepdims=True), sink)
        e = np.exp(s - top)
        out[:, hh] = (e / (e.sum(-1, keepdims=True) + np.exp(sink - top))) @ v[:, g] * gate[:, hh:hh + 1]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ----------------------------------------------------------------------------- recurrences

def selective_walk(x, dt, A, B, C, D, S):
    """x, dt [T, inner], A [inner, N], B, C [T, N]; from the state S [inner, N].  Returns (y, S)."""
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba(m, w, p, h):
    n, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + "in"].T
    x, z = xz[:, :n], xz[:, n:]
    x = silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    low = x @ w[p + "x"].T
    dt = softplus(low[:, :R] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_walk(x, dt, -np.exp(w[p + "A_log"]), low[:, R:R + N], low[:, R + N:], w[p + "D"], np.zeros((n, N)))
    return (y * silu(z)) @ w[p + "o"].T


def gated_lru_walk(u, r, i, lam, S):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam); returns (S of every token, the last)."""
    out = np.zeros_like(u)
    log_a = -8.0 * r * softplus(lam)
    a, b = np.exp(log_a), np.sqrt(-np.expm1(2.0 * log_a))
    for t in range(u.shape[0]):
        S = a[t] * S + b[t] * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(m, w, p, h):
    nb = m["blocks"]
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    T, n = u.shape
    ub = u.reshape(T, nb, n // nb)
    r = sigmoid(np.einsum("boi,tbi->tbo", w[p + "ra"], ub) + w[p + "ra.b"]).reshape(T, n)
    i = sigmoid(np.einsum("boi,tbi->tbo", w[p + "ri"], ub) + w[p + "ri.b"]).reshape(T, n)
    S, _ = gated_lru_walk(u, r, i, w[p + "lam"], np.zeros(n))
    return (S * y) @ w[p + "o"].T


def ssd_walk(x, dt, A, B, C, S):
    """x [T, H, dv], dt [T, H], A [H] (negative), B, C [T, H, N]; from the state S [H, N, dv].  Returns (y, S)."""
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(A * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, C[t])
    return y, S


def gate_then_group_norm(y, z, w, groups, eps):
    v = y * silu(z)
    T, n = v.shape
    g = v.reshape(T, groups, n // groups)
    return (g / np.sqrt((g * g).mean(-1, keepdims=True) + eps)).reshape(T, n) * w


def mamba2(m, w, p, h, eps):
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    n, T = H * dv, h.shape[0]
    zx = h @ w[p + "in"].T
    z, xbc, dt = zx[:, :n], zx[:, n:2 * n + 2 * G * N], zx[:, 2 * n + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :n].reshape(T, H, dv)
    B = np.repeat(xbc[:, n:n + G * N].reshape(T, G, N), H // G, axis=1)
    C = np.repeat(xbc[:, n + G * N:].reshape(T, G, N), H // G, axis=1)
    dt = softplus(dt + w[p + "dt_bias"])
    y, _ = ssd_walk(x, dt, -np.exp(w[p + "A_log"]), B, C, np.zeros((H, N, dv)))
    y = y + w[p + "D"][:, None] * x
    return gate_then_group_norm(y.reshape(T, n), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ----------------------------------------------------------------------------- mixers, feed-forward

def halves_of_a_pair(left, right, w_left, w_right, eps):
    return 0.5 * (rms_norm(left, w_left, eps) + rms_norm(right, w_right, eps))


def mixer(layer, w, p, h, eps):
    kind, m = layer["type"], layer["mixer"]
    if kind == "parallel":
        left = chunk_attention(m["left"], w, p + "left.", h)
        right = mamba(m["right"], w, p + "right.", h)
        return halves_of_a_pair(left, right, w[p + "left.out"], w[p + "right.out"], eps)
    if kind == "rglru":
        return rglru(m, w, p, h)
    if kind == "mamba2":
        return mamba2(m, w, p, h, eps)
    raise ValueError(kind)


def expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """The chosen experts and their weights for router logits z [T, E]: the largest softmax scores, made to sum to one."""
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    weights = np.take_along_axis(s, chosen, -1)
    return chosen, weights / (weights.sum(-1, keepdims=True) + 1e-20)


def moe(mlp, w, p, h):
    r = mlp["router"]
    chosen, weights = route(h @ w[p + "router"].T, r["top"])
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weights[rows, place][:, None] * expert(w, f"{p}e{e}.", h[rows])
    return out


# ----------------------------------------------------------------------------- the model

def layer_step(cfg, w, i, x):
    """x + (mixer(norm1 x) + ff(norm2 x)) of layer i."""
    layer, eps = cfg["layers"][i], cfg["norm"]["eps"]
    y = mixer(layer, w, f"l{i}.mix.", named_tanh_norm(x, w, f"l{i}.norm1"), eps)
    if layer.get("mlp") is not None:
        y = y + moe(layer["mlp"], w, f"l{i}.mlp.", named_tanh_norm(x, w, f"l{i}.norm2"))
    return x + y


def enter_pass(w, x, x0, t):
    """What happens to the stream before pass number t of the loop."""
    return np.concatenate([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one whole sequence; with `want_layers` also the stream after every layer run [runs, T, width]."""
    x0 = w["embed"][np.asarray(tokens, dtype=np.int64)]
    x, after, n = x0, [], len(cfg["layers"])
    loop = cfg.get("loop")
    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)

    def run(i, x):
        x = layer_step(cfg, w, i, x)
        after.append(x)
        return x
    for i in range(start):
        x = run(i, x)
    for t in range(times):
        x = enter_pass(w, x, x0, t)
        for i in range(start, stop):
            x = run(i, x)
    for i in range(stop, n):
        x = run(i, x)
    logits = named_tanh_norm(x, w, "final.norm") @ w["head"].T
    return (logits, np.stack(after)) if want_layers else logits


def greedy(cfg, w, prompt, n_new):
    """The tokens a greedy decoder appends to `prompt`, each step a whole forward pass."""
    tokens, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(np.argmax(forward(cfg, w, tokens)[-1]))
        out.append(nxt)
        tokens.append(nxt)
    return out
