"""A plain, slow Vofinex in numpy float64: one function per mechanism, written from the design's equations.

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

def silu(z):
    return z / (1.0 + np.exp(-z))


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def unit_rms(x, eps):
    """x over its root mean square along the last axis; no weight."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rotate(x, pos, dims, base):
    """x [T, heads, d]: element i < dims / 2 of a head turns together with element i + dims / 2 by pos * base^(-2i/dims);
    the elements from dims on stay."""
    if dims == 0:
        return x
    half = dims // 2
    a = np.asarray(pos, dtype=np.float64)[:, None] * float(base) ** (-2.0 * np.arange(half) / dims)[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def queries_and_keys(m, q, k, pos, eps):
    """Rotated first, then every head brought to a root mean square of one."""
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    return tuple(unit_rms(rotate(x, pos, rot["dims"], rot["base"]), eps) for x in (q, k))


def visible_keys(n, size):
    """[n, n]: which keys j a query i sees: its own chunk's up to itself (size 0: all up to itself)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def attend(q, k, v, scale, sink, visible):
    """Softmax attention of q [T, H, d] over k [T, G, d] and v [T, G, dv] (query head h reads key head h // (H / G)), exp(sink[h])
    one more term of the denominator: [T, H, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for hh in range(H):
        g = hh // (H // G)
        s = np.where(visible, (q[:, hh] @ k[:, g].T) * scale, -np.inf)
        top = np.maximum(s.max(-1, keepdims=True), sink[hh])
        e = np.exp(s - top)
        out[:, hh] = (e / (e.sum(-1, keepdims=True) + np.exp(sink[hh] - top))) @ v[:, g]
    return out


def attention(m, w, p, h, eps):
    """Grouped softmax attention inside chunks of positions, with a learned sink per head in the denominator."""
    T = h.shape[0]
    H, d = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    q, k = queries_and_keys(m, (h @ w[p + "q"].T).reshape(T, H, d), (h @ w[p + "k"].T).reshape(T, G, d), np.arange(T), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, dv)
    out = attend(q, k, v, m["scale"], w[p + "sink"], visible_keys(T, (m.get("mask") or {}).get("size", 0)))
    return out.reshape(T, H * dv) @ w[p + "o"].T


def gated_unit(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, top):
    """The chosen experts and their weights for router logits z [T, E]: a softmax over all, the correction counts for the
    choice only, the weights are the scores as they are."""
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    chosen = np.argsort(-(s + correction), axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, -1)


def moe(mlp, w, p, h):
    """Experts 0 .. experts - 1 have matrices; the router's last `identity` outputs return h itself."""
    r = mlp["router"]
    chosen, weights = route(h @ w[p + "router"].T, w[p + "correction"], r["top"])
    out = np.zeros_like(h)
    for e in range(r["experts"] + (r.get("identity") or 0)):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            y = gated_unit(w, f"{p}e{e}.", h[rows]) if e < r["experts"] else h[rows]
            out[rows] += weights[rows, place][:, None] * y
    return out


# ----------------------------------------------------------------------------- the model

def layer_step(cfg, w, i, x):
    """x + m (mixer(h) + ff(h)), h the one norm of x that both read."""
    layer, eps = cfg["layers"][i], cfg["norm"]["eps"]
    h = layer_norm(x, w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
    y = attention(layer["mixer"], w, f"l{i}.mix.", h, eps)
    mlp = layer.get("mlp")
    if mlp is not None:
        y = y + (gated_unit(w, f"l{i}.mlp.", h) if mlp["kind"] == "dense" else moe(mlp, w, f"l{i}.mlp.", h))
    return x + cfg["residual_mult"] * y


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of one whole sequence; with `want_layers` also the stream after every layer run [runs, T, width]."""
    x = w["embed"][np.asarray(tokens, dtype=np.int64)] * cfg["embedding"]["scale"]
    after, n = [], len(cfg["layers"])
    loop = cfg.get("loop")
    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)

    def run(i, x):
        x = layer_step(cfg, w, i, x)
        after.append(x)
        return x
    for i in range(start):
        x = run(i, x)
    for t in range(times):
        x = x + w["loop.step"][t]
        for i in range(start, stop):
            x = run(i, x)
    for i in range(stop, n):
        x = run(i, x)
    z = layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"])
    logits = z @ w["embed"].T * cfg["logit_scale"]
    return (logits, np.stack(after)) if want_layers else logits


def greedy(cfg, w, prompt, n_new):
    """The tokens a greedy decoder appends to `prompt`, each step a whole forward pass."""
    tokens, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(np.argmax(forward(cfg, w, tokens)[-1]))
        out.append(nxt)
        tokens.append(nxt)
    return out
