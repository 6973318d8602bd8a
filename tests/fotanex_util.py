"""Small Fotanex models for the tests: configurations that differ in every size and option, and weights drawn here
with numpy so that every mechanism carries weight in the logits (recurrences whose memories reach from a few tokens to
hundreds, sinks of the order of the scores, routers far from uniform, tanh norms in and out of saturation)."""
from __future__ import annotations

import json

import numpy as np
import torch

from qstream_b200.weights.safetensors_io import SafetensorsFile, write_safetensors


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def parallel_layer(heads, kv_heads, dim, vdim, chunk, scale, inner, state, dt_rank, conv, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        left["mask"] = {"size": chunk}
    return {"type": "parallel", "mixer": {"left": left, "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}, "mlp": mlp}


def rglru_layer(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def mamba2_layer(heads, vdim, state, groups, conv, parts, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": parts},
            "mlp": mlp}


def model(vocab, width, eps, layers, loop=None):
    cfg = {"architecture": "Fotanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: every mixer; recurrences wider and narrower than the model, chunks that are no multiple of a page, a loop of two
#    layers that runs three times behind a first layer, a layer without feed-forward, norm parts that cut through heads.
CONFIG_A = model(97, 64, 1e-5, [
    rglru_layer(48, 3, 4, moe(6, 2, 20)),
    parallel_layer(4, 2, 16, 8, 37, 0.4, 40, 6, 5, 3, moe(5, 1, 24)),
    mamba2_layer(6, 8, 10, 3, 2, 4, None),
    parallel_layer(2, 1, 8, 12, 100, 0.5, 72, 18, 4, 4, moe(4, 3, 16)),
], loop=(1, 3, 3))
# B: sizes that are no multiples of 8, one head, as many key heads as heads, no chunks at all and chunks of three, one
#    state, one tap, one block, one group, one part, one expert, every expert chosen; no loop.
CONFIG_B = model(131, 50, 2e-6, [
    mamba2_layer(1, 14, 7, 1, 1, 1, moe(1, 1, 10)),
    parallel_layer(3, 3, 6, 10, None, 0.6, 22, 1, 1, 1, moe(3, 3, 14)),
    rglru_layer(34, 1, 1, None),
    parallel_layer(1, 1, 10, 6, 3, 0.8, 30, 33, 9, 5, None),
    mamba2_layer(5, 6, 3, 5, 6, 15, moe(7, 2, 6)),
])
# C: sizes that the tensor-core kernels take, chunks of one page and of two, a loop over all layers that runs twice.
CONFIG_C = model(160, 128, 1e-6, [
    parallel_layer(8, 2, 32, 64, 64, 0.25, 128, 16, 8, 4, moe(8, 2, 48)),
    mamba2_layer(8, 32, 64, 2, 4, 4, moe(8, 4, 32)),
    rglru_layer(192, 6, 4, moe(16, 3, 16)),
    parallel_layer(4, 4, 64, 32, 128, 0.15, 256, 8, 16, 2, None),
], loop=(0, 4, 2))
# D: a loop over the last layers that runs once, and no feed-forward anywhere: every step can be captured.
CONFIG_D = model(80, 48, 1e-5, [
    mamba2_layer(4, 16, 16, 1, 3, 2, None),
    parallel_layer(4, 1, 16, 16, 50, 0.4, 64, 4, 8, 3, None),
    rglru_layer(48, 2, 2, None),
], loop=(1, 3, 1))
# E: wider, for long requests: five query heads to a key head, chunks that span several pages and are no multiple of one,
#    long enough prompts for the scans' chunks.
CONFIG_E = model(400, 256, 1e-6, [
    mamba2_layer(6, 64, 96, 3, 4, 3, moe(10, 3, 64)),
    parallel_layer(10, 2, 48, 80, 230, 0.2, 384, 32, 24, 3, moe(6, 2, 80)),
    rglru_layer(320, 5, 4, None),
], loop=(0, 2, 2))
# single mixers: one layer each, no feed-forward; and the experts alone
CONFIG_P = model(64, 48, 1e-5, [parallel_layer(4, 2, 8, 16, 23, 0.6, 32, 8, 4, 4, None)])
CONFIG_R = model(64, 48, 1e-5, [rglru_layer(64, 4, 4, None)])
CONFIG_S = model(64, 48, 1e-5, [mamba2_layer(3, 16, 12, 1, 3, 1, None)])
CONFIG_M = model(64, 48, 1e-5, [rglru_layer(16, 2, 2, moe(10, 3, 12))])
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E, "P": CONFIG_P, "R": CONFIG_R, "S": CONFIG_S, "M": CONFIG_M}


def inverse_softplus(y):
    return np.log(np.expm1(y))


def make_weights(cfg: dict, seed: int, gain_all: float = 1.0) -> dict[str, np.ndarray]:
    """float32 arrays by checkpoint name; the caller rounds them to the stored type.  `gain_all` scales every matrix."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(n_out, n_in, gain=1.0):
        return rng.normal(0.0, gain_all * gain / np.sqrt(n_in), size=(n_out, n_in))

    def around_one(n):
        return 1.0 + rng.normal(0, 0.2, n)

    w = {"embed": rng.normal(0, 1.0, (V, D)), "head": mat(V, D, 1.5)}

    def tanh_norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = around_one(D), rng.normal(0, 0.1, D), rng.uniform(0.4, 0.9)

    def conv(p, channels, taps):
        w[p + "conv"], w[p + "conv.b"] = rng.normal(0, 0.8 / np.sqrt(taps), (channels, taps)), rng.normal(0, 0.2, channels)

    tanh_norm("final.norm")
    if cfg.get("loop"):
        w["loop.in"], w["loop.step"] = mat(D, 2 * D, 1.4), rng.normal(0, 0.5, (cfg["loop"]["times"], D))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        tanh_norm(f"l{i}.norm1")
        if layer["type"] == "parallel":
            a, r = m["left"], m["right"]
            H, G, d, dv, q = a["heads"], a["kv_heads"], a["dim"], a["vdim"], p + "left."
            w[q + "q"], w[q + "k"], w[q + "v"] = mat(H * d, D, 2.5), mat(G * d, D, 2.5), mat(G * dv, D, 1.5)
            w[q + "sink"], w[q + "g"], w[q + "o"], w[q + "out"] = rng.normal(0, 1.5, H), mat(H, D, 2.0), mat(D, H * dv, 1.5), around_one(D)
            n, N, R, q = r["inner"], r["state"], r["dt_rank"], p + "right."
            w[q + "in"], w[q + "x"], w[q + "o"], w[q + "out"] = mat(2 * n, D, 1.5), mat(R + 2 * N, n, 2.0), mat(D, n, 1.5), around_one(D)
            conv(q, n, r["conv"])
            w[q + "dt"], w[q + "dt.b"] = mat(n, R, 1.0), inverse_softplus(np.exp(rng.uniform(np.log(0.003), np.log(0.5), n)))
            w[q + "A_log"], w[q + "D"] = np.log(rng.uniform(0.05, 4.0, (n, N))), around_one(n)
        elif layer["type"] == "rglru":
            n, nb = m["width"], m["blocks"]
            k = n // nb
            for name in ("y", "x"):
                w[p + name], w[p + name + ".b"] = mat(n, D, 1.5), rng.normal(0, 0.2, n)
            conv(p, n, m["conv"])
            for name in ("ra", "ri"):
                w[p + name], w[p + name + ".b"] = rng.normal(0, gain_all * 1.5 / np.sqrt(k), (nb, k, k)), rng.normal(0, 0.5, (nb, k))
            w[p + "lam"] = inverse_softplus(np.exp(rng.uniform(np.log(3e-4), np.log(0.5), n)))
            w[p + "o"] = mat(D, n, 2.0)
        else:
            H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            n = H * dv
            w[p + "in"], w[p + "o"], w[p + "norm"] = mat(2 * n + 2 * G * N + H, D, 1.5), mat(D, n, 1.5), around_one(n)
            conv(p, n + 2 * G * N, m["conv"])
            w[p + "dt_bias"] = inverse_softplus(np.exp(rng.uniform(np.log(0.003), np.log(0.5), H)))
            w[p + "A_log"], w[p + "D"] = np.log(rng.uniform(0.1, 2.0, H)), around_one(H)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        tanh_norm(f"l{i}.norm2")
        q, F = f"l{i}.mlp.", mlp["expert"]["ff"]
        w[q + "router"] = mat(mlp["router"]["experts"], D, 3.0)
        for e in range(mlp["router"]["experts"]):
            w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = mat(F, D, 2.0), mat(F, D, 2.0), mat(D, F, 1.5)
    return {k: np.asarray(v, dtype=np.float32) for k, v in w.items()}


def write_folder(folder, cfg: dict, weights: dict, dtype: str):
    """config.json + model.safetensors with the weights rounded to `dtype`."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    dt = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype]
    write_safetensors(folder / "model.safetensors", {k: torch.from_numpy(np.array(v, dtype=np.float32)).to(dt) for k, v in weights.items()})
    return folder


def make_folder(tmp_path, which: str, dtype: str, seed: int = 0):
    cfg = CONFIGS[which]
    weights = make_weights(cfg, seed + sorted(CONFIGS).index(which), gain_all=1.0 if dtype == "float32" else 0.5)
    return write_folder(tmp_path / f"fotanex_{which}_{dtype}", cfg, weights, dtype), cfg


def load_plain(folder):
    """(config dict, {name: float64 array}) of a folder, as the plain model takes them: the stored values exactly."""
    cfg = json.loads((folder / "config.json").read_text())
    f = SafetensorsFile(folder / "model.safetensors")
    try:
        w = {name: f.read(name).to(torch.float64).numpy().copy() for name in f.names()}
    finally:
        f.close()
    return cfg, w


def logits_error(got, ref):
    """Per row: the root mean square of the difference (means taken off) over that of the reference."""
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert np.isfinite(got).all()
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    r = ref - ref.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((r * r).mean(-1))


# float32: rounding of 32-bit sums and exponentials only (typical rows are off by 1e-6); a structural fault moves the
# rows it touches by 3e-2 at least.  bfloat16 (with the gentler weights): a row may be off by a quarter of its spread, a
# request's rows (where there are enough of them for a median to mean something) by 5 % in the median.  A router that
# meets two nearly equal scores may pick the other expert in bfloat16, and the rows behind it read what that row left: one
# row in twenty, and always one, may therefore be off by more.  A fault of a bfloat16 kernel moves the median; a fault of
# the structure fails the float32 runs of the same tests.
F32_LIMIT = 1e-3
BF16_ROW_LIMIT, BF16_MEDIAN_LIMIT, BF16_ROWS_BEYOND = 2.5e-1, 5e-2, 0.05


def assert_close(got, ref, dtype, what=""):
    e = logits_error(got, ref)
    if dtype == "float32":
        assert e.max() <= F32_LIMIT, f"{what}: error {e.max():.3e} of the logits' spread at row {int(e.argmax())} (limit {F32_LIMIT})"
        return
    beyond = int((e > BF16_ROW_LIMIT).sum())
    assert beyond <= max(1, int(BF16_ROWS_BEYOND * len(e))), \
        f"{what}: {beyond} of {len(e)} rows beyond {BF16_ROW_LIMIT} of the logits' spread, the worst {e.max():.3e} at row {int(e.argmax())}"
    if len(e) >= 16:
        assert np.median(e) <= BF16_MEDIAN_LIMIT, f"{what}: median error {np.median(e):.3e} of the logits' spread"
