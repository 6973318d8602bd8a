"""Small Vofinex models for the tests: configurations that differ in every size and option, and weights drawn here
with numpy so that every mechanism carries weight in the logits (scores of several units, sinks of the order of the scores,
routers far from uniform whose corrections change the choice, experts that return their input among the chosen)."""
from __future__ import annotations

import json

import numpy as np
import torch

from qstream_b200.weights.safetensors_io import SafetensorsFile, write_safetensors


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff):
    router = {"experts": experts, "top": top}
    if identity is not None:
        router["identity"] = identity
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def layer(heads, kv_heads, dim, vdim, chunk, scale, rot=None, mlp=None):
    m = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if vdim is not None:
        m["vdim"] = vdim
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def model(vocab, width, eps, layers, loop=None, scale=3.0, mult=0.7, logit_scale=1.7):
    cfg = {"architecture": "Vofinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "residual_mult": mult, "logit_scale": logit_scale, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# A: heads, key heads, values, chunks, rotations and feed-forwards that differ from layer to layer, chunks that are no multiple
#    of a page, a loop of two layers that runs three times behind a first layer, a layer without feed-forward.
CONFIG_A = model(97, 64, 1e-5, [
    layer(4, 2, 16, 8, 37, 0.4, (8, 1e4), dense(72)),
    layer(2, 1, 8, 12, 100, 0.6, (8, 500.0), moe(6, 2, 3, 20)),
    layer(6, 3, 12, 20, 23, 0.5, (4, 3e5), None),
    layer(3, 1, 24, 16, 64, 0.3, (16, 1e3), moe(3, 5, 2, 24)),
], loop=(1, 3, 3))
# B: sizes that are no multiples of 8, one head, as many key heads as heads, no chunks at all and chunks of three, no rotation, one
#    expert, no identity outputs, every output chosen, more identity outputs than experts, constants of one; no loop.
CONFIG_B = model(131, 50, 2e-6, [
    layer(1, None, 14, None, None, 0.5, None, moe(1, 0, 1, 10)),
    layer(3, 3, 6, 10, 3, 0.9, (6, 77.0), moe(2, 3, 5, 14)),
    layer(5, 1, 10, 6, 50, 0.7, (2, 1e4), dense(33)),
    layer(2, 2, 18, 7, 1, 0.5, (0, 1e4), moe(4, None, 2, 6)),
], scale=1.0, mult=1.0, logit_scale=1.0)
# C: sizes that the tensor-core kernels take, chunks of one page and of two, a loop over all layers that runs twice.
CONFIG_C = model(160, 128, 1e-6, [
    layer(8, 2, 32, 64, 64, 0.25, (32, 1e4), dense(192)),
    layer(4, 4, 64, 32, 128, 0.15, (16, 2e4), moe(8, 4, 4, 48)),
    layer(6, 2, 48, 16, 90, 0.2, (48, 1e5), moe(16, 1, 3, 16)),
], loop=(0, 3, 2), scale=5.0, mult=0.5, logit_scale=0.8)
# D: no experts anywhere, so that every step can be captured; a loop over the last layers that runs once.
CONFIG_D = model(80, 48, 1e-5, [
    layer(4, 1, 16, 16, 50, 0.4, (16, 1e4), dense(40)),
    layer(2, 2, 32, 24, 40, 0.3, (32, 1e4), None),
    layer(4, 2, 16, 8, None, 0.4, (8, 1e4), dense(64)),
], loop=(1, 3, 1), mult=-0.6)
# E: wider, for long requests: five query heads to a key head, chunks that span several pages and are no multiple of one.
CONFIG_E = model(400, 320, 1e-6, [
    layer(10, 2, 48, 80, 230, 0.25, (32, 1e5), moe(6, 3, 2, 80)),
    layer(4, 1, 128, 128, 500, 0.1, (64, 1e6), dense(512)),
    layer(5, 5, 96, 32, 333, 0.12, (16, 1e4), moe(10, 2, 4, 64)),
], loop=(0, 2, 2), scale=8.0, mult=0.35)
# single mechanisms: attention alone; dense alone beside it; experts with a majority of identity outputs
CONFIG_P = model(64, 48, 1e-5, [layer(4, 2, 8, 16, 29, 0.8, (4, 1e3), None)])
CONFIG_F = model(64, 48, 1e-5, [layer(2, 1, 16, 8, None, 0.3, None, dense(64))])
CONFIG_M = model(64, 40, 1e-5, [layer(2, 1, 8, 8, 16, 0.3, (8, 1e4), moe(4, 6, 3, 12))])
CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D, "E": CONFIG_E, "P": CONFIG_P, "F": CONFIG_F, "M": CONFIG_M}


def make_weights(cfg: dict, seed: int, gain_all: float = 1.0) -> dict[str, np.ndarray]:
    """float32 arrays by checkpoint name; the caller rounds them to the stored type.  `gain_all` scales every matrix."""
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(n_out, n_in, gain=1.0):
        return rng.normal(0.0, gain_all * gain / np.sqrt(n_in), size=(n_out, n_in))

    w = {"embed": rng.normal(0, 0.4, (V, D))}

    def norm(name):
        w[name], w[name + ".b"] = 1.0 + rng.normal(0, 0.2, D), rng.normal(0, 0.2, D)

    norm("final.norm")
    if cfg.get("loop"):
        w["loop.step"] = rng.normal(0, 0.5, (cfg["loop"]["times"], D))
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", lay["mixer"]
        norm(f"l{i}.norm1")
        H, d = m["heads"], m["dim"]
        G, dv = m.get("kv_heads", H), m.get("vdim", d)
        w[p + "q"], w[p + "k"], w[p + "v"] = mat(H * d, D, 2.0), mat(G * d, D, 2.0), mat(G * dv, D, 1.5)
        w[p + "sink"], w[p + "o"] = rng.normal(1.0, 1.5, H), mat(D, H * dv, 2.0)
        mlp = lay.get("mlp")
        if mlp is None:
            continue
        q = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            w[q + "gate"], w[q + "up"], w[q + "down"] = mat(F, D, 1.5), mat(F, D, 1.5), mat(D, F, 1.5)
            continue
        r, F = mlp["router"], mlp["expert"]["ff"]
        outputs = r["experts"] + (r.get("identity") or 0)
        w[q + "router"], w[q + "correction"] = mat(outputs, D, 2.0), rng.normal(0, 0.15, outputs)
        for e in range(r["experts"]):
            w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = mat(F, D, 2.0), mat(F, D, 2.0), mat(D, F, 2.0)
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
    weights = make_weights(cfg, seed + sorted(CONFIGS).index(which), gain_all=1.0 if dtype == "float32" else 0.7)
    return write_folder(tmp_path / f"vofinex_{which}_{dtype}", cfg, weights, dtype), cfg


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
# rows it touches by 3e-2 at least.  bfloat16: a row may be off by a quarter of its spread, a request's rows (where there are
# enough of them for a median to mean something) by 5 % in the median.  A router that meets two nearly equal scores may pick the
# other expert in bfloat16, and the rows behind it read what that row left: one row in twenty, and always one, may
# therefore be off by more.  A fault of a bfloat16 kernel moves the median; a fault of the structure fails the float32
# runs of the same tests.
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
