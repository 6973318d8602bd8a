"""Fotanex's configuration, read from its own config.json keys.

A Fotanex model lists its layers: `layers[i]` names the layer's mixer (`type`: "parallel", "rglru" or "mamba2"), the
mixer's sizes and constants (`mixer`), and its feed-forward (`mlp`: {"kind": "moe", "expert": {"ff"}, "router":
{"experts", "top"}} or null).  Around them: `vocab`, `width`, `norm.eps`, and `loop` {"start", "stop", "times"} (absent:
no loop): layers start .. stop - 1 run `times` times in a row with the same weights and a cache of their own per pass, each
pass entered through W_in [x; embedding output] and a vector per pass.  Every size and constant comes from these keys.
Mixer and feed-forward read the same x through a dynamic tanh each and are added to the 32-bit stream together; the head
has a matrix of its own.  The model names no longest sequence; `max_positions` (the library's own key, default 32,768)
bounds the engine's context only: positions enter no layer but through the chunks.

Mixers:
  "parallel": `left`, grouped softmax attention without positions inside chunks of `mask.size` positions (absent or 0: all
      keys), `scale` on the scores, a sink per head, a sigmoid gate per head; beside `right`, Mamba (`inner`, `state`,
      `dt_rank`, `conv` taps); half the sum of the two results, each under an RMS norm of its own.
  "rglru": Griffin's recurrent block (`width` channels in `blocks` blocks, `conv` taps).
  "mamba2": Mamba-2 (`heads`, `vdim`, `state`, `groups`, `norm_groups`, `conv` taps).

Tensor names: `embed`, `loop.in`, `loop.step`, `l<i>.norm1|norm2` (and `.alpha`, `.b`), `l<i>.mix.<name>`
(`l<i>.mix.left|right.<name>`), `l<i>.mlp.router`, `l<i>.mlp.e<j>.gate|up|down`, `final.norm`, `head`; linear weights are
[out, in].
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional

from ..errors import QsError
from .lutelorn import _bad, _get, _positive_int
from .specs import (AttentionSpec, BlockSpec, HeadSpec, LayerRun, LoopEntrySpec, Mamba2Spec, MambaSpec, ModelSpec,
                    PairEmbeddingSpec, PairMixerSpec, RgLruSpec, RoutedExpertsSpec, TanhNormSpec)

MIXERS = ("parallel", "rglru", "mamba2")
DEFAULT_MAX_POSITIONS = 32768
# fixed by the design
PAIR_SCALE = 0.5            # the weight of each of two mixers side by side
RENORM_EPS = 1e-20          # added to the sum that the chosen experts' scores are divided by


def _number(d, key, what):
    return float(_get(d, key, what, (int, float)))


@dataclass(frozen=True)
class FotanexConfig:
    vocab: int
    width: int
    layers: tuple                       # the config's own layer objects (dicts), checked
    eps: float
    loop: Optional[tuple] = None        # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Fotanex"
    model_type = "fotanex"

    # ----------------------------------------------------------------- reading
    @classmethod
    def from_dict(cls, d: dict) -> "FotanexConfig":
        layers = _get(d, "layers", "config", list)
        if not layers:
            raise _bad("'layers' is empty")
        loop = _get(d, "loop", "config", dict, optional=True)
        if loop is not None:
            loop = tuple(_get(loop, key, "loop", int) for key in ("start", "stop", "times"))
        cfg = cls(vocab=_positive_int(d, "vocab", "config"), width=_positive_int(d, "width", "config"),
                  layers=tuple(copy.deepcopy(layer) for layer in layers), eps=_number(_get(d, "norm", "config", dict), "eps", "norm"),
                  loop=loop,
                  max_positions=_positive_int(d, "max_positions", "config", optional=True, default=DEFAULT_MAX_POSITIONS))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if not self.eps > 0:
            raise _bad(f"norm.eps={self.eps} must be positive")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise _bad(f"loop: start={start}, stop={stop}, times={times} with {len(self.layers)} layers")
        for i, layer in enumerate(self.layers):
            what = f"layers[{i}]"
            kind = _get(layer, "type", what, str)
            if kind not in MIXERS:
                raise _bad(f"{what}.type '{kind}' is not one of {MIXERS}", QsError.UNSUPPORTED_ARCH)
            m = _get(layer, "mixer", what, dict)
            what += ".mixer"
            if kind == "parallel":
                left, right = _get(m, "left", what, dict), _get(m, "right", what, dict)
                heads, dim = _positive_int(left, "heads", what + ".left"), _positive_int(left, "dim", what + ".left")
                kv = _positive_int(left, "kv_heads", what + ".left", optional=True, default=heads)
                _positive_int(left, "vdim", what + ".left", optional=True, default=dim)
                if heads % kv:
                    raise _bad(f"{what}.left: {heads} heads are no multiple of {kv} kv_heads")
                _number(left, "scale", what + ".left")
                if self._chunk(left, what + ".left") < 0:
                    raise _bad(f"{what}.left.mask.size must not be negative")
                for key in ("inner", "state", "dt_rank", "conv"):
                    _positive_int(right, key, what + ".right")
            elif kind == "rglru":
                n, blocks = _positive_int(m, "width", what), _positive_int(m, "blocks", what)
                _positive_int(m, "conv", what)
                if n % blocks:
                    raise _bad(f"{what}: width={n} is no multiple of blocks={blocks}")
            else:
                heads, vdim, _, groups, _, parts = (_positive_int(m, key, what) for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
                if heads % groups or (heads * vdim) % parts:
                    raise _bad(f"{what}: {heads} heads of {vdim} in groups={groups} and norm_groups={parts}")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            what = f"layers[{i}].mlp"
            if _get(mlp, "kind", what, str) != "moe":
                raise _bad(f"{what}.kind '{mlp['kind']}' is not 'moe'", QsError.UNSUPPORTED_ARCH)
            _positive_int(_get(mlp, "expert", what, dict), "ff", what + ".expert")
            r = _get(mlp, "router", what, dict)
            E, top = _positive_int(r, "experts", what + ".router"), _positive_int(r, "top", what + ".router")
            if top > E:
                raise _bad(f"{what}.router: top={top} of {E} experts")

    @staticmethod
    def _chunk(left: dict, what: str) -> int:
        mask = _get(left, "mask", what, dict, optional=True, default={})
        return _get(mask, "size", what + ".mask", int, optional=True, default=0)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "model_type": self.model_type, "vocab": self.vocab, "width": self.width,
             "layers": [copy.deepcopy(layer) for layer in self.layers], "norm": {"eps": self.eps}, "max_positions": self.max_positions}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    # ----------------------------------------------------------------- the model
    def _norm(self, name: str) -> TanhNormSpec:
        return TanhNormSpec(self.width, names={"weight": name, "shift": name + ".b", "alpha": name + ".alpha"})

    def _mixer_spec(self, i: int, kind: str, m: dict):
        D, p = self.width, f"l{i}.mix."
        if kind == "parallel":
            left, right = m["left"], m["right"]
            heads, dim = left["heads"], left["dim"]
            names = {n: f"{p}left.{n}" for n in ("q", "k", "v", "sink")}
            names.update({"gate": p + "left.g", "out": p + "left.o"})
            chunked = AttentionSpec(width=D, n_heads=heads, n_kv_heads=left.get("kv_heads", heads), head_dim=dim,
                                    v_head_dim=left.get("vdim", dim), score_scale=float(left["scale"]),
                                    chunk=self._chunk(left, "mixer.left"), sink=True, gate="head", names=names)
            names = {n: f"{p}right.{n}" for n in ("in", "conv", "x", "dt", "A_log", "D", "o")}
            names.update({"conv_bias": p + "right.conv.b", "dt_bias": p + "right.dt.b"})
            scan = MambaSpec(width=D, inner=right["inner"], state=right["state"], dt_rank=right["dt_rank"], conv_taps=right["conv"], names=names)
            return PairMixerSpec(left=chunked, right=scan, left_scale=PAIR_SCALE, right_scale=PAIR_SCALE, width=D, eps=self.eps,
                                 norm_names=(p + "left.out", p + "right.out"))
        if kind == "rglru":
            names = {n: p + n for n in ("y", "x", "conv", "lam", "o")}
            names.update({"y_bias": p + "y.b", "x_bias": p + "x.b", "conv_bias": p + "conv.b", "r": p + "ra", "r_bias": p + "ra.b",
                          "i": p + "ri", "i_bias": p + "ri.b"})
            return RgLruSpec(width=D, inner=m["width"], blocks=m["blocks"], conv_taps=m["conv"], names=names)
        names = {n: p + n for n in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
        names["conv_bias"] = p + "conv.b"
        return Mamba2Spec(width=D, n_heads=m["heads"], value_dim=m["vdim"], state=m["state"], groups=m["groups"], conv_taps=m["conv"],
                          norm_parts=m["norm_groups"], eps=self.eps, names=names)

    def _ffn_spec(self, i: int, mlp: dict):
        p, r = f"l{i}.mlp.", mlp["router"]
        names = {"router": p + "router"}
        for e in range(r["experts"]):
            names.update({f"{n}{e}": f"{p}e{e}.{n}" for n in ("gate", "up", "down")})
        return RoutedExpertsSpec(width=self.width, n_experts=r["experts"], inner=mlp["expert"]["ff"], top=r["top"], activation="silu",
                                 scores="softmax", group_score="max", correction=False, shared_gate=False, gated="act",
                                 normalize=True, normalize_eps=RENORM_EPS, names=names)

    def model_spec(self) -> ModelSpec:
        D = self.width
        blocks = []
        for i, layer in enumerate(self.layers):
            norms, ffn = {"input": self._norm(f"l{i}.norm1")}, None
            if layer.get("mlp") is not None:
                norms["ffn_input"], ffn = self._norm(f"l{i}.norm2"), self._ffn_spec(i, layer["mlp"])
            blocks.append(BlockSpec(arrangement="twin_norm", norms=norms, ffn=ffn, mixer=self._mixer_spec(i, layer["type"], layer["mixer"])))
        start, stop, times = self.loop or (0, 0, 0)
        runs = [(i, None) for i in range(start)]
        runs += [(i, (0, t) if i == start else None) for t in range(times) for i in range(start, stop)]
        runs += [(i, None) for i in range(stop, len(self.layers))]
        schedule, entry = [], 0
        for i, enter in runs:                           # every run keeps what it keeps for itself, each pass of the loop too
            if self.layers[i]["type"] == "parallel":    # two parts that keep something: an entry each
                schedule.append(LayerRun(layer=i, cache=(entry, entry + 1), enter=enter))
                entry += 2
            else:
                schedule.append(LayerRun(layer=i, cache=entry, enter=enter))
                entry += 1
        joints = (LoopEntrySpec(width=D, times=times, names={"in": "loop.in", "step": "loop.step"}),) if self.loop else ()
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, width=D, max_positions=self.max_positions,
            embedding=PairEmbeddingSpec(vocab_size=self.vocab, width=D, stream_dtype="float32", names={"weight": "embed"}),
            layers=tuple(blocks), schedule=tuple(schedule), joints=joints, final_norm=self._norm("final.norm"),
            head=HeadSpec(vocab_size=self.vocab, width=D, bias=False, tied=False, names={"weight": "head"}),
        )
