"""Vofinex's configuration, read from its own config.json keys.

A Vofinex model lists its layers: `layers[i]` names the layer's mixer (`type`: "attention"), the mixer's sizes and constants
(`mixer`), and its feed-forward (`mlp`: {"kind": "dense", "ff": n}, {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top",
"identity"}}, or null).  Around them: `vocab`, `width`, `norm.eps`, `embedding.scale`, `residual_mult`, `logit_scale`, and `loop`
{"start", "stop", "times"} (absent: no loop): layers start .. stop - 1 run `times` times in a row with the same weights and a
cache of their own per pass, a vector per pass added to the stream before it.  Every size and constant comes from these keys.
Mixer and feed-forward read the same layer norm of the 32-bit stream; the sum of their results, times `residual_mult`, is added
to it; the head is the embedding table.  The model names no longest sequence; `max_positions` (the library's own key,
default 32,768) bounds the tables of rotation angles and the engine's context.

"attention": grouped softmax attention inside chunks of `mask.size` positions (absent or 0: all keys), rotate-half positions on the
first `rot.dims` dims of each head (absent: none), then a unit RMS per head of q and k, `scale` on the scores, a sink per head.
"moe": `experts` gated silu experts and `identity` more router outputs that return their input; softmax scores over all
of them, a correction that counts for the choice only, the chosen scores as weights.

Tensor names: `embed`, `loop.step`, `l<i>.norm1` (and `.b`), `l<i>.mix.q|k|v|o|sink`, `l<i>.mlp.gate|up|down`,
`l<i>.mlp.router|correction`, `l<i>.mlp.e<j>.gate|up|down`, `final.norm` (and `.b`); linear weights are [out, in].
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Optional

from ..errors import QsError
from .lutelorn import _bad, _get, _positive_int
from .specs import (AttentionSpec, BlockSpec, BranchSumNormSpec, GatedMlpSpec, HeadSpec, LayerRun, LoopStepSpec, ModelSpec,
                    PairEmbeddingSpec, PositionHalfSpec, RoutedExpertsSpec)

MIXERS = ("attention",)
DEFAULT_MAX_POSITIONS = 32768


def _number(d, key, what, optional=False, default=None):
    v = _get(d, key, what, (int, float), optional, default)
    return None if v is None else float(v)


def _rot(m: dict, what: str):
    """(rotated dims, base); (0, 1) without a rotation."""
    rot = _get(m, "rot", what, dict, optional=True)
    if rot is None:
        return 0, 1.0
    return _get(rot, "dims", what + ".rot", int), _number(rot, "base", what + ".rot")


def _chunk(m: dict, what: str) -> int:
    mask = _get(m, "mask", what, dict, optional=True) or {}
    return _get(mask, "size", what + ".mask", int, optional=True, default=0) or 0


def _identity(r: dict, what: str) -> int:
    return _get(r, "identity", what, int, optional=True, default=0) or 0


@dataclass(frozen=True)
class VofinexConfig:
    vocab: int
    width: int
    layers: tuple                       # the config's own layer objects (dicts), checked
    eps: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    loop: Optional[tuple] = None        # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS

    architecture = "Vofinex"
    model_type = "vofinex"

    # ----------------------------------------------------------------- reading
    @classmethod
    def from_dict(cls, d: dict) -> "VofinexConfig":
        layers = _get(d, "layers", "config", list)
        if not layers:
            raise _bad("'layers' is empty")
        loop = _get(d, "loop", "config", dict, optional=True)
        if loop is not None:
            loop = tuple(_get(loop, key, "loop", int) for key in ("start", "stop", "times"))
        emb = _get(d, "embedding", "config", dict, optional=True) or {}
        cfg = cls(vocab=_positive_int(d, "vocab", "config"), width=_positive_int(d, "width", "config"),
                  layers=tuple(copy.deepcopy(layer) for layer in layers), eps=_number(_get(d, "norm", "config", dict), "eps", "norm"),
                  embedding_scale=_number(emb, "scale", "embedding", optional=True, default=1.0),
                  residual_mult=_number(d, "residual_mult", "config", optional=True, default=1.0),
                  logit_scale=_number(d, "logit_scale", "config", optional=True, default=1.0), loop=loop,
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
            heads, dim = _positive_int(m, "heads", what), _positive_int(m, "dim", what)
            kv = _positive_int(m, "kv_heads", what, optional=True, default=heads)
            _positive_int(m, "vdim", what, optional=True, default=dim)
            if heads % kv:
                raise _bad(f"{what}: {heads} heads are no multiple of {kv} kv_heads")
            _number(m, "scale", what)
            dims, base = _rot(m, what)
            if dims < 0 or dims % 2 or dims > dim or not base > 0:
                raise _bad(f"{what}.rot: dims={dims} must be even and within dim={dim}, base={base} positive")
            if _chunk(m, what) < 0:
                raise _bad(f"{what}.mask.size must not be negative")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            what = f"layers[{i}].mlp"
            mk = _get(mlp, "kind", what, str)
            if mk == "dense":
                _positive_int(mlp, "ff", what)
            elif mk == "moe":
                _positive_int(_get(mlp, "expert", what, dict), "ff", what + ".expert")
                r = _get(mlp, "router", what, dict)
                E, top = _positive_int(r, "experts", what + ".router"), _positive_int(r, "top", what + ".router")
                same = _identity(r, what + ".router")
                if same < 0 or top > E + same:
                    raise _bad(f"{what}.router: top={top} of {E} experts and identity={same}")
            else:
                raise _bad(f"{what}.kind '{mk}' is not 'dense' or 'moe'", QsError.UNSUPPORTED_ARCH)

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "model_type": self.model_type, "vocab": self.vocab, "width": self.width,
             "layers": [copy.deepcopy(layer) for layer in self.layers], "norm": {"eps": self.eps}, "embedding": {"scale": self.embedding_scale},
             "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "max_positions": self.max_positions}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return d

    # ----------------------------------------------------------------- the model
    def _norm(self, name: str) -> BranchSumNormSpec:
        return BranchSumNormSpec(self.width, self.eps, center=True, bias=True, names={"weight": name, "bias": name + ".b"})

    def _mixer_spec(self, i: int, m: dict) -> AttentionSpec:
        p, heads, dim = f"l{i}.mix.", m["heads"], m["dim"]
        dims, base = _rot(m, "mixer")
        position = PositionHalfSpec(rotary_dim=dims, base=base, max_positions=self.max_positions) if dims else None
        names = {n: p + n for n in ("q", "k", "v", "sink")}
        names["out"] = p + "o"
        return AttentionSpec(width=self.width, n_heads=heads, n_kv_heads=m.get("kv_heads") or heads, head_dim=dim, v_head_dim=m.get("vdim") or dim,
                             position=position, score_scale=float(m["scale"]), chunk=_chunk(m, "mixer"), sink=True, qk_norm="head",
                             eps=self.eps, names=names)

    def _ffn_spec(self, i: int, mlp: dict):
        p = f"l{i}.mlp."
        if mlp["kind"] == "dense":
            return GatedMlpSpec(width=self.width, inner=mlp["ff"], activation="silu", names={n: p + n for n in ("gate", "up", "down")})
        r = mlp["router"]
        names = {"router": p + "router", "correction": p + "correction"}
        for e in range(r["experts"]):
            names.update({f"{n}{e}": f"{p}e{e}.{n}" for n in ("gate", "up", "down")})
        return RoutedExpertsSpec(width=self.width, n_experts=r["experts"], inner=mlp["expert"]["ff"], top=r["top"], activation="silu",
                                 scores="softmax", group_score="max", correction=True, shared_gate=False, gated="act",
                                 identity=_identity(r, "router"), names=names)

    def model_spec(self) -> ModelSpec:
        D = self.width
        blocks = [BlockSpec(arrangement="scaled_parallel", norms={"input": self._norm(f"l{i}.norm1")}, residual_scale=self.residual_mult,
                            mixer=self._mixer_spec(i, layer["mixer"]),
                            ffn=self._ffn_spec(i, layer["mlp"]) if layer.get("mlp") is not None else None)
                  for i, layer in enumerate(self.layers)]
        start, stop, times = self.loop or (0, 0, 0)
        runs = [(i, None) for i in range(start)]
        runs += [(i, (0, t) if i == start else None) for t in range(times) for i in range(start, stop)]
        runs += [(i, None) for i in range(stop, len(self.layers))]
        joints = (LoopStepSpec(width=D, times=times, names={"step": "loop.step"}),) if self.loop else ()
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, width=D, max_positions=self.max_positions,
            embedding=PairEmbeddingSpec(vocab_size=self.vocab, width=D, scale=self.embedding_scale, buckets=0, stream_dtype="float32",
                                        names={"weight": "embed"}),
            layers=tuple(blocks), joints=joints, final_norm=self._norm("final.norm"),
            # every run keeps keys and values of its own, each pass of the loop too
            schedule=tuple(LayerRun(layer=i, cache=n, enter=enter) for n, (i, enter) in enumerate(runs)),
            head=HeadSpec(vocab_size=self.vocab, width=D, bias=False, tied=True, scale=self.logit_scale, names={}),
        )
