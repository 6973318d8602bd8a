"""Vofinex's configuration: reading, validation, the model it describes; and the plain model's own pieces on inputs
whose results are known."""
import copy
import math

import numpy as np
import pytest

import qstream_b200 as qs
from qstream_b200.config.vofinex import VofinexConfig
from qstream_b200.engine.model import declared_tensors
from qstream_b200.errors import QStreamError

import plain_vofinex as P
from vofinex_util import CONFIGS, make_weights


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_the_declared_tensors_are_the_checkpoint_s(which):
    cfg = qs.config_from_dict(CONFIGS[which])
    assert isinstance(cfg, VofinexConfig)
    decl = declared_tensors(cfg.model_spec())
    weights = make_weights(CONFIGS[which], 0)
    assert set(decl) == set(weights)
    for name, d in decl.items():
        assert tuple(d.shape) == weights[name].shape, name
    assert qs.config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


def test_the_schedule_and_the_parts_follow_the_layers():
    spec = qs.config_from_dict(CONFIGS["A"]).model_spec()
    assert [r.layer for r in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [r.cache for r in spec.schedule] == list(range(8))                 # every pass keeps its own
    assert [r.enter for r in spec.schedule] == [None, (0, 0), None, (0, 1), None, (0, 2), None, None]
    assert (spec.joints[0].kind, spec.joints[0].times, spec.joints[0].width) == ("loop_step", 3, 64)
    assert [b.arrangement for b in spec.layers] == ["scaled_parallel"] * 4 and all(b.residual_scale == 0.7 for b in spec.layers)
    assert all(set(b.norms) == {"input"} and b.norms["input"].center and b.norms["input"].bias for b in spec.layers)
    m = spec.layers[3].mixer
    assert (m.n_heads, m.n_kv_heads, m.head_dim, m.value_dim, m.chunk, m.scale) == (3, 1, 24, 16, 64, 0.3)
    assert (m.sink, m.qk_norm, m.gate, m.eps, m.position.rotary_dim, m.position.base) == (True, "head", False, 1e-5, 16, 1e3)
    assert spec.layers[2].ffn is None and spec.layers[0].ffn.kind == "gated_mlp" and spec.layers[0].ffn.activation == "silu"
    e = spec.layers[3].ffn
    assert (e.n_experts, e.identity, e.top, e.inner, e.scores, e.gated, e.normalize, e.correction, e.shared_inner) == (3, 5, 2, 24, "softmax", "act", False, True, 0)
    assert spec.head.tied and spec.head.scale == 1.7 and spec.embedding.scale == 3.0 and spec.embedding.stream_dtype == "float32"


def test_what_the_file_leaves_out():
    spec = qs.config_from_dict(CONFIGS["B"]).model_spec()
    assert spec.joints == () and [r.layer for r in spec.schedule] == [0, 1, 2, 3] and all(r.enter is None for r in spec.schedule)
    m = spec.layers[0].mixer
    assert (m.n_kv_heads, m.value_dim, m.chunk, m.position) == (1, 14, 0, None)
    assert spec.layers[3].mixer.position is None and spec.layers[3].mixer.n_kv_heads == 2         # a rotation of no dims
    assert spec.layers[0].ffn.identity == 0 and spec.layers[3].ffn.identity == 0
    cfg = copy.deepcopy(CONFIGS["P"])
    for key in ("embedding", "residual_mult", "logit_scale"):
        cfg.pop(key)
    spec = qs.config_from_dict(cfg).model_spec()
    assert (spec.embedding.scale, spec.layers[0].residual_scale, spec.head.scale) == (1.0, 1.0, 1.0)
    spec = qs.config_from_dict(CONFIGS["D"]).model_spec()
    assert [r.enter for r in spec.schedule] == [None, (0, 0), None]           # a loop that runs once still enters its pass


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1), "mask"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=0), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "router"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "router"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_bad_configurations_are_refused(change, needle):
    cfg = copy.deepcopy(CONFIGS["A"])
    change(cfg)
    with pytest.raises(QStreamError) as e:
        qs.config_from_dict(cfg)
    assert needle in str(e.value)


def test_options_that_do_not_go_together_are_refused():
    from dataclasses import replace
    import torch
    from qstream_b200.parts import Runtime, part_class
    spec = qs.config_from_dict(CONFIGS["P"]).model_spec().layers[0].mixer
    rt = Runtime(dtype=torch.float32, device=torch.device("cpu"))
    cls = part_class("mixer", "attention")
    for bad in (replace(spec, value_mix="first"), replace(spec, maps=2), replace(spec, qk_norm="rows")):
        tensors = {n: torch.zeros(d.shape) for n, d in cls.declare(bad).items()}
        with pytest.raises(QStreamError):
            cls(bad, tensors, rt)


# ----------------------------------------------------------------------------- the plain model's pieces

def test_the_plain_rotation_turns_halves_and_leaves_the_rest():
    x = np.zeros((2, 1, 6))
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 2.0, 7.0
    out = P.rotate(x, [0, 3], 4, 100.0)
    np.testing.assert_allclose(out[0], x[0])
    # dims 0 and 2 turn by 3, dims 1 and 3 by 3 / 10; dims 4 and 5 stay
    np.testing.assert_allclose(out[1, 0], [math.cos(3), -2 * math.sin(0.3), math.sin(3), 2 * math.cos(0.3), 0.0, 7.0])


def test_the_plain_queries_are_normed_behind_the_rotation_over_the_whole_head():
    q = np.array([[[3.0, 0.0, 4.0, 12.0]]])
    m = {"rot": {"dims": 2, "base": 10.0}}
    got, _ = P.queries_and_keys(m, q, q, [1], 0.0)
    np.testing.assert_allclose(got[0, 0], np.array([3 * math.cos(1), 3 * math.sin(1), 4.0, 12.0]) / 6.5)
    got, _ = P.queries_and_keys({}, q, q, [1], 1.0)
    np.testing.assert_allclose(got[0, 0], q[0, 0] / math.sqrt(169 / 4 + 1))


def test_the_plain_layer_norm_has_a_bias():
    out = P.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 3.0]), np.array([0.5, -1.0]), 3.0)
    np.testing.assert_allclose(out, [[-2 / 2 + 0.5, 3 / 2 - 1.0]])            # mean 2, deviations -1 and 1, root of 1 + 3


def test_the_plain_router_s_correction_counts_for_the_choice_only():
    z = np.log(np.array([[0.1, 0.4, 0.2, 0.3]]))
    chosen, weights = P.route(z, np.array([0.0, 0.0, 0.3, 0.0]), 2)
    assert chosen.tolist() == [[2, 1]]
    np.testing.assert_allclose(weights, [[0.2, 0.4]])                         # as they are: not made to sum to one


def test_the_plain_identity_experts_return_the_input():
    rng = np.random.default_rng(0)
    D, F = 6, 4
    w = {"router": np.zeros((3, D)), "correction": np.array([0.0, 1.0, 2.0])}
    w.update({"e0.gate": rng.normal(size=(F, D)), "e0.up": rng.normal(size=(F, D)), "e0.down": rng.normal(size=(D, F))})
    h = rng.normal(size=(5, D))
    mlp = {"router": {"experts": 1, "identity": 2, "top": 2}}
    np.testing.assert_allclose(P.moe(mlp, w, "", h), 2 / 3 * h)
    w["correction"] = np.array([5.0, 1.0, 2.0])
    np.testing.assert_allclose(P.moe(mlp, w, "", h), (h + P.gated_unit(w, "e0.", h)) / 3)


def test_the_plain_chunks_end_where_the_next_begins():
    """Values are one-hot in the position, all scores equal, sinks far below: each row is the mean over its chunk so far."""
    T = 7
    w = {"q": np.zeros((1, T)), "k": np.zeros((1, T)), "v": np.eye(T), "o": np.eye(T), "sink": np.array([-80.0])}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": T, "scale": 1.0, "mask": {"size": 3}}
    out = P.attention(m, w, "", np.eye(T), 1e-5)
    want = np.zeros((T, T))
    for i in range(T):
        first = i // 3 * 3
        want[i, first:i + 1] = 1.0 / (i - first + 1)
    np.testing.assert_allclose(out, want, atol=1e-12)
    w["sink"] = np.array([0.0])                              # a sink as large as the scores: one more term in the sum
    np.testing.assert_allclose(P.attention(m, w, "", np.eye(T), 1e-5)[3:5, 3:5], [[0.5, 0.0], [1 / 3, 1 / 3]], atol=1e-12)


def test_the_plain_model_scales_stream_branches_and_logits():
    """No mixer output, no feed-forward: the stream is the scaled embedding plus the passes' vectors."""
    cfg = copy.deepcopy(CONFIGS["P"])
    cfg["loop"] = {"start": 0, "stop": 1, "times": 2}
    w = {k: v.astype(np.float64) for k, v in make_weights(cfg, 1).items()}
    w["l0.mix.o"] *= 0
    toks = [5, 9, 5]
    logits, after = P.forward(cfg, w, toks, want_layers=True)
    x = w["embed"][toks] * 3.0 + w["loop.step"].sum(0)
    np.testing.assert_allclose(after[-1], x)
    np.testing.assert_allclose(logits, P.layer_norm(x, w["final.norm"], w["final.norm.b"], 1e-5) @ w["embed"].T * 1.7)
