"""Fotanex's configuration: reading, validation, the model it describes; and the plain model's own pieces on inputs
whose results are known."""
import copy
import math

import numpy as np
import pytest

import qstream_b200 as qs
from qstream_b200.config.fotanex import FotanexConfig
from qstream_b200.engine.model import declared_tensors
from qstream_b200.errors import QStreamError

import plain_fotanex as P
from fotanex_util import CONFIGS, make_weights


@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_the_declared_tensors_are_the_checkpoint_s(which):
    cfg = qs.config_from_dict(CONFIGS[which])
    assert isinstance(cfg, FotanexConfig)
    decl = declared_tensors(cfg.model_spec())
    weights = make_weights(CONFIGS[which], 0)
    assert set(decl) == set(weights)
    for name, d in decl.items():
        assert tuple(d.shape) == weights[name].shape, name
    assert qs.config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()


def test_the_schedule_and_the_parts_follow_the_layers():
    spec = qs.config_from_dict(CONFIGS["A"]).model_spec()
    assert [r.layer for r in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [r.cache for r in spec.schedule] == [0, (1, 2), 3, (4, 5), 6, (7, 8), 9, (10, 11)]      # every pass keeps its own
    assert [r.enter for r in spec.schedule] == [None, (0, 0), None, (0, 1), None, (0, 2), None, None]
    assert (spec.joints[0].times, spec.joints[0].width) == (3, 64)
    assert [b.arrangement for b in spec.layers] == ["twin_norm"] * 4
    assert set(spec.layers[2].norms) == {"input"} and spec.layers[2].ffn is None
    assert set(spec.layers[0].norms) == {"input", "ffn_input"} and not spec.head.tied
    lru, pair, ssd = (spec.layers[i].mixer for i in range(3))
    assert (lru.kind, lru.inner, lru.blocks, lru.conv_taps) == ("rglru", 48, 3, 4)
    assert (ssd.kind, ssd.inner, ssd.groups, ssd.norm_parts) == ("mamba2", 48, 3, 4)
    assert (pair.left_scale, pair.right_scale, pair.eps) == (0.5, 0.5, 1e-5)
    assert (pair.left.chunk, pair.left.gate, pair.left.sink, pair.left.position, pair.left.value_dim) == (37, "head", True, None, 8)
    assert (pair.right.inner, pair.right.state, pair.right.dt_rank, pair.right.conv_taps) == (40, 6, 5, 3)
    experts = spec.layers[3].ffn
    assert (experts.scores, experts.gated, experts.normalize, experts.top, experts.inner) == ("softmax", "act", True, 3, 16)


def test_without_a_loop_there_is_no_joint_and_every_layer_runs_once():
    spec = qs.config_from_dict(CONFIGS["B"]).model_spec()
    assert spec.joints == () and [r.layer for r in spec.schedule] == [0, 1, 2, 3, 4]
    assert all(r.enter is None for r in spec.schedule)
    assert spec.layers[1].mixer.left.chunk == 0
    spec = qs.config_from_dict(CONFIGS["D"]).model_spec()
    assert [r.enter for r in spec.schedule] == [None, (0, 0), None]           # a loop that runs once still enters its pass


@pytest.mark.parametrize("change,needle", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=-1), "mask"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(dt_rank=0), "dt_rank"),
    (lambda c: c["layers"][0]["mixer"].update(blocks=5), "blocks"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][2]["mixer"].update(groups=4), "groups"),
    (lambda c: c["layers"][2]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "router"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_bad_configurations_are_refused(change, needle):
    cfg = copy.deepcopy(CONFIGS["A"])
    change(cfg)
    with pytest.raises(QStreamError) as e:
        qs.config_from_dict(cfg)
    assert needle in str(e.value)


def test_a_joint_that_no_model_has_is_refused():
    from dataclasses import replace
    spec = qs.config_from_dict(CONFIGS["D"]).model_spec()
    spec = replace(spec, schedule=(replace(spec.schedule[0], enter=(1, 0)), *spec.schedule[1:]))
    with pytest.raises(QStreamError, match="joint"):
        qs.CausalLM(spec, _zeros(spec), "float32", "cpu")


def _zeros(spec):
    import torch
    return {name: torch.zeros(d.shape) for name, d in declared_tensors(spec).items()}


# ----------------------------------------------------------------------------- the plain model's pieces

def test_the_plain_convolution_weighs_the_current_token_with_the_last_tap():
    x = np.array([[1.0], [10.0], [100.0], [1000.0]])
    out = P.causal_conv(x, np.array([[3.0, 2.0, 1.0]]), np.array([0.5]))
    np.testing.assert_allclose(out[:, 0], [1.5, 12.5, 123.5, 1230.5])          # current + 2 previous + 3 the one before
    np.testing.assert_allclose(P.causal_conv(x, np.array([[7.0]]), np.array([0.0]))[:, 0], 7.0 * x[:, 0])


def test_the_plain_tanh_norm_has_no_statistics():
    x = np.array([[0.0, 1.0, -50.0]])
    np.testing.assert_allclose(P.tanh_norm(x, 2.0, np.array([1.0, 3.0, 5.0]), np.array([0.5, 0.0, 1.0])),
                               [[0.5, 3.0 * math.tanh(2.0), -4.0]])


def test_the_plain_recurrences_on_hand_made_cases():
    """Two tokens each, by hand."""
    # selective scan: one channel, two states, one of which forgets nothing and one almost everything
    y, S = P.selective_walk(np.array([[2.0], [3.0]]), np.array([[0.5], [1.0]]), np.array([[-1e-12, -50.0]]),
                            np.array([[1.0, 1.0], [2.0, 4.0]]), np.array([[1.0, 0.0], [1.0, 1.0]]), np.array([10.0]), np.zeros((1, 2)))
    np.testing.assert_allclose(y[:, 0], [1.0 + 20.0, (1.0 + 6.0) + 12.0 + 30.0])
    np.testing.assert_allclose(S, [[7.0, 12.0]])
    # the gated unit: r = 1 and softplus(lam) = ln(2) / 8 halve the state; sqrt(1 - 1/4) scales what comes in
    lam = P.softplus(0.0) * 0 + math.log(math.expm1(math.log(2.0) / 8.0))
    out, S = P.gated_lru_walk(np.array([[4.0], [2.0]]), np.ones((2, 1)), np.ones((2, 1)), np.array([lam]), np.zeros(1))
    c = math.sqrt(0.75)
    np.testing.assert_allclose(out[:, 0], [4.0 * c, 2.0 * c + 2.0 * c])
    # the state-space dual form: one head, one state, a value of two
    y, S = P.ssd_walk(np.array([[[1.0, 2.0]], [[3.0, 5.0]]]), np.array([[0.5], [math.log(2.0)]]), np.array([-1.0]),
                      np.array([[[2.0]], [[1.0]]]), np.array([[[1.0]], [[10.0]]]), np.zeros((1, 1, 2)))
    np.testing.assert_allclose(y[0, 0], [1.0, 2.0])
    np.testing.assert_allclose(y[1, 0], [10 * (0.5 + 3 * math.log(2.0)), 10 * (1.0 + 5 * math.log(2.0))])


def test_the_plain_gate_comes_before_the_norm_of_each_part():
    y, z = np.array([[3.0, 4.0, 6.0, 8.0]]), np.array([[0.0, 50.0, 50.0, 50.0]])
    out = P.gate_then_group_norm(y, z, np.ones(4), 2, 0.0)
    np.testing.assert_allclose(out, [[0.0, math.sqrt(2.0), 0.6 * math.sqrt(2.0), 0.8 * math.sqrt(2.0)]])


def test_the_plain_router_makes_the_chosen_scores_sum_to_one():
    z = np.log(np.array([[0.1, 0.4, 0.2, 0.3]]))
    chosen, weights = P.route(z, 2)
    assert chosen.tolist() == [[1, 3]]
    np.testing.assert_allclose(weights, [[4 / 7, 3 / 7]])
    chosen, weights = P.route(z, 1)
    np.testing.assert_allclose(weights, [[1.0]])


def test_the_plain_chunks_end_where_the_next_begins():
    """Values are one-hot in the position, all scores equal, sinks far below: each row is the mean over its chunk so far."""
    T = 7
    w = {"q": np.zeros((1, T)), "k": np.zeros((1, T)), "v": np.eye(T), "g": np.full((1, T), 60.0), "o": np.eye(T), "sink": np.array([-80.0])}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": T, "scale": 1.0, "mask": {"size": 3}}
    out = P.chunk_attention(m, w, "", np.eye(T))
    want = np.zeros((T, T))
    for i in range(T):
        first = i // 3 * 3
        want[i, first:i + 1] = 1.0 / (i - first + 1)
    np.testing.assert_allclose(out, want, atol=1e-12)
    w["sink"] = np.array([0.0])                              # a sink as large as the scores: one more term in the sum
    np.testing.assert_allclose(P.chunk_attention(m, w, "", np.eye(T))[3:5, 3:5], [[0.5, 0.0], [1 / 3, 1 / 3]], atol=1e-12)
