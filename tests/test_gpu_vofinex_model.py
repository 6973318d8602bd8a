"""Vofinex through the engine, against the plain float64 model: whole prompts, token-by-token decoding, prompts cut
into portions, batches of unequal requests, slots and pages used again, long decoding across pages and chunks, sharp
scores that rest on single keys at the chunks' edges, a far token, loops of every shape, greedy generation through the library's
entry point."""
import copy
import json

import numpy as np
import pytest

import qstream_b200 as qs
import plain_vofinex as P
from vofinex_util import (CONFIGS, assert_close, dense, layer, load_plain, logits_error, make_folder, make_weights, model as model_config,
                          moe, write_folder)
from util import random_tokens

pytestmark = pytest.mark.gpu

CASES = [(which, dtype) for dtype in ("float32", "bfloat16") for which in "ABCD"]
SINGLE = [(which, dtype) for dtype in ("float32", "bfloat16") for which in "PFM"]
_REFS = {}


def reference(key, pcfg, w, toks):
    """The plain model's logits of a sequence, computed once per (model, sequence)."""
    k = (key, tuple(toks))
    if k not in _REFS:
        _REFS[k] = P.forward(pcfg, w, toks)
    return _REFS[k]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """(key, plain config, plain weights, library model) per configuration and type, made once."""
    made = {}

    def get(which, dtype):
        if (which, dtype) not in made:
            folder, _ = make_folder(tmp_path_factory.mktemp("vofinex"), which, dtype)
            pcfg, w = load_plain(folder)
            made[which, dtype] = ((which, dtype), pcfg, w, qs.load_model(folder, dtype=dtype, device="cuda"))
        return made[which, dtype]
    return get


def all_places(n):
    return list(range(n))


@pytest.mark.parametrize("which", ["A", "B", "C", "D"])
def test_layer_by_layer(models, which):
    """The residual stream after every layer, in 32-bit."""
    key, pcfg, w, model = models(which, "float32")
    toks = random_tokens(np.random.default_rng(0), 90, pcfg["vocab"])
    _, after = P.forward(pcfg, w, toks, want_layers=True)
    engine = qs.Engine(model, max_tokens=256, max_batch=1, use_graphs=False)
    got = []

    def watched(block, forward):
        def run(x, step, cache_id):
            x = forward(x, step, cache_id)
            got.append(step.pending.apply(x.clone()))       # the layer's last branch is still pending: add it to a copy
            return x
        return run
    for block in model.blocks:
        block.forward = watched(block, block.forward)
    try:
        slot = engine.acquire()
        engine.step([slot], [toks], [[len(toks) - 1]])
        engine.release(slot)
    finally:
        for block in model.blocks:
            del block.forward
    assert len(got) == len(after)
    for i, (g, ref) in enumerate(zip(got, after)):      # typical rows are off by 1e-6
        err = np.abs(g.cpu().numpy() - ref).max(1) / np.abs(ref).max()
        assert err.max() <= 2e-4 and np.median(err) <= 5e-6, f"run {i} (layer {model.spec.schedule[i].layer}): {err.max():.3e}, median {np.median(err):.3e} of the largest value"


@pytest.mark.parametrize("which,dtype", CASES + SINGLE)
def test_whole_prompts(models, which, dtype):
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=512, max_batch=2)
    rng = np.random.default_rng(1)
    for n in (1, 2, 33, 64, 65, 389):
        toks = random_tokens(rng, n, pcfg["vocab"])
        slot = engine.acquire()
        got = engine.step([slot], [toks], [all_places(n)]).cpu().numpy()
        engine.release(slot)
        assert_close(got, reference(key, pcfg, w, toks), dtype, f"{n} tokens")
    engine.check_status()
    engine.cache.check()


@pytest.mark.parametrize("which,dtype", CASES + SINGLE)
@pytest.mark.parametrize("graphs", [True, False])
def test_token_by_token_equals_the_prompt(models, which, dtype, graphs):
    """From an empty cache on across page borders and every chunk's edge."""
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=256, max_batch=2, use_graphs=graphs)
    toks = random_tokens(np.random.default_rng(2), 140, pcfg["vocab"])
    ref = reference(key, pcfg, w, toks)
    slot = engine.acquire()
    got = [engine.step([slot], [[t]], [[0]]).cpu().numpy()[0] for t in toks]
    engine.release(slot)
    assert_close(np.stack(got), ref, dtype, "one by one")
    engine.check_status()


@pytest.mark.parametrize("which,dtype", CASES)
@pytest.mark.parametrize("portion", [2, 3, 7, 64, 65])
def test_portions(models, which, dtype, portion):
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=256, max_batch=2)
    toks = random_tokens(np.random.default_rng(3), 150, pcfg["vocab"])
    ref = reference(key, pcfg, w, toks)
    slot = engine.acquire()
    got = []
    for a in range(0, len(toks), portion):
        piece = toks[a:a + portion]
        got.append(engine.step([slot], [piece], [all_places(len(piece))]).cpu().numpy())
    engine.release(slot)
    assert_close(np.concatenate(got), ref, dtype, f"portions of {portion}")
    engine.check_status()


@pytest.mark.parametrize("which,dtype", [("A", "float32"), ("C", "bfloat16")])
def test_a_long_prompt_in_long_portions(models, which, dtype):
    """The chunks are counted from the sequence's start, not the portion's."""
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=1024, max_batch=1)
    toks = random_tokens(np.random.default_rng(9), 700, pcfg["vocab"])
    ref = reference(key, pcfg, w, toks)
    slot = engine.acquire()
    got = [engine.step([slot], [toks[a:b]], [all_places(b - a)]).cpu().numpy() for a, b in ((0, 300), (300, 301), (301, 700))]
    engine.release(slot)
    assert_close(np.concatenate(got), ref, dtype, "portions of 300, 1 and 399")
    engine.check_status()


@pytest.mark.parametrize("which,dtype", CASES)
def test_batches_of_unequal_requests_and_reused_slots(models, which, dtype):
    """Prompts of unequal lengths in one step, then one token each until the shorter ones end; a second batch
    takes the slots and pages the first gave back (fewer pages than the two batches need together)."""
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=64 * 8, max_batch=3)
    rng = np.random.default_rng(4)
    for lens, prompt in (((130, 1, 67), (100, 1, 40)), ((64, 129, 3), (33, 128, 2)), ((300, 20, 5), (290, 3, 1))):
        reqs = [random_tokens(rng, n, pcfg["vocab"]) for n in lens]
        refs = [reference(key, pcfg, w, t) for t in reqs]
        slots = [engine.acquire() for _ in reqs]
        got = [[] for _ in reqs]
        first = engine.step(slots, [t[:p] for t, p in zip(reqs, prompt)], [all_places(p) for p in prompt]).cpu().numpy()
        at = 0
        for i, p in enumerate(prompt):
            got[i].append(first[at:at + p])
            at += p
        pos = list(prompt)
        live = list(range(len(reqs)))
        for i in [i for i in live if pos[i] == len(reqs[i])]:       # a request that was all prompt
            engine.release(slots[i])
            live.remove(i)
        while live:
            out = engine.step([slots[i] for i in live], [[reqs[i][pos[i]]] for i in live], [[0]] * len(live)).cpu().numpy()
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
                pos[i] += 1
            for i in [i for i in live if pos[i] == len(reqs[i])]:
                engine.release(slots[i])
                live.remove(i)
        for i, ref in enumerate(refs):
            assert_close(np.concatenate(got[i]), ref, dtype, f"request {i} of lengths {lens}")
        engine.cache.check()
    engine.check_status()
    assert engine.cache.slots.n_free == engine.cache.slots.n_slots


@pytest.mark.parametrize("which,dtype", [("A", "float32"), ("B", "bfloat16"), ("C", "bfloat16")])
def test_long_decoding(models, which, dtype):
    """300 tokens one by one after a short prompt: across page borders, into every chunk several times over (the pages of
    chunks that are over are given back and handed out again) and the 256-token border at which the engine changes to
    another captured step; a second sequence runs along and ends early."""
    key, pcfg, w, model = models(which, dtype)
    engine = qs.Engine(model, max_tokens=64 * 8, max_batch=2)
    rng = np.random.default_rng(5)
    a, b = random_tokens(rng, 330, pcfg["vocab"]), random_tokens(rng, 90, pcfg["vocab"])
    ra, rb = reference(key, pcfg, w, a), reference(key, pcfg, w, b)
    sa, sb = engine.acquire(), engine.acquire()
    first = engine.step([sa, sb], [a[:30], b[:5]], [[29], [4]]).cpu().numpy()
    ga, gb = [first[0]], [first[1]]
    for i in range(300):
        both = 5 + i < len(b)
        out = engine.step([sa, sb] if both else [sa], [[a[30 + i]], [b[5 + i]]] if both else [[a[30 + i]]]).cpu().numpy()
        ga.append(out[0])
        if both:
            gb.append(out[1])
        elif sb is not None:
            engine.release(sb)
            sb = None
    engine.release(sa)
    assert_close(np.stack(ga), ra[29:], dtype, "long sequence")
    assert_close(np.stack(gb), rb[4:], dtype, "short sequence")
    engine.check_status()
    engine.cache.check()


# Sharp scores: queries and keys of unit RMS score up to dim * scale, here 20; a query's softmax rests on one or two of the keys it
# sees, so a chunk's edge being one place off, a key read from the wrong page or a sink left out moves many rows' logits by much
# of their spread.
def sharp_config(chunk=23, wide=70, mult=0.7, dims=4, base=1e3):
    return model_config(80, 64, 1e-5, [
        layer(4, 2, 8, 16, chunk, 2.5, (dims, base), None),
        layer(6, 3, 16, 8, wide, 1.2, (8, 1e4), moe(3, 2, 2, 16)),
        layer(2, 1, 8, 16, chunk, 2.5, None, dense(48))], loop=(0, 2, 2), mult=mult)


def sharp_weights(cfg, seed=11, gain_all=1.0):
    weights = make_weights(cfg, seed, gain_all=gain_all)
    weights["l0.mix.sink"] = np.array([14.0, 12.0, 16.0, 13.0], dtype=np.float32)     # of the order of the largest scores
    return weights


def plain_logits(tmp_path, name, cfg, weights, toks, dtype):
    pcfg, w = load_plain(write_folder(tmp_path / name, cfg, weights, dtype))
    return P.forward(pcfg, w, toks)


def test_the_sharp_model_shows_every_edge(tmp_path):
    """The plain model itself: each chunk size changed by one, the sinks left out, the sequence's first page cut off, the pass's
    vector, a norm's bias or the correction forgotten, the rotation of another base or width, branches or stream without their factors
    change a good part of the rows by far more than the limits the library is held to below."""
    cfg, toks = sharp_config(), random_tokens(np.random.default_rng(12), 330, 80)
    weights = sharp_weights(cfg)
    ref = plain_logits(tmp_path, "ref", cfg, weights, toks, "float32")

    def moved(name, c, changes=None):
        return logits_error(plain_logits(tmp_path, name, c, {**weights, **(changes or {})}, toks, "float32"), ref)
    for what, other in (("chunk + 1", sharp_config(chunk=24)), ("chunk - 1", sharp_config(chunk=22)),
                        ("wide + 1", sharp_config(wide=71)), ("wide - 1", sharp_config(wide=69)),
                        ("mult", sharp_config(mult=0.75)), ("dims", sharp_config(dims=2)), ("base", sharp_config(base=900.0)),
                        ("no scale", {**cfg, "embedding": {"scale": 1.0}})):
        e = moved(what.replace(" ", ""), other)
        assert (e > 0.03).sum() >= 30, (what, (e > 0.03).sum())
    assert (moved("nosink", cfg, {"l0.mix.sink": np.full(4, -80.0, dtype=np.float32)}) > 0.03).sum() >= 100
    for name in ("loop.step", "l0.norm1.b", "final.norm.b"):
        assert np.median(moved("no" + name, cfg, {name: weights[name] * 0})) > 0.03, name
    assert (moved("nocorr", cfg, {"l1.mlp.correction": weights["l1.mlp.correction"] * 0}) > 0.03).sum() >= 30
    cut = plain_logits(tmp_path, "cut", cfg, weights, toks[64:], "float32")
    assert np.median(logits_error(cut[-100:], ref[-100:])) > 0.02


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("prompt", [200, 64, 3])
def test_sharp_edges_in_prompts_and_in_decoding(tmp_path, dtype, prompt):
    """A prompt, then token by token: every edge of `sharp_config` falls among keys of the prompt and among decoded ones
    (the chunk of 23 many times, the chunk of 70 across pages)."""
    cfg = sharp_config()
    folder = write_folder(tmp_path / "sharp", cfg, sharp_weights(cfg), dtype)
    pcfg, w = load_plain(folder)
    toks = random_tokens(np.random.default_rng(12), 330, cfg["vocab"])
    ref = P.forward(pcfg, w, toks)
    model = qs.load_model(folder, dtype=dtype, device="cuda")
    engine = qs.Engine(model, max_tokens=512, max_batch=2)
    slot = engine.acquire()
    got = [engine.step([slot], [toks[:prompt]], [all_places(prompt)]).cpu().numpy()]
    got += [engine.step([slot], [[t]], [[0]]).cpu().numpy() for t in toks[prompt:]]
    engine.release(slot)
    e = logits_error(np.concatenate(got), ref)
    if dtype == "float32":
        assert e.max() <= 2e-3 and np.median(e) <= 1e-4, (e.max(), int(e.argmax()), np.median(e))
    else:                                               # sharp scores amplify the rounding of q and k as well
        assert np.median(e) <= 0.06 and np.quantile(e, 0.9) <= 0.25, (np.median(e), np.quantile(e, 0.9), e.max(), int(e.argmax()))
    engine.check_status()
    engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk", [None, 750])
def test_a_far_token_weighs_on_the_last_ones(tmp_path, dtype, chunk):
    """An early token whose key every query looks for, 700 tokens later, among hundreds of others: the norm's bias gives all queries
    one direction (in dims that no rotation turns), that token's keys point there.  The plain model first shows that the last rows
    change when that token is another one; the library must agree with it in a whole prompt, in portions that start behind the
    token's page, and token by token."""
    cfg = model_config(64, 48, 1e-5, [layer(4, 2, 16, 16, chunk, 1.0, (8, 1e4), dense(40)), layer(2, 1, 24, 16, chunk, 0.7, (16, 1e3), None)])
    weights, special, rng = make_weights(cfg, 5, gain_all=0.7), 7, np.random.default_rng(3)
    a = rng.normal(size=48)
    a /= np.linalg.norm(a)
    weights["embed"][special] = 6.0 * a
    for i, (H, G, d) in enumerate(((4, 2, 16), (2, 1, 24))):
        c = weights[f"l{i}.norm1.b"] = (0.5 * rng.normal(size=48)).astype(np.float32)
        for name, n, towards in (("q", H, c / np.linalg.norm(c)), ("k", G, a)):
            u = np.zeros(n * d)
            u.reshape(n, d)[:, d - 6:] = np.sign(np.random.default_rng(9 + i).normal(size=6))
            weights[f"l{i}.mix.{name}"] += (3.0 * np.outer(u, towards)).astype(np.float32)
    folder = write_folder(tmp_path / "far", cfg, weights, dtype)
    pcfg, w = load_plain(folder)
    toks = [int(t) for t in rng.integers(8, cfg["vocab"], 700)]
    toks[2] = special
    ref = P.forward(pcfg, w, toks)
    other = list(toks)
    other[2] = 9
    moved = logits_error(P.forward(pcfg, w, other)[-100:], ref[-100:])
    assert (moved > 3e-2).sum() >= 50, ((moved > 3e-2).sum(), np.median(moved))
    model = qs.load_model(folder, dtype=dtype, device="cuda")
    engine = qs.Engine(model, max_tokens=1024, max_batch=2)
    slot = engine.acquire()
    got = engine.step([slot], [toks], [all_places(700)]).cpu().numpy()
    engine.release(slot)
    assert_close(got, ref, dtype, "whole")
    slot = engine.acquire()
    got = [engine.step([slot], [toks[a:b]], [all_places(b - a)]).cpu().numpy() for a, b in ((0, 70), (70, 400), (400, 640))]
    got += [engine.step([slot], [[t]], [[0]]).cpu().numpy() for t in toks[640:]]
    engine.release(slot)
    assert_close(np.concatenate(got), ref, dtype, "portions, then one by one")
    engine.check_status()


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 1), (0, 3, 3), (1, 2, 4), (2, 3, 2)])
def test_loops_of_every_shape(tmp_path, loop):
    """No loop, one layer, all layers, the middle and the last one, one pass and several, in one portion and in three, and
    one by one: every pass keeps a cache of its own."""
    layers = [layer(2, 1, 8, 8, 11, 0.6, (4, 1e3), moe(4, 2, 2, 10)), layer(3, 3, 10, 4, 7, 0.4, None, None), layer(2, 2, 6, 8, None, 0.5, (6, 50.0), dense(20))]
    cfg = model_config(60, 40, 1e-5, layers, loop)
    folder = write_folder(tmp_path / "loop", cfg, make_weights(cfg, 3), "float32")
    pcfg, w = load_plain(folder)
    toks = random_tokens(np.random.default_rng(2), 45, 60)
    ref = P.forward(pcfg, w, toks)
    engine = qs.Engine(qs.load_model(folder, dtype="float32", device="cuda"), max_tokens=192, max_batch=2)
    for cuts in ((0, 45), (0, 2, 20, 45), tuple(range(46))):
        slot = engine.acquire()
        got = [engine.step([slot], [toks[a:b]], [all_places(b - a)]).cpu().numpy() for a, b in zip(cuts, cuts[1:])]
        engine.release(slot)
        assert_close(np.concatenate(got), ref, "float32", f"{loop} cut at {cuts[1:3]}")
    engine.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_steps_with_short_prompts_are_captured_where_no_experts_run(models, dtype):
    """A model without experts: prompts in portions that want only their last logits replay captured steps padded to
    a larger size; the logits and what they leave in the cache equal the plain model's."""
    key, pcfg, w, model = models("D", dtype)
    engine = qs.Engine(model, max_tokens=512, max_batch=4)
    assert engine.captures_prefill
    rng = np.random.default_rng(17)
    reqs = [random_tokens(rng, n, pcfg["vocab"]) for n in (150, 40, 97)]
    refs = [reference(key, pcfg, w, t) for t in reqs]
    slots = [engine.acquire() for _ in reqs]
    pos = [0, 0, 0]
    rows = [[] for _ in reqs]
    for sizes in ((50, 1, 2), (1, 1, 1), (64, 30, 40), (1, 1, 1), (30, 2, 50)):
        out = engine.step(slots, [t[a:a + n] for t, a, n in zip(reqs, pos, sizes)]).cpu().numpy()
        for i, n in enumerate(sizes):
            pos[i] += n
            rows[i].append((pos[i] - 1, out[i]))
    for i, r in enumerate(rows):
        assert_close(np.stack([x for _, x in r]), refs[i][[p for p, _ in r]], dtype, f"request {i}")
    assert engine._prefill_graphs
    engine.check_status()


@pytest.mark.parametrize("which,dtype", CASES)
def test_greedy_generation_through_the_entry_point(models, which, dtype):
    """More requests than slots, so batches follow one another through the generation loop and the scheduler
    hands slots on.  Every token must be the plain model's choice given the tokens before it."""
    key, pcfg, w, model = models(which, dtype)
    rng = np.random.default_rng(6)
    prompts = [random_tokens(rng, n, pcfg["vocab"]) for n in (5, 1, 40, 2, 66)]
    engine = qs.Engine(model, max_tokens=64 * 6, max_batch=2)
    res = qs.generate(engine, prompts, max_new_tokens=8, sampling=qs.SamplingConfig.greedy(), stop_tokens=())
    assert len(res.batches) >= 3 and all(len(t) == 8 for t in res.tokens)
    for prompt, got in zip(prompts, res.tokens):
        toks = list(prompt)
        for g in got:
            logits = P.forward(pcfg, w, toks)[-1]
            best = int(np.argmax(logits))
            if g != best:
                assert dtype == "bfloat16" and logits[best] - logits[g] < 0.1 * (logits.max() - logits.min()), (toks, g, best)
            toks.append(g)
    engine.cache.check()
    assert engine.cache.slots.n_free == engine.cache.slots.n_slots


def test_a_model_made_from_a_seed_runs_and_saves(tmp_path):
    """`CausalLM.random` and the folder that `write_model_folder` writes hold the same model."""
    config = qs.config_from_dict(copy.deepcopy(CONFIGS["A"]))
    scales = qs.InitScales(0.2, 0.1, 0.1)
    folder = qs.write_model_folder(tmp_path / "made", config, seed=3, dtype="float32", scales=scales)
    pcfg, w = load_plain(folder)
    assert w["l3.mlp.correction"].shape == (8,) and w["loop.step"].shape == (3, 64) and "head" not in w
    toks = random_tokens(np.random.default_rng(7), 50, pcfg["vocab"])
    ref = P.forward(pcfg, w, toks)
    for model in (qs.load_model(folder, dtype="float32"), qs.CausalLM.random(config, 3, "float32", "cuda", scales)):
        engine = qs.Engine(model, max_tokens=128, max_batch=1)
        slot = engine.acquire()
        assert_close(engine.step([slot], [toks], [all_places(50)]).cpu().numpy(), ref, "float32", "seeded model")


def test_the_arrangement_s_ways_give_the_same_layer(models):
    """Where the two output projections run as one product (prompts) and where they do not (decode on two streams, or in order
    without a second stream), a model's logits agree to rounding."""
    key, pcfg, w, model = models("C", "bfloat16")
    assert model.blocks[0].fused_weight is not None and model.blocks[1].fused_weight is None
    assert model.blocks[0].ffn.down.data_ptr() == model.blocks[0].fused_weight[:, model.blocks[0].k_mixer:].data_ptr()
    toks = random_tokens(np.random.default_rng(19), 40, pcfg["vocab"])
    ref = reference(key, pcfg, w, toks)
    for side in (True, False):
        engine = qs.Engine(model, max_tokens=128, max_batch=2, use_graphs=False)
        if not side:
            engine.side_stream = None
        slot = engine.acquire()
        got = [engine.step([slot], [toks[:20]], [all_places(20)]).cpu().numpy()]
        got += [engine.step([slot], [[t]], [[0]]).cpu().numpy() for t in toks[20:]]
        engine.release(slot)
        assert_close(np.concatenate(got), ref, "bfloat16", f"side stream {side}")
    engine.check_status()


@pytest.mark.parametrize("which,dtype", [("A", "float32"), ("E", "bfloat16")])
def test_a_row_does_not_depend_on_its_batch(models, which, dtype):
    """The same request alone, in the middle of others and behind used pages: the same logits to rounding (tighter than the
    distance to the plain model in bfloat16)."""
    key, pcfg, w, model = models(which, dtype)
    rng = np.random.default_rng(23)
    reqs = [random_tokens(rng, n, pcfg["vocab"]) for n in (45, 120, 3, 77)]
    engine = qs.Engine(model, max_tokens=64 * 12, max_batch=4)

    def run(ids):
        slots = [engine.acquire() for _ in ids]
        out = engine.step(slots, [reqs[i][:-2] for i in ids], [all_places(len(reqs[i]) - 2) for i in ids]).cpu().numpy()
        parts, at = {}, 0
        for i in ids:
            parts[i] = [out[at:at + len(reqs[i]) - 2]]
            at += len(reqs[i]) - 2
        for j in (-2, -1):
            out = engine.step(slots, [[reqs[i][j]] for i in ids]).cpu().numpy()
            for k, i in enumerate(ids):
                parts[i].append(out[k:k + 1])
        for s in slots:
            engine.release(s)
        return {i: np.concatenate(p) for i, p in parts.items()}
    alone = {}
    for i in range(4):
        alone.update(run([i]))
    for ids in ([0, 1, 2, 3], [3, 1], [2, 0, 3]):
        for i, got in run(ids).items():
            e = logits_error(got, alone[i])
            if dtype == "float32":
                assert e.max() <= 1e-4, (ids, i, e.max())
            else:
                assert np.median(e) <= 2e-2, (ids, i, np.median(e))
    engine.check_status()
    engine.cache.check()


def test_a_config_without_a_loop_ignores_nothing(tmp_path):
    """A checkpoint with vectors for passes that its config does not have is refused, and so is one that lacks them."""
    folder, cfg = make_folder(tmp_path, "A", "float32")
    without = {k: v for k, v in cfg.items() if k != "loop"}
    (folder / "config.json").write_text(json.dumps(without))
    with pytest.raises(qs.QStreamError, match="loop.step"):
        qs.load_model(folder, dtype="float32", device="cuda")
    weights = make_weights(CONFIGS["A"], 0)
    del weights["loop.step"]
    with pytest.raises(qs.QStreamError, match="loop.step"):
        qs.load_model(write_folder(tmp_path / "lacks", cfg, weights, "float32"), dtype="float32", device="cuda")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_wider_model_with_long_requests(models, dtype):
    """Sizes that the tensor-core kernels take, requests of up to 900 tokens: a whole prompt; a prompt and 260 tokens
    one by one (chunks begin among decoded tokens, pages are given back); three unequal
    requests in one batch, decoded together until each ends."""
    key, pcfg, w, model = models("E", dtype)
    rng = np.random.default_rng(21)
    reqs = [random_tokens(rng, n, pcfg["vocab"]) for n in (900, 300, 70)]
    refs = [reference(key, pcfg, w, t) for t in reqs]
    engine = qs.Engine(model, max_tokens=64 * 24, max_batch=3)
    slot = engine.acquire()
    got = engine.step([slot], [reqs[0]], [all_places(900)]).cpu().numpy()
    engine.release(slot)
    assert_close(got, refs[0], dtype, "whole")
    slot = engine.acquire()
    got = [engine.step([slot], [reqs[0][:640]], [all_places(640)]).cpu().numpy()]
    got += [engine.step([slot], [[t]], [[0]]).cpu().numpy() for t in reqs[0][640:]]
    engine.release(slot)
    assert_close(np.concatenate(got), refs[0], dtype, "a prompt, then one by one")
    prompt = (830, 290, 1)
    slots = [engine.acquire() for _ in reqs]
    first = engine.step(slots, [t[:p] for t, p in zip(reqs, prompt)], [[p - 1] for p in prompt]).cpu().numpy()
    rows = [[first[i]] for i in range(3)]
    pos, live = list(prompt), [0, 1, 2]
    while live:
        for i in [i for i in live if pos[i] == len(reqs[i])]:
            engine.release(slots[i])
            live.remove(i)
        if not live:
            break
        out = engine.step([slots[i] for i in live], [[reqs[i][pos[i]]] for i in live], [[0]] * len(live)).cpu().numpy()
        for j, i in enumerate(live):
            rows[i].append(out[j])
            pos[i] += 1
    for i in range(3):
        assert_close(np.stack(rows[i]), refs[i][prompt[i] - 1:], dtype, f"request {i} in a batch")
    engine.check_status()
    engine.cache.check()
    assert engine.cache.slots.n_free == engine.cache.slots.n_slots
