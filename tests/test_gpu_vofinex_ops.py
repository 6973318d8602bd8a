"""Vofinex's mechanisms one at a time, each kernel (or kernel option) against the plain model's function for it: branches and
a vector joining the stream under a layer norm with a bias, rotation + unit RMS per head + cache write, chunks and sinks in the
three attention kernels, the router with a correction, experts with matrices among experts that return their input (through the
routing table and ordered by expert), the factor on the logits."""
import numpy as np
import pytest
import torch

import plain_vofinex as P
from qstream_b200.csrc import attention_bf16, ops
from qstream_b200.parts.rotary import _table

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device=DEV)


def i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device=DEV)


def rounded(a, dtype=torch.float32):
    """Rounded to `dtype`, as float64: what the kernels are given."""
    return torch.tensor(np.asarray(a), dtype=torch.float64).to(dtype).double().numpy()


# ----------------------------------------------------------------------------- the stream

@pytest.mark.parametrize("T,D", [(5, 50), (5, 64), (3, 1000), (2, 2048), (3, 4096), (2, 6000), (260, 72), (257, 1024), (256, 2304), (256, 9000)])
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("n_branches", [0, 1, 2, 3])
def test_branches_join_the_stream_under_a_layer_norm(T, D, dtype, n_branches):
    """Every number of branches, one of them a vector for all tokens; widths that take the 16-byte form with one, two and
    four pieces a thread and widths that do not; a stream with a mean far from zero."""
    rng = np.random.default_rng(D + n_branches)
    eps = 1e-3
    x = rounded(rng.normal(5.0, 2, (T, D)))
    ys, vec = [rounded(rng.normal(0, s, (T, D))) for s in (3.0, 0.5)], rounded(rng.normal(0, 1, D))
    parts = [(0.3, ys[0]), (1.0, np.broadcast_to(vec, (T, D))), (-0.7, ys[1])][:n_branches]
    on_device = [(0.3, dev(ys[0])), (1.0, dev(vec).expand(T, -1)), (-0.7, dev(ys[1]))][:n_branches]
    new = x + sum((c * y for c, y in parts), np.zeros((T, D)))
    w, b = rounded(1 + rng.normal(0, 0.3, D), dtype), rounded(rng.normal(0, 0.5, D), dtype)
    xd = dev(x)
    before = xd.clone()
    h = ops.stream_norm(xd, on_device, dev(w, dtype), dev(b, dtype), eps, True, dtype)
    if n_branches:
        np.testing.assert_allclose(xd.cpu().numpy(), new, rtol=0, atol=4e-6)
    else:
        assert torch.equal(xd, before)
    tol = dict(rtol=0, atol=2e-5) if dtype == F32 else dict(rtol=2 ** -8, atol=1e-3)
    np.testing.assert_allclose(h.double().cpu().numpy(), P.layer_norm(new, w, b, eps), **tol)
    # an RMS norm without a bias, and a weight stored in another type than the result
    h = ops.stream_norm(dev(new), (), dev(w), None, eps, False, dtype, settled=True)
    np.testing.assert_allclose(h.double().cpu().numpy(), P.unit_rms(rounded(new), eps) * rounded(w), **tol)


def test_the_factor_on_the_logits():
    x = torch.randn(7, 333, device=DEV)
    want = x.double().cpu().numpy() * 1.7
    np.testing.assert_allclose(ops.scale(x, 1.7).cpu().numpy(), want, rtol=2e-7)


# ----------------------------------------------------------------------------- queries and keys

QK_SIZES = [(4, 2, 16, 8, 8, True), (3, 1, 24, 40, 16, True), (6, 2, 64, 64, 32, True), (5, 5, 128, 16, 64, True), (2, 1, 6, 10, 4, True), (3, 3, 14, 14, 0, True),
            (20, 4, 128, 128, 128, True), (2, 1, 256, 96, 16, True), (1, 1, 250, 6, 48, True), (2, 2, 400, 64, 32, True), (7, 1, 80, 48, 48, True),
            (4, 2, 32, 24, 16, False), (3, 1, 72, 8, 8, False), (2, 2, 10, 4, 6, False), (30, 10, 48, 48, 16, True), (4, 1, 64, 32, 24, True)]


@pytest.mark.parametrize("H,G,d,dv,dims,half", QK_SIZES)
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("copies", [1, 40])
def test_rotation_then_a_unit_rms_per_head_then_the_cache(H, G, d, dv, dims, half, dtype, copies):
    """q, k, v are views of one product's result; positions across pages that lie in no order; a row of nobody stays as it is;
    few tokens (several blocks each) and many (one block each).  A tiny head shows eps."""
    rng = np.random.default_rng(H * d + dims)
    base, eps = 1e3, 1e-2
    pos = np.array([0, 1, 63, 64, 65, 130, 191, 5])
    slots = np.array([0] * 7 + [-1])
    if copies > 1:                                          # the same sequence positions in `copies` slots
        pos, slots = np.tile(pos, copies), np.concatenate([np.where(slots < 0, -1, c) for c in range(copies)])
    T = len(pos)
    x = rounded(rng.normal(size=(T, (H + G) * d + G * dv + 8)), dtype)
    x[:, :d] *= 0.05
    x = rounded(x, dtype)
    q, k, v = x[:, :H * d].reshape(T, H, d), x[:, H * d:(H + G) * d].reshape(T, G, d), x[:, (H + G) * d:(H + G) * d + G * dv]
    if half:
        want_q, want_k = P.queries_and_keys({"rot": {"dims": dims, "base": base}}, q, k, pos, eps)
    else:                                                   # neighbours: the same turn after sorting even and odd dims
        order = np.concatenate([np.arange(0, dims, 2), np.arange(1, dims, 2), np.arange(dims, d)])
        want_q, want_k = (np.empty_like(a) for a in (q, k))
        for a, out in ((q, want_q), (k, want_k)):
            out[..., order] = P.unit_rms(P.rotate(a[..., order], pos, dims, base), eps)
    pages = np.stack([rng.permutation(4 * copies)[:3] for _ in range(1)] if copies == 1 else np.split(rng.permutation(3 * copies), copies))
    kc, vc = torch.zeros((4 * copies, G, 64, d), dtype=dtype, device=DEV), torch.zeros((4 * copies, G, 64, dv), dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    xd = dev(x, dtype)
    ops.rope_unit_store(xd[:, :H * d], xd[:, H * d:(H + G) * d], xd[:, (H + G) * d:(H + G) * d + G * dv], eps, H, G, d, dims,
                        _table(dims, base, 4096, DEV) if dims else None, i32(slots), i32(pos), i32(pages), 64, kc, vc, status,
                        v_head_dim=dv, half_layout=half)
    got = xd.double().cpu().numpy()
    live = slots >= 0
    tol = dict(rtol=0, atol=4e-6) if dtype == F32 else dict(rtol=2 ** -8, atol=1e-3)
    np.testing.assert_allclose(got[live, :H * d].reshape(-1, H, d), want_q[live], **tol)
    np.testing.assert_array_equal(got[~live], x[~live])
    np.testing.assert_array_equal(got[:, H * d:], x[:, H * d:])               # k and v themselves stay as projected
    kh, vh = kc.double().cpu().numpy(), vc.double().cpu().numpy()
    for t in np.nonzero(live)[0]:
        page, at = pages[slots[t]][pos[t] // 64], pos[t] % 64
        np.testing.assert_allclose(kh[page, :, at], want_k[t], **tol)
        np.testing.assert_array_equal(vh[page, :, at], v[t].reshape(G, dv))
    assert int(status.item()) == 0
    # queries only
    xd = dev(x, dtype)
    ops.rope_unit_store(xd[:, :H * d], None, None, eps, H, 0, d, dims, _table(dims, base, 4096, DEV) if dims else None, i32(slots), i32(pos), None, 64,
                        None, None, status, half_layout=half)
    got = xd.double().cpu().numpy()
    np.testing.assert_allclose(got[live, :H * d].reshape(-1, H, d), want_q[live], **tol)
    np.testing.assert_array_equal(got[:, H * d:], x[:, H * d:])


def test_a_position_outside_the_table_and_a_page_nobody_holds_are_reported():
    x = torch.randn(1, 48, dtype=BF, device=DEV)
    kc = torch.zeros((1, 1, 64, 16), dtype=BF, device=DEV)
    for pos, table, code in ((200, [[0, 0, 0, 0]], 1), (70, [[0, -1, -1, -1]], 2)):
        for d in (16, 12):                                  # the 16-byte form and the other
            status = torch.zeros(1, dtype=torch.int32, device=DEV)
            ops.rope_unit_store(x[:, :d], x[:, 16:16 + d], x[:, 32:32 + d], 1e-5, 1, 1, d, 0 if code == 2 else (16 if d == 16 else 4),
                                None if code == 2 else _table(16 if d == 16 else 4, 1e4, 128, DEV), i32([0]), i32([pos]), i32(table), 64, kc[..., :d].contiguous(),
                                kc[..., :d].contiguous(), status, half_layout=True)
            assert int(status.item()) == code


# ----------------------------------------------------------------------------- attention

@pytest.mark.parametrize("H,G,d,dv,chunk", [(6, 2, 48, 32, 50), (4, 4, 64, 64, 64), (8, 1, 32, 80, 0), (5, 1, 96, 48, 130), (7, 1, 64, 16, 100)])
def test_chunks_and_sinks_in_the_attention_kernels(H, G, d, dv, chunk):
    """The tensor-core prompt kernel, the split-key decode kernel and the generic kernel, over unit-RMS queries and keys, against
    the plain attention; one query and key far back in a chunk stand out."""
    rng = np.random.default_rng(H * d)
    T, scale = 300, 0.2
    q, k, v = (rng.normal(size=(T, n, e)) for n, e in ((H, d), (G, d), (G, dv)))
    far = (T - 1) - (T - 1) % chunk if chunk else 0                          # the first key the last query sees
    q[T - 1] = np.repeat(k[far], H // G, axis=0)
    if far:
        k[far - 1] = 3 * k[far]                                               # and one it must not
    q, k, v = rounded(P.unit_rms(q, 1e-5), BF), rounded(P.unit_rms(k, 1e-5), BF), rounded(v, BF)
    sink = rounded(rng.normal(1, 1.5, H))
    want = P.attend(q, k, v, scale, sink, P.visible_keys(T, chunk)).reshape(T, -1)
    pages = -(-T // 64)
    order = rng.permutation(pages + 2)[:pages]
    kc, vc = torch.zeros((pages + 2, G, 64, d), dtype=BF, device=DEV), torch.zeros((pages + 2, G, 64, dv), dtype=BF, device=DEV)
    for t in range(T):
        kc[order[t // 64], :, t % 64], vc[order[t // 64], :, t % 64] = dev(k[t], BF), dev(v[t], BF)
    table, status = i32(order[None]), torch.zeros(1, dtype=torch.int32, device=DEV)
    qd = dev(q.reshape(T, -1), BF)
    tiles = i32([(a, min(128, T - a), a, 0) for a in range(0, T, 128)])
    opts = dict(v_head_dim=dv, chunk=chunk, sink=dev(sink))
    got = attention_bf16.prefill(qd, H, G, d, scale, 0, tiles, table, 64, kc, vc, status, **opts)
    np.testing.assert_allclose(got.double().cpu().numpy(), want, rtol=0, atol=2e-2 * np.abs(want).max())
    rows = np.array([0, 1, 49, 50, 63, 64, 99, 100, 129, 130, 255, 256, 299])
    got = attention_bf16.decode(qd[rows].contiguous(), H, G, d, scale, 0, i32(np.zeros(len(rows))), i32(rows), table, 64, kc, vc, 320, status, **opts)
    np.testing.assert_allclose(got.double().cpu().numpy(), want[rows], rtol=0, atol=1e-2 * np.abs(want).max())
    got = ops.attention(qd, H, G, d, scale, 0, i32(np.zeros(T)), i32(np.arange(T)), table, 64, kc, vc, status, out_dtype=F32, **opts)
    np.testing.assert_allclose(got.cpu().numpy(), want, rtol=0, atol=1e-5 * np.abs(want).max())
    assert int(status.item()) == 0


# ----------------------------------------------------------------------------- experts

@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (4, 4), (1, 1), (40, 7)])
def test_the_router_with_a_correction(E, top):
    rng = np.random.default_rng(E)
    z, corr = rounded(rng.normal(0, 2, (200, E))), rounded(rng.normal(0, 0.3, E))
    z[0] = -60.0 + z[0] * 0.01
    chosen, weights = P.route(rounded(z), corr, top)
    idx, wts, _ = ops.moe_route(dev(z), dev(corr), E, top, 1, 1, 1.0, scores="softmax", group_score="max")
    np.testing.assert_array_equal(idx.cpu().numpy(), chosen)
    np.testing.assert_allclose(wts.cpu().numpy(), weights, rtol=0, atol=1e-6)
    if 1 < top < E:
        plain, _ = P.route(z, 0 * corr, top)
        assert (np.sort(plain, 1) != np.sort(chosen, 1)).any()                 # the correction did change choices


@pytest.mark.parametrize("T,D,F,E,same,top,dtype,tol", [(11, 40, 12, 3, 2, 2, F32, 2e-5), (3, 50, 7, 1, 4, 3, F32, 2e-5), (9, 64, 16, 4, 1, 5, BF, 4e-2),
                                                        (70, 64, 24, 5, 3, 4, BF, 4e-2), (90, 42, 10, 4, 0, 2, F32, 2e-5), (64, 48, 8, 2, 9, 1, F32, 2e-5)])
def test_experts_that_return_their_input_among_the_others(T, D, F, E, same, top, dtype, tol):
    """Through the routing table, and ordered by expert with one product each; tokens with only such experts, tokens with none of
    them, and (last) a batch in which hardly any expert has work."""
    rng = np.random.default_rng(T)
    x = rounded(rng.normal(size=(T, D)), dtype)
    w = {}
    for e in range(E):
        for n, s in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F))):
            w[f"e{e}.{n}"] = rounded(rng.normal(0, s[1] ** -0.5, s), dtype)
    idx = np.stack([rng.permutation(E + same)[:top] for _ in range(T)])
    if same >= top:
        idx[0] = E + np.arange(top)
    if E >= top:
        idx[1] = np.arange(top)
    wts = rounded(rng.uniform(0.1, 0.9, (T, top)))
    want = np.zeros((T, D))
    for t in range(T):
        for e, c in zip(idx[t], wts[t]):
            want[t] += c * (P.gated_unit(w, f"e{e}.", x[t:t + 1])[0] if e < E else x[t])
    w_up = torch.stack([torch.cat([dev(w[f"e{e}.gate"], dtype), dev(w[f"e{e}.up"], dtype)]) for e in range(E)]).contiguous()
    w_down = torch.stack([dev(w[f"e{e}.down"], dtype) for e in range(E)]).contiguous()
    slots = np.zeros(T)
    slots[-1] = -1
    wide = dev(np.concatenate([x, x], 1), dtype)[:, :D]                        # rows that are not next to one another
    got = ops.moe_experts_indirect(wide, w_up, w_down, i32(idx), dev(wts), i32(slots), "silu", gated=True).cpu().numpy()
    np.testing.assert_allclose(got[:-1], want[:-1], rtol=0, atol=tol)
    assert not got[-1].any()
    offsets, place_token, pair_place = ops.moe_sort(i32(idx), E + same)
    rows = ops.gather_rows(wide, place_token)
    bounds = offsets.tolist()[:E + 1]
    rows = rows[:bounds[-1]]
    hidden, y = torch.empty((rows.shape[0], 2 * F), dtype=dtype, device=DEV), torch.empty((rows.shape[0], D), dtype=F32, device=DEV)
    ops.expert_products(hidden, rows, w_up, bounds)
    ops.expert_products(y, ops.gated_act(hidden, "silu"), w_down, bounds)
    got = ops.moe_combine(y, pair_place, dev(wts), i32(slots), x=wide).cpu().numpy()
    np.testing.assert_allclose(got[:-1], want[:-1], rtol=0, atol=tol)
    assert not got[-1].any()


def test_a_step_in_which_every_choice_returns_its_input():
    T, D = 40, 32
    x = torch.randn(T, D, device=DEV)
    idx, wts = i32(np.tile([3, 2], (T, 1))), dev(np.tile([0.5, 0.25], (T, 1)))
    offsets, place_token, pair_place = ops.moe_sort(idx, 4)
    bounds = offsets.tolist()[:3]
    assert bounds == [0, 0, 0]
    rows = ops.gather_rows(x, place_token)[:0]
    w_up, w_down = torch.randn(2, 16, D, device=DEV), torch.randn(2, D, 8, device=DEV)
    hidden, y = torch.empty((0, 16), device=DEV), torch.empty((0, D), device=DEV)
    ops.expert_products(hidden, rows, w_up, bounds)
    ops.expert_products(y, ops.gated_act(hidden, "silu"), w_down, bounds)
    out = ops.moe_combine(y, pair_place, wts, i32(np.zeros(T)), x=x)
    torch.testing.assert_close(out, 0.75 * x, rtol=0, atol=1e-6)
