"""Fotanex's mechanisms one at a time, each kernel (or kernel option) against the plain model's function for it: branches
joining the stream under norms of their own and the tanh reads behind them, the short convolution and its state, the
selective scan, the gated linear recurrent unit and the state-space dual form (in order, carried from step to step, in
chunks), the gate and norm behind the last, the gate per head inside the attention kernels, block products with 32-bit
results, the renormalised router and gated experts through the routing table."""
import numpy as np
import pytest
import torch

import plain_fotanex as P
from qstream_b200.csrc import attention_bf16, ops

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


def chunks_of(n, size=64):
    starts = list(range(0, n, size)) + [n]
    k = len(starts) - 1
    return i32(starts), i32(np.arange(k)), i32([0, k]), k


# ----------------------------------------------------------------------------- the stream

@pytest.mark.parametrize("D", [50, 64, 1000, 2048])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_branches_join_the_stream_and_are_read_through_two_tanh_norms(D, dtype):
    rng = np.random.default_rng(D)
    T, eps = 5, 1e-5
    x, ys = rounded(rng.normal(0, 2, (T, D))), [rounded(rng.normal(0, s, (T, D))) for s in (3.0, 0.5, 1.0)]
    ws = [rounded(1 + rng.normal(0, 0.3, D), dtype) for _ in range(6)]
    new = x + 0.5 * P.rms_norm(ys[0], ws[0], eps) + 0.5 * P.rms_norm(ys[1], ws[1], eps) + ys[2]
    xd = dev(x)
    reads = [(0.7, dev(ws[2], dtype), dev(ws[3], dtype), None), (1.9, dev(ws[4], dtype), dev(ws[5], dtype), None)]
    hs = ops.stream_tanh_norm(xd, [(0.5, dev(ys[0]), dev(ws[0], dtype)), (0.5, dev(ys[1]), dev(ws[1], dtype)), (1.0, dev(ys[2]), None)],
                              eps, reads, dtype)
    np.testing.assert_allclose(xd.cpu().numpy(), new, rtol=0, atol=4e-6)
    tol = 4e-6 if dtype == F32 else 2e-2
    np.testing.assert_allclose(hs[0].double().cpu().numpy(), P.tanh_norm(new, 0.7, ws[2], ws[3]), rtol=0, atol=tol)
    np.testing.assert_allclose(hs[1].double().cpu().numpy(), P.tanh_norm(new, 1.9, ws[4], ws[5]), rtol=0, atol=tol)
    # a read of x itself, into one half of a wider buffer; no branches: x stays
    both = torch.full((T, 2 * D), 7.0, dtype=dtype, device=DEV)
    before = xd.clone()
    ops.stream_tanh_norm(xd, reads=[(0.0, None, None, both[:, D:])], out_dtype=dtype)
    assert torch.equal(xd, before) and torch.equal(both[:, D:], xd.to(dtype)) and bool((both[:, :D] == 7.0).all())
    ops.stream_tanh_norm(xd, [(2.0, dev(ys[2]), None)])                            # a branch and no read
    np.testing.assert_allclose(xd.cpu().numpy(), new + 2.0 * ys[2], rtol=0, atol=8e-6)


# ----------------------------------------------------------------------------- the short convolution

@pytest.mark.parametrize("C,taps", [(24, 4), (16, 3), (13, 2), (40, 5), (7, 1), (32, 2)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_the_short_convolution_over_steps_of_every_size(C, taps, dtype):
    """Two sequences in one batch, their tokens in steps of unequal sizes (longer and shorter than the filter), then one
    by one, then a longer step again; a third slot stays as it is, rows of no sequence come out as zeros."""
    rng = np.random.default_rng(C * taps)
    n_tok = {2: 37, 0: 30}
    xs = {s: rounded(rng.normal(size=(n, C + 3)), dtype) for s, n in n_tok.items()}       # a view of a wider product
    w, b = rounded(rng.normal(size=(C, taps)), dtype), rounded(rng.normal(size=C), dtype)
    want = {s: P.silu(P.causal_conv(x[:, :C], w, b)) for s, x in xs.items()}
    held = torch.zeros((3, taps - 1, C), dtype=dtype, device=DEV) if taps > 1 else None
    if held is not None:
        held[1] = 5.0
    got, at = {2: [], 0: []}, {2: 0, 0: 0}
    for sizes in ((5, 1), (1, 2), (2, 3), (1, 1), (1, 1), (1, 1), (20, 18), (1, 1), (3, 0), (2, 2)):
        rows, slots, pos, starts, seqs = [], [], [], [0], []
        for s, n in zip((2, 0), sizes):
            if not n:
                continue
            rows.append(xs[s][at[s]:at[s] + n])
            slots += [s] * n
            pos += list(range(at[s], at[s] + n))
            starts.append(starts[-1] + n)
            seqs.append(s)
        decode = all(n == 1 for n in sizes)
        slots, pos = slots + [-1], pos + [0]                                # a row of no sequence
        x = dev(np.concatenate([*rows, np.ones((1, C + 3))]), dtype)[:, :C]
        out = ops.short_conv(x, dev(w, dtype), dev(b, dtype), held, i32(slots), i32(pos), "silu", decode=decode).double().cpu().numpy()
        if held is not None and not decode:
            ops.conv_keep(held, x, i32(starts), i32(seqs), len(seqs))
        assert not out[-1].any()
        for k, s in enumerate(seqs):
            got[s].append(out[starts[k]:starts[k + 1]])
            at[s] += starts[k + 1] - starts[k]
    for s in (2, 0):
        g = np.concatenate(got[s])
        np.testing.assert_allclose(g, want[s][:len(g)], rtol=0 if dtype == F32 else 2 ** -8, atol=5e-6 if dtype == F32 else 1e-3)
        if held is not None:
            np.testing.assert_array_equal(held[s].double().cpu().numpy(), xs[s][at[s] - taps + 1:at[s], :C])
    assert held is None or bool((held[1] == 5.0).all())


# ----------------------------------------------------------------------------- recurrences

PIECES = (((300,), False), ((1,) * 40 + (2, 3, 64, 65, 126), False), ((300,), True), ((130, 170), True))


@pytest.mark.parametrize("inner,N,dtype", [(40, 6, F32), (7, 1, F32), (30, 33, F32), (64, 16, F32), (20, 130, F32), (300, 16, BF), (64, 24, BF), (24, 260, BF)])
def test_the_selective_scan_in_order_in_steps_and_in_chunks(inner, N, dtype):
    rng = np.random.default_rng(inner * N)
    T = 300
    x, z, B, C = (rounded(rng.normal(size=(T, n)), dtype) for n in (inner, inner, N, N))
    raw = rounded(P.softplus(rng.normal(size=inner)) + np.log(np.expm1(np.exp(rng.uniform(np.log(1e-3), np.log(0.3), inner)))) + rng.normal(0, 0.5, (T, inner)))
    a_log = rounded(np.log(rng.uniform(0.02, 3.0, (inner, N))), dtype)
    D = rounded(rng.normal(size=inner))
    y, S_end = P.selective_walk(x, P.softplus(raw), -np.exp(a_log), B, C, D, np.zeros((inner, N)))
    want = y * P.silu(z)
    rates = ops.selective_rates(dev(a_log, dtype), dtype)
    scale = np.abs(want).max()
    for pieces, chunked in PIECES:
        state = torch.zeros((2, inner, N), dtype=F32, device=DEV)
        out, at = [], 0
        for n in pieces:
            sl = slice(at, at + n)
            bc = dev(np.concatenate([B[sl], C[sl]], 1), dtype)
            out.append(ops.selective_scan(dev(x[sl], dtype), dev(raw[sl]), rates, bc[:, :N], bc[:, N:], dev(D), dev(z[sl], dtype), state,
                                          i32([0, n]), i32([1]), 1, chunks=chunks_of(n) if chunked else None).double().cpu().numpy())
            at += n
        assert float(state[0].abs().max()) == 0.0                                  # another sequence's slot is untouched
        err, tol = np.abs(np.concatenate(out) - want).max() / scale, 3e-5 if dtype == F32 else 5e-3
        assert err <= tol, (pieces, chunked, err)
        assert np.abs(state[1].cpu().numpy() - S_end).max() <= 3e-5 * np.abs(S_end).max(), (pieces, chunked)


@pytest.mark.parametrize("n,block,dtype", [(48, 16, F32), (34, 34, F32), (30, 3, F32), (256, 64, F32), (192, 32, BF)])
def test_the_gated_recurrent_unit_in_order_in_steps_and_in_chunks(n, block, dtype):
    rng = np.random.default_rng(n)
    T, nb = 300, n // block
    u, y = rounded(rng.normal(size=(T, n)), dtype), rounded(rng.normal(0, 2, (T, n)), dtype)
    gates, bias = rounded(rng.normal(0, 1.5, (T, nb, 2, block))), rounded(rng.normal(0, 0.5, (nb, 2, block)))
    lam = np.log(np.expm1(np.exp(rng.uniform(np.log(3e-4), np.log(0.5), n))))
    rate = rounded(8.0 * P.softplus(lam))
    lam = np.log(np.expm1(rate / 8.0))
    ri = P.sigmoid(gates + bias)
    S, S_end = P.gated_lru_walk(u, ri[:, :, 0].reshape(T, n), ri[:, :, 1].reshape(T, n), lam, np.zeros(n))
    want = S * P.gelu_tanh(y)
    scale = np.abs(want).max()
    for pieces, chunked in PIECES:
        state = torch.zeros((3, n), dtype=F32, device=DEV)
        out, at = [], 0
        for k in pieces:
            sl = slice(at, at + k)
            out.append(ops.gated_lru(dev(u[sl], dtype), dev(gates[sl].reshape(k, -1)), dev(bias.reshape(-1)), dev(rate), dev(y[sl], dtype), state,
                                     block, i32([0, k]), i32([2]), 1, chunks=chunks_of(k) if chunked else None).double().cpu().numpy())
            at += k
        assert float(state[:2].abs().max()) == 0.0
        err, tol = np.abs(np.concatenate(out) - want).max() / scale, 3e-5 if dtype == F32 else 5e-3
        assert err <= tol, (pieces, chunked, err)
        assert np.abs(state[2].cpu().numpy() - S_end).max() <= 3e-5 * np.abs(S_end).max()


@pytest.mark.parametrize("H,G,N,dv,dtype", [(6, 3, 10, 8, F32), (1, 1, 7, 14, F32), (5, 5, 3, 6, F32), (8, 2, 64, 32, BF), (4, 1, 128, 64, BF)])
def test_the_dual_form_in_order_in_steps_and_in_chunks(H, G, N, dv, dtype):
    """q, k and v are views of one product's result, heads share a group's q and k, the gates come from their kernel."""
    rng = np.random.default_rng(H * N)
    T = 300
    xbc = rounded(rng.normal(size=(T, H * dv + 2 * G * N)) * 0.7, dtype)
    raw = rounded(np.log(np.expm1(np.exp(rng.uniform(np.log(2e-3), np.log(0.5), H)))) + rng.normal(0, 0.5, (T, H)))
    a_log = rounded(np.log(rng.uniform(0.05, 2.0, H)))
    n = H * dv
    x = xbc[:, :n].reshape(T, H, dv)
    B, C = (np.repeat(xbc[:, a:a + G * N].reshape(T, G, N), H // G, axis=1) for a in (n, n + G * N))
    dt = P.softplus(raw)
    less_one, dts = ops.ssd_gates(dev(raw), dev(a_log))
    np.testing.assert_allclose(dts.cpu().numpy(), dt, rtol=2e-6)
    np.testing.assert_allclose(less_one.cpu().numpy(), np.expm1(-np.exp(a_log) * dt), rtol=3e-6)
    want, S_end = P.ssd_walk(x, dt, -np.exp(a_log), B, C, np.zeros((H, N, dv)))
    scale = np.abs(want).max()
    for pieces, chunked in PIECES:
        state = torch.zeros((2, H, dv, N), dtype=F32, device=DEV)
        out, at = [], 0
        for k in pieces:
            t = dev(xbc[at:at + k], dtype)
            a, w = ops.ssd_gates(dev(raw[at:at + k]), dev(a_log))
            out.append(ops.state_scan("ssd", t[:, n + G * N:], t[:, n:n + G * N], t[:, :n], state, i32([0, k]), i32([1]), 1, H, N, dv,
                                      token_decay=a, token_weight=w, qk_group=H // G, chunks=chunks_of(k) if chunked else None).cpu().numpy())
            at += k
        assert float(state[0].abs().max()) == 0.0
        err = np.abs(np.concatenate(out).reshape(T, H, dv) - want).max() / scale
        assert err <= 3e-5, (pieces, chunked, err)
        assert np.abs(state[1].cpu().numpy().transpose(0, 2, 1) - S_end).max() <= 3e-5 * np.abs(S_end).max()


def test_a_far_token_is_still_there_after_thousands():
    """One channel (or head) that forgets a ten-thousandth per token among others that forget fast: what the first token wrote is
    read back 3,000 tokens later, in order as in chunks, without the drift that rounded decays would add up to."""
    T, far = 3000, 1e-4
    for chunked in (False, True):
        chunks = chunks_of(T) if chunked else None
        # selective scan: channel 0 keeps, the token's x is an impulse
        x = np.zeros((T, 2)); x[0] = 3.0
        raw = np.full((T, 2), np.log(np.expm1(0.25)))
        a_log = np.log(np.array([[far * 4], [20.0]]))
        st = torch.zeros((1, 2, 1), device=DEV)
        one = np.ones((T, 1))
        out = ops.selective_scan(dev(x), dev(raw), ops.selective_rates(dev(a_log), F32), dev(one), dev(one), dev(np.zeros(2)), dev(np.full((T, 2), 40.0)),
                                 st, i32([0, T]), i32([0]), 1, chunks=chunks).cpu().numpy()
        np.testing.assert_allclose(out[-1], [0.25 * 3.0 * np.exp(-far * (T - 1)) * 40.0, 0.0], rtol=1e-5, atol=1e-30)
        # the gated unit: rate far * 2 with r = sigmoid(0)
        u = np.zeros((T, 2)); u[0] = 3.0
        st = torch.zeros((1, 2), device=DEV)
        rate = np.array([2 * far, 10.0])
        out = ops.gated_lru(dev(u), dev(np.zeros((T, 4))), dev(np.zeros(4)), dev(rate), dev(np.full((T, 2), 30.0)), st, 2, i32([0, T]), i32([0]), 1,
                            chunks=chunks).cpu().numpy()
        np.testing.assert_allclose(out[-1], [1.5 * np.sqrt(-np.expm1(-2 * far)) * np.exp(-far * (T - 1)) * 30.0, 0.0], rtol=1e-5, atol=1e-30)
        # the dual form: two heads
        k, q, v = np.ones((T, 1)), np.ones((T, 1)), np.zeros((T, 2)); v[0] = 3.0
        st = torch.zeros((1, 2, 1, 1), device=DEV)
        a, w = ops.ssd_gates(dev(raw), dev(a_log[:, 0]))
        out = ops.state_scan("ssd", dev(q), dev(k), dev(v), st, i32([0, T]), i32([0]), 1, 2, 1, 1, token_decay=a, token_weight=w, qk_group=2,
                             chunks=chunks).cpu().numpy()
        np.testing.assert_allclose(out[-1], [0.75 * np.exp(-far * (T - 1)), 0.0], rtol=1e-5, atol=1e-30)


@pytest.mark.parametrize("scan", ["selective", "lru", "dual"])
def test_unequal_sequences_and_empty_rows_share_a_batch(scan):
    """Three sequences (one with nothing to do in this step), slots in no order, rows of nobody behind them: each as if
    alone, their states in their own slots."""
    rng = np.random.default_rng(5)
    lens, slots, T = (9, 0, 1, 20), (3, 1, 0, 2), 33
    starts = np.concatenate([[0], np.cumsum(lens)])

    def go(sl, st, seq_starts, seq_slots):
        if scan == "selective":
            return ops.selective_scan(dev(X[sl]), dev(R[sl]), rates, dev(Bm[sl]), dev(Cm[sl]), dev(np.ones(12)), dev(Z[sl]), st, i32(seq_starts), i32(seq_slots), len(seq_slots))
        if scan == "lru":
            return ops.gated_lru(dev(X[sl]), dev(G2[sl]), dev(np.zeros(24)), dev(np.full(12, 0.3)), dev(Z[sl]), st, 4, i32(seq_starts), i32(seq_slots), len(seq_slots))
        return ops.state_scan("ssd", dev(Cm[sl]), dev(Bm[sl]), dev(X[sl]), st, i32(seq_starts), i32(seq_slots), len(seq_slots), 3, 5, 4,
                              token_decay=dev(-np.abs(R[sl][:, :3]) * 0.1), token_weight=dev(np.abs(R[sl][:, 3:6])), qk_group=3)
    X, R, Z, Bm, Cm, G2 = (rng.normal(size=(T, k)) for k in (12, 12, 12, 5, 5, 24))
    rates = ops.selective_rates(dev(rng.normal(size=(12, 5))), F32)
    shape = {"selective": (4, 12, 5), "lru": (4, 12), "dual": (4, 3, 4, 5)}[scan]
    init = dev(rng.normal(size=shape))
    st = init.clone()
    got = go(slice(0, T), st, starts, slots).cpu().numpy()
    assert not got[30:].any()
    for i, (n, slot) in enumerate(zip(lens, slots)):
        alone = init.clone()
        if n:
            ref = go(slice(starts[i], starts[i + 1]), alone, [0, n], [slot]).cpu().numpy()
            np.testing.assert_array_equal(got[starts[i]:starts[i + 1]], ref)
        assert torch.equal(st[slot], alone[slot])


@pytest.mark.parametrize("n,dv,parts,dtype", [(48, 8, 4, F32), (14, 14, 1, F32), (30, 6, 15, F32), (256, 32, 4, BF), (2048, 64, 1, BF), (2048, 128, 16, BF)])
def test_the_gate_and_the_norm_over_parts_behind_the_dual_form(n, dv, parts, dtype):
    rng = np.random.default_rng(n + parts)
    T = 6
    o, x, z = rounded(rng.normal(0, 2, (T, n))), rounded(rng.normal(size=(T, n)), dtype), rounded(rng.normal(0, 2, (T, n)), dtype)
    D, w = rounded(rng.normal(size=n // dv)), rounded(1 + rng.normal(0, 0.3, n), dtype)
    want = P.gate_then_group_norm(o + np.repeat(D, dv) * x, z, w, parts, 1e-5)
    got = ops.ssd_output(dev(o), dev(x, dtype), dev(z, dtype), dev(D), dev(w, dtype), dv, parts, 1e-5).double().cpu().numpy()
    np.testing.assert_allclose(got, want, rtol=2e-6 if dtype == F32 else 2 ** -8, atol=3e-6 if dtype == F32 else 1e-3)


# ----------------------------------------------------------------------------- attention, products, experts

@pytest.mark.parametrize("H,G,d,dv,chunk", [(6, 2, 48, 32, 50), (4, 4, 64, 64, 64), (8, 2, 32, 80, 0), (5, 1, 96, 48, 130)])
def test_a_gate_value_per_head_inside_the_attention_kernels(H, G, d, dv, chunk):
    """The tensor-core prompt kernel and the split-key decode kernel with a gate [T, heads] at any row stride, chunks and
    sinks, and the generic kernel with the gate behind it, against the plain chunk attention."""
    rng = np.random.default_rng(H * d)
    T, scale = 300, d ** -0.5
    q, k, v = (rounded(rng.normal(size=(T, n, e)), BF) for n, e in ((H, d), (G, d), (G, dv)))
    g, sink = rounded(rng.normal(0, 2, (T, H)), BF), rounded(rng.normal(0, 1.5, H))
    # the plain function gets the projections through one-hot inputs
    w = {"q": q.reshape(T, -1).T, "k": k.reshape(T, -1).T, "v": v.reshape(T, -1).T, "g": g.T, "sink": sink, "o": np.eye(H * dv)}
    want = P.chunk_attention({"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": scale, "mask": {"size": chunk}}, w, "", np.eye(T))
    pages = -(-T // 64)
    order = rng.permutation(pages + 2)[:pages]
    kc, vc = torch.zeros((pages + 2, G, 64, d), dtype=BF, device=DEV), torch.zeros((pages + 2, G, 64, dv), dtype=BF, device=DEV)
    for t in range(T):
        kc[order[t // 64], :, t % 64], vc[order[t // 64], :, t % 64] = dev(k[t], BF), dev(v[t], BF)
    table, status = i32(order[None]), torch.zeros(1, dtype=torch.int32, device=DEV)
    gate = torch.zeros((T, H + 3), dtype=BF, device=DEV)[:, 1:H + 1]
    gate.copy_(dev(g, BF))
    qd = dev(q.reshape(T, -1), BF)
    tiles = i32([(a, min(128, T - a), a, 0) for a in range(0, T, 128)])
    opts = dict(v_head_dim=dv, chunk=chunk, sink=dev(sink))
    got = attention_bf16.prefill(qd, H, G, d, scale, 0, tiles, table, 64, kc, vc, status, gate=gate, head_gate=True, **opts)
    np.testing.assert_allclose(got.double().cpu().numpy(), want, rtol=0, atol=2e-2 * np.abs(want).max())
    rows = np.array([0, 1, 49, 50, 63, 64, 129, 130, 255, 256, 299])
    got = attention_bf16.decode(qd[rows].contiguous(), H, G, d, scale, 0, i32(np.zeros(len(rows))), i32(rows), table, 64, kc, vc, 320, status,
                                gate=gate[rows], head_gate=True, **opts)
    np.testing.assert_allclose(got.double().cpu().numpy(), want[rows], rtol=0, atol=1e-2 * np.abs(want).max())
    o = ops.attention(qd, H, G, d, scale, 0, i32(np.zeros(T)), i32(np.arange(T)), table, 64, kc, vc, status, out_dtype=F32, **opts)
    o = ops.gated_group_norm(o, 0, None, dev(g), "sigmoid", 0.0, F32, gate_span=dv)
    np.testing.assert_allclose(o.cpu().numpy(), want, rtol=0, atol=1e-4 * np.abs(want).max())
    assert int(status.item()) == 0


@pytest.mark.parametrize("nb,k,T,dtype", [(3, 16, 9, F32), (1, 34, 5, F32), (4, 64, 40, BF), (6, 32, 7, BF), (5, 10, 50, BF)])
def test_block_products_keep_32_bit_results(nb, k, T, dtype):
    rng = np.random.default_rng(nb * k)
    x, w = rounded(rng.normal(size=(T, nb * k)), dtype), rounded(rng.normal(0, k ** -0.5, (nb, 2 * k, k)), dtype)
    want = np.einsum("boi,tbi->tbo", w, x.reshape(T, nb, k)).reshape(T, -1)
    for fn in (ops.head_linear, ops.head_products):
        out = torch.empty((T, 2 * nb * k), dtype=F32, device=DEV)
        fn(out, dev(x, dtype), dev(w, dtype), nb)
        np.testing.assert_allclose(out.cpu().numpy(), want, rtol=0, atol=1e-5)


@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (4, 4), (1, 1), (40, 3)])
def test_the_router_s_weights_sum_to_one(E, top):
    z = rounded(np.random.default_rng(E).normal(0, 2, (200, E)))
    z[0] = -60.0 + z[0] * 0.01
    chosen, weights = P.route(z, top)
    idx, wts, _ = ops.moe_route(dev(z), None, E, top, 1, 1, 1.0, scores="softmax", group_score="max", renorm_eps=1e-20)
    np.testing.assert_array_equal(idx.cpu().numpy(), chosen)
    np.testing.assert_allclose(wts.cpu().numpy(), weights, rtol=0, atol=1e-6)
    np.testing.assert_allclose(wts.cpu().numpy().sum(1), 1.0, rtol=0, atol=1e-6)


@pytest.mark.parametrize("T,D,F,dtype,tol", [(11, 40, 12, F32, 2e-5), (3, 50, 7, F32, 2e-5), (9, 64, 16, BF, 4e-2)])
def test_gated_experts_through_the_routing_table(T, D, F, dtype, tol):
    rng = np.random.default_rng(T)
    E, top = 5, 2
    x = rounded(rng.normal(size=(T, D)), dtype)
    w = {}
    for e in range(E):
        for n, s in (("gate", (F, D)), ("up", (F, D)), ("down", (D, F))):
            w[f"e{e}.{n}"] = rounded(rng.normal(0, s[1] ** -0.5, s), dtype)
    idx = np.stack([rng.permutation(E)[:top] for _ in range(T)])
    wts = rounded(rng.uniform(0.1, 0.9, (T, top)))
    want = np.zeros((T, D))
    for t in range(T):
        for e, c in zip(idx[t], wts[t]):
            want[t] += c * P.expert(w, f"e{e}.", x[t:t + 1])[0]
    w_up = torch.stack([torch.cat([dev(w[f"e{e}.gate"], dtype), dev(w[f"e{e}.up"], dtype)]) for e in range(E)]).contiguous()
    w_down = torch.stack([dev(w[f"e{e}.down"], dtype) for e in range(E)]).contiguous()
    slots = np.zeros(T)
    slots[-1] = -1
    got = ops.moe_experts_indirect(dev(x, dtype), w_up, w_down, i32(idx), dev(wts), i32(slots), "silu", gated=True).cpu().numpy()
    np.testing.assert_allclose(got[:-1], want[:-1], rtol=0, atol=tol)
    assert not got[-1].any()
