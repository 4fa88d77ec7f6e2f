"""Mafuzen on the GPU against the plain float64 statement in mafuzen_ref.py: every mechanism alone through the C ABI, then whole
models through the loader, the batch step, the sequence cache and the engine (prefill against decoding, portions, mixed batches,
cells and slots that are used again, far keys and window edges, greedy generation)."""
from __future__ import annotations

import ctypes as C
import math

import numpy as np
import pytest

import koboldcpp_b200.host as H
import mafuzen_ref as R
from koboldcpp_b200.lib import BF16, F32, I32, LinearAttnArgs, NormChainArgs, QkvStoreArgs, SinkAttnArgs, Tensor, TimeMixArgs, TokenShiftArgs, check, lib

pytestmark = pytest.mark.gpu


def dev(a, dtype=np.float32):
    return H.DeviceBuffer.from_numpy(np.ascontiguousarray(a, dtype=dtype), pad=256)


def rel(got, want):
    return float(np.abs(got - want).max() / (np.abs(want).max() + 1e-30))


def seq_info(runs):
    """runs: [(first token, count, slot, fresh)] -> the int32 [4][n] table the scans read."""
    return np.array(runs, dtype=np.int32).T.copy()


# ------------------------------------------------------------------------------------------------ norms
@pytest.mark.parametrize("n,T,ny,shared,h,kind1", [(40, 3, 1, False, True, 0), (70, 2, 1, False, False, 1), (61, 4, 3, True, True, 0), (320, 5, 1, True, True, 1), (1030, 2, 2, False, True, 0),
                                                   (4096, 3, 2, True, True, 0), (5000, 2, 1, False, True, 1), (13001, 1, 2, True, True, 0)])
def test_norm_chain(n, T, ny, shared, h, kind1):
    """x = res + N1(scale * sum y + shared) w1 + b1; h = layer norm of x, with rows inside wider rows and a mean far from zero."""
    rng = np.random.default_rng(n)
    row = n + (n % 4 == 0) * 4 + (n % 4 != 0) * 3
    y, sh, res = rng.standard_normal((T, ny, row)) * 2 + 5, rng.standard_normal((T, row)), rng.standard_normal((T, row)) * 3
    w1, b1, w2, b2 = (rng.standard_normal(n) for _ in range(4))
    eps, scale = 1e-5, 1.0 / ny
    bufs = [dev(a) for a in (y, sh, res, w1, b1, w2, b2)]
    out = H.DeviceBuffer(4 * 2 * T * row + 256)
    a = NormChainArgs(y=bufs[0].ptr, y_s_slot=row, y_s_tok=ny * row, shared=bufs[1].ptr if shared else None, shared_stride=row, res=bufs[2].ptr, res_stride=row, w1=bufs[3].ptr,
                      b1=bufs[4].ptr if kind1 == 0 else None, w2=bufs[5].ptr, b2=bufs[6].ptr, x=out.ptr, x_stride=row, h=out.ptr + 4 * T * row if h else None, h_stride=row, n=n, n_tok=T, n_y=ny,
                      kind1=kind1, kind2=0, y_scale=scale, eps=eps)
    check(lib().b200_op_norm_chain(C.byref(a), None))
    got = out.to_numpy(np.float32, (2, T, row))[:, :, :n]
    s = y[..., :n].sum(1) * scale + (sh[:, :n] if shared else 0.0)
    x = res[:, :n] + (R.layer_norm(s, w1, b1, eps) if kind1 == 0 else R.rms_unit(s, eps) * w1)
    assert rel(got[0], x) < 5e-6
    if h:
        assert rel(got[1], R.layer_norm(x, w2, b2, eps)) < 1e-5


@pytest.mark.parametrize("V,Hh,T,weighted", [(16, 5, 5, True), (64, 3, 9, True), (20, 3, 2, False), (128, 2, 3, False), (200, 2, 3, True), (300, 3, 2, True)])
def test_head_norm_with_a_weight_per_head_and_a_silu_gate(V, Hh, T, weighted):
    rng = np.random.default_rng(V)
    x, gate, w, eps = rng.standard_normal((T, Hh, V)) * 3, rng.standard_normal((T, Hh, V)) * 2, 1 + 0.3 * rng.standard_normal((Hh, V)), 1e-6
    x[:, 0] *= 50.0  # a loud head must not move the others
    row = Hh * V + 5
    gbuf, dx, dw, dout = np.zeros((T, row)), dev(x), dev(w), H.DeviceBuffer(4 * T * row + 256)
    gbuf[:, 2:2 + Hh * V] = gate.reshape(T, -1)
    dg = dev(gbuf)
    tx, tg, to = Tensor.contiguous(dx.ptr, F32, (V, Hh, T)), Tensor.contiguous(dg.ptr + 8, F32, (V, Hh, T)), Tensor.contiguous(dout.ptr, F32, (V, Hh, T))
    tg.nb[2] = to.nb[2] = 4 * row
    check(lib().b200_op_norm_affine(C.byref(tx), dw.ptr if weighted else None, Hh, None, C.byref(tg), None, 2, None, C.byref(to), eps, 1, None))
    got = dout.to_numpy(np.float32, (T, row))[:, :Hh * V].reshape(T, Hh, V)
    want = R.rms_unit(x, eps) * (w if weighted else 1.0) * R.silu(gate)
    for h in range(Hh):
        assert rel(got[:, h], want[:, h]) < 3e-6


# ------------------------------------------------------------------------------------------------ recurrences
def run_retention(q, k, v, decay, pos0, dims, base, portions):
    """q, k [T, H, D], v [T, H, V]; one sequence in portions in slot 1 of 2, the other slot full of stale values; rotation in the scan."""
    T, Hh, D = q.shape
    V = v.shape[2]
    state, dd = dev(np.full((2, Hh * D * V + 8), 5.0)), dev(decay)
    df = dev([base ** (-2.0 * i / dims) for i in range(dims // 2)] or [0.0])
    out, done = np.zeros((T, Hh, V)), 0
    for n in portions:
        sl = slice(done, done + n)
        dq, dk, dv, dp = dev(q[sl].reshape(n, -1)), dev(k[sl].reshape(n, -1)), dev(v[sl].reshape(n, -1)), dev(np.arange(done, done + n) + pos0, np.int32)
        dy, info = H.DeviceBuffer(4 * n * Hh * V + 256), dev(seq_info([(0, n, 1, 1 if done == 0 else 0)]), np.int32)
        a = LinearAttnArgs(q=dq.ptr, k=dk.ptr, v=dv.ptr, q_stride=Hh * D, k_stride=Hh * D, v_stride=Hh * V, decay=dd.ptr, seq_info=info.ptr, n_seq=1, state=state.ptr,
                           slot_stride=Hh * D * V + 8, dst=dy.ptr, dst_stride=Hh * V, heads=Hh, dim=D, vdim=V, act=0, k_scale=D ** -0.5, pos=dp.ptr, freqs=df.ptr, n_dims=dims)
        check(lib().b200_op_linear_attn_scan(C.byref(a), None))
        out[sl] = dy.to_numpy(np.float32, (n, Hh, V))
        done += n
    return out


@pytest.mark.parametrize("Hh,D,V,dims,portions", [(2, 16, 12, 16, [21]), (3, 24, 40, 10, [1, 1, 2, 17, 16, 1]), (1, 130, 9, 130, [20, 3]), (2, 32, 64, 0, [40, 1, 1])])
def test_retention_whole_and_in_portions(Hh, D, V, dims, portions):
    rng = np.random.default_rng(D + V)
    T, base = sum(portions), 300.0
    q, k, v, decay = rng.standard_normal((T, Hh, D)), rng.standard_normal((T, Hh, D)), rng.standard_normal((T, Hh, V)), rng.uniform(0.6, 0.99, Hh)
    pos = np.arange(T)
    qr, kr = (R.rotate_halves(x, pos, dims, base) if dims else x for x in (q, k))
    S, want = np.zeros((Hh, D, V)), np.zeros((T, Hh, V))
    for t in range(T):
        for h in range(Hh):
            S[h], want[t, h] = R.retention_step(S[h], qr[t, h], kr[t, h] * D ** -0.5, v[t, h], decay[h])
    assert rel(run_retention(q, k, v, decay, 0, dims, base, portions), want) < 2e-5
    assert rel(run_retention(q, k, v, decay, 0, dims, base, [T]), want) < 2e-5
    if dims:  # only differences of positions matter
        assert rel(run_retention(q, k, v, decay, 50, dims, base, portions), want) < 5e-5


@pytest.mark.parametrize("width,n_mix,portions", [(5, 1, [7]), (130, 5, [1, 1, 3, 40, 16, 1]), (320, 2, [33])])
def test_token_shift_whole_and_in_portions(width, n_mix, portions):
    """Mixes with the previous token beside a second sequence in another slot; stale values in every slot."""
    rng = np.random.default_rng(width)
    T, lead = sum(portions), 3
    h, mu, other = rng.standard_normal((T, width)), rng.standard_normal((n_mix, width)), rng.standard_normal((2, width))
    prev, dmu, got, done = dev(np.full((3, width + 2), 9.0)), dev(mu), np.zeros((n_mix, T, width)), 0
    for n in portions:
        row = width + lead
        buf = np.zeros((n + 2, row))
        buf[:2, lead:], buf[2:, lead:] = other, h[done:done + n]
        dh, dy, info = dev(buf), H.DeviceBuffer(4 * n_mix * (n + 2) * width + 256), dev(seq_info([(0, 2, 0, 1), (2, n, 2, 1 if done == 0 else 0)]), np.int32)
        a = TokenShiftArgs(h=dh.ptr + 4 * lead, h_stride=row, mu=dmu.ptr, seq_info=info.ptr, n_seq=2, prev=prev.ptr, slot_stride=width + 2, dst=dy.ptr, dst_s_mix=(n + 2) * width,
                           dst_s_tok=width, width=width, n_mix=n_mix, n_tokens=n + 2)
        check(lib().b200_op_token_shift(C.byref(a), None))
        got[:, done:done + n] = dy.to_numpy(np.float32, (n_mix, n + 2, width))[:, 2:]
        done += n
    back = R.token_shift(h, np.zeros(width))
    assert rel(got, h + (back - h) * mu[:, None]) < 1e-6


def run_time_mix(r, k, v, z, w0, u, portions):
    T, Hh, D = r.shape
    state, dw0, du = dev(np.full((2, Hh * D * D + 4), 5.0)), dev(w0), dev(u)
    out, done = np.zeros((T, Hh, D)), 0
    for n in portions:
        sl = slice(done, done + n)
        dr, dk, dv, dz = (dev(x[sl].reshape(n, -1)) for x in (r, k, v, z))
        dy, info = H.DeviceBuffer(4 * n * Hh * D + 256), dev(seq_info([(0, n, 1, 1 if done == 0 else 0)]), np.int32)
        a = TimeMixArgs(r=dr.ptr, k=dk.ptr, v=dv.ptr, z=dz.ptr, r_stride=Hh * D, k_stride=Hh * D, v_stride=Hh * D, z_stride=Hh * D, w0=dw0.ptr, u=du.ptr, seq_info=info.ptr, n_seq=1,
                        state=state.ptr, slot_stride=Hh * D * D + 4, dst=dy.ptr, dst_stride=Hh * D, heads=Hh, dim=D)
        check(lib().b200_op_time_mix_scan(C.byref(a), None))
        out[sl] = dy.to_numpy(np.float32, (n, Hh, D))
        done += n
    return out


@pytest.mark.parametrize("Hh,D,portions", [(3, 8, [5]), (2, 64, [37]), (4, 40, [1, 1, 2, 17, 16, 1]), (1, 130, [20, 3]), (2, 256, [11, 1])])
def test_time_mixing_whole_and_in_portions(Hh, D, portions):
    rng = np.random.default_rng(Hh * D)
    T = sum(portions)
    r, k, v, z = (rng.standard_normal((T, Hh, D)) for _ in range(4))
    w0, u = rng.uniform(-6.0, 0.0, (Hh, D)), rng.standard_normal((Hh, D))
    w = np.exp(-np.exp(z + w0))
    S, want = np.zeros((Hh, D, D)), np.zeros((T, Hh, D))
    for t in range(T):
        for h in range(Hh):
            S[h], want[t, h] = R.time_mix_step(S[h], r[t, h], k[t, h], v[t, h], w[t, h], u[h])
    assert rel(run_time_mix(r, k, v, z, w0, u, portions), want) < 2e-5
    assert rel(run_time_mix(r, k, v, z, w0, u, [T]), want) < 2e-5


def test_time_mixing_bonus_belongs_to_the_current_token_only():
    """Without decay a key read one token later returns its value unweighted; at its own token it returns the bonus."""
    D = 8
    r, k, v, z = (np.zeros((2, 1, D)) for _ in range(4))
    r[:, 0, 2], k[0, 0, 2], v[0, 0] = 1.0, 1.0, np.arange(D)
    u = np.zeros((1, D)); u[0, 2] = -3.0
    got = run_time_mix(r, k, v, z, np.full((1, D), -60.0), u, [2])
    assert np.abs(got[0, 0] + 3.0 * np.arange(D)).max() < 1e-5 and np.abs(got[1, 0] - np.arange(D)).max() < 1e-5


# ------------------------------------------------------------------------------------------------ attention
def run_attn(q, kc, vc, cell_seq, cell_pos, tok_seq, tok_pos, scale, G, slopes=None, window=0, keep=0, gate=None, out_scale=0.0, bf16=0):
    T, Hh, D = q.shape
    V = vc.shape[1] // G
    bufs = [dev(q), dev(kc), dev(vc), dev(cell_seq, np.int32), dev(cell_pos, np.int32), dev(tok_seq, np.int32), dev(tok_pos, np.int32)]
    ds = dev(-np.asarray(slopes)) if slopes is not None else None
    row = Hh * V + 3
    if gate is not None:
        gbuf = np.zeros((T, row)); gbuf[:, 1:1 + Hh * V] = gate.reshape(T, -1)
        dg = dev(gbuf)
    out = dev(np.full((T, row), 7.0))
    a = SinkAttnArgs(q=bufs[0].ptr, q_stride=Hh * D, k_cache=bufs[1].ptr, k_cache_stride=kc.shape[1], v_cache=bufs[2].ptr, v_cache_stride=vc.shape[1], cell_seq=bufs[3].ptr,
                     cell_pos=bufs[4].ptr, tok_seq=bufs[5].ptr, tok_pos=bufs[6].ptr, dst=out.ptr, dst_stride=row, n_head=Hh, n_head_kv=G, dim=D, vdim=V, n_tokens=T, n_kv=len(cell_seq),
                     window=window, keep_first=keep, scale=scale, bf16_products=bf16, gate=dg.ptr + 4 if gate is not None else None, gate_stride=row, gate_per_value=1 if gate is not None else 0,
                     dist_bias=ds.ptr if ds else None, n_dist=1 if ds else 0, dist_linear=1 if ds else 0, out_scale=out_scale)
    need = int(lib().b200_sink_attn_workspace_bytes(C.byref(a)))  # > 0: few tokens and many cells, the cells are split over CTAs
    ws = H.DeviceBuffer(need + 256) if need else None
    check(lib().b200_op_sink_attn_ws(C.byref(a), ws.ptr if ws else None, need, None))
    full = out.to_numpy(np.float32, (T, row))
    if need:  # without a workspace the unsplit form must give the same
        check(lib().b200_op_sink_attn(C.byref(a), None))
        assert np.allclose(out.to_numpy(np.float32, (T, row)), full, rtol=1e-5, atol=1e-6, equal_nan=True)
    assert (full[:, Hh * V:] == 7.0).all()
    return full[:, :Hh * V].reshape(T, Hh, V)


def scattered_cache(rng, n_cells, lens, width_k, width_v):
    """Sequences of the given lengths shuffled into one cache; free cells hold NaN."""
    total = sum(lens)
    order = rng.permutation(n_cells)[:total]
    cell_seq, cell_pos = np.full(n_cells, -1), np.full(n_cells, -1)
    at = 0
    for s, n in enumerate(lens):
        cell_seq[order[at:at + n]], cell_pos[order[at:at + n]] = s, np.arange(n)
        at += n
    kc, vc = np.full((n_cells, width_k), np.nan), np.full((n_cells, width_v), np.nan)
    kc[order], vc[order] = rng.standard_normal((total, width_k)), rng.standard_normal((total, width_v))
    return cell_seq, cell_pos, kc, vc


def rows_of_sequence(cell_seq, cell_pos, s, n):
    return [int(np.where((cell_seq == s) & (cell_pos == j))[0][0]) for j in range(n)]


@pytest.mark.parametrize("Hh,G,D,V,window,keep,biased", [(4, 2, 16, 24, 0, 0, True), (6, 3, 40, 40, 7, 3, False), (8, 1, 64, 64, 1, 0, False), (1, 1, 200, 33, 0, 0, True), (3, 3, 32, 32, 20, 5, True)])
@pytest.mark.parametrize("n_cells", [96, 2304])
def test_attention_single_tokens_scattered_cells_two_sequences(Hh, G, D, V, window, keep, biased, n_cells):
    """The decode form (split over CTAs at 2304 cells): linear distance penalty or window with kept first tokens, gate per value, factor."""
    rng = np.random.default_rng(Hh + D)
    La, Lb = 41, 52
    cell_seq, cell_pos, kc, vc = scattered_cache(rng, n_cells, [La, Lb], G * D, G * V)
    toks = [(0, La - 1), (1, Lb - 1), (0, 0), (1, 7), (0, 2), (0, 6), (1, 20), (0, 23), (1, 1)]
    q, gate, scale, f = rng.standard_normal((len(toks), Hh, D)), rng.standard_normal((len(toks), Hh, V)) * 2, 1.7 / math.sqrt(D), 0.6
    got = run_attn(q, kc, vc, cell_seq, cell_pos, [s for s, _ in toks], [p for _, p in toks], scale, G, [R.slope(h, Hh) for h in range(Hh)] if biased else None, window, keep, gate, f)
    for i, (s, p) in enumerate(toks):
        idx = rows_of_sequence(cell_seq, cell_pos, s, p + 1)
        want = R.softmax_attention(q[i:i + 1], kc[idx].reshape(-1, G, D), vc[idx].reshape(-1, G, V), [p], np.arange(p + 1), scale, biased, window or None, keep)[0]
        assert rel(got[i], want * R.sigmoid(gate[i]) * f) < 2e-5, (i, s, p)


@pytest.mark.parametrize("Hh,G,D,V,T,window,keep,biased", [(4, 2, 16, 24, 70, 0, 0, True), (2, 2, 64, 64, 129, 33, 4, False), (3, 1, 40, 72, 33, 0, 0, True), (1, 1, 128, 128, 64, 17, 1, False)])
@pytest.mark.parametrize("bf16", [0, 1])
def test_attention_prompt_batches_behind_cached_tokens(Hh, G, D, V, T, window, keep, biased, bf16):
    """A portion of T tokens behind P0 cached ones, beside a second sequence in the same cache; f32 products and the tensor cores."""
    rng = np.random.default_rng(T)
    P0, Lb = 23, 30
    cell_seq, cell_pos, kc, vc = scattered_cache(rng, 256, [Lb, P0 + T], G * D, G * V)
    q, gate, scale = rng.standard_normal((T, Hh, D)), rng.standard_normal((T, Hh, V)), 1.3 / math.sqrt(D)
    pos = list(range(P0, P0 + T))
    got = run_attn(q, kc, vc, cell_seq, cell_pos, [1] * T, pos, scale, G, [R.slope(h, Hh) for h in range(Hh)] if biased else None, window, keep, gate, 1.5, bf16)
    idx = rows_of_sequence(cell_seq, cell_pos, 1, P0 + T)
    src = (lambda a: R.bf16_round(a).astype(np.float64)) if bf16 else (lambda a: a)
    want = R.softmax_attention(src(q), src(kc[idx]).reshape(-1, G, D), src(vc[idx]).reshape(-1, G, V), pos, np.arange(P0 + T), scale, biased, window or None, keep) * R.sigmoid(gate) * 1.5
    assert rel(got, want) < (2e-2 if bf16 else 2e-5)


@pytest.mark.parametrize("T,bf16", [(1, 0), (40, 0), (40, 1)])
def test_attention_one_loud_key_at_every_edge(T, bf16):
    """One key's score stands out by far: just inside and just outside the window, the last kept and the first unkept token, itself, and
    hundreds of positions back; and with the distance penalty the loud key wins until its distance eats its lead."""
    rng = np.random.default_rng(5)
    D, V, n, window, keep = 32, 16, 700, 50, 6
    q = np.zeros((T, 1, D)); q[:, 0, 3] = 1.0
    v, p = rng.standard_normal((n, V)), n - 1
    cell_seq, cell_pos = np.zeros(n, dtype=np.int64), np.arange(n)
    tol = 2e-2 if bf16 else 1e-4
    for loud, seen in ((p, True), (p - window + 1, True), (p - window, False), (keep - 1, True), (keep, False), (0, True), (37, False)):
        k = np.zeros((n, D)); k[loud, 3] = 60.0
        got = run_attn(q, k, v, cell_seq, cell_pos, [0] * T, [p] * T, 1.0, 1, None, window, keep, bf16=bf16)
        vis = [j for j in range(n) if R.visible(p, j, window, keep)]
        want = v[loud] if seen else v[vis].mean(0)
        assert np.abs(got[:, 0] - want).max() < tol, loud
    k = np.zeros((n, D)); k[37, 3] = 60.0  # 662 positions back
    for slope in (2.0 ** -8, 0.5):  # the penalty is 2.6: the key wins; 331: the key loses against the nearest ones
        got = run_attn(q, k, v, cell_seq, cell_pos, [0] * T, [p] * T, 1.0, 1, [slope], bf16=bf16)
        s = 60.0 * (np.arange(n) == 37) - slope * (p - np.arange(n))
        w = np.exp(s - s.max())
        assert np.abs(got[:, 0] - (w / w.sum()) @ v).max() < tol


def test_store_with_keys_as_values():
    """q and k are divided by their root mean square per head; the value cache takes the keys as projected."""
    rng = np.random.default_rng(2)
    T, Hh, G, D, n_cells, eps = 5, 4, 2, 20, 16, 1e-5
    q, k = rng.standard_normal((T, Hh, D)) * 4, rng.standard_normal((T, G, D))
    k[:, 0] *= 30.0
    pos, cells = np.arange(T), np.array([5, 0, 15, 7, 2])
    dq, dk, dp, dc = dev(q), dev(k), dev(pos, np.int32), dev(cells, np.int32)
    kc, vc = dev(np.full((n_cells, G * D), 7.0)), dev(np.full((n_cells, G * D), 7.0))
    a = QkvStoreArgs(q=dq.ptr, q_stride=Hh * D, k=dk.ptr, k_stride=G * D, v=dk.ptr, v_stride=G * D, pos=dp.ptr, cells=dc.ptr, k_cache=kc.ptr, k_cache_stride=G * D, v_cache=vc.ptr,
                     v_cache_stride=G * D, n_head=Hh, n_head_kv=G, dim=D, vdim=D, n_dims=0, n_tokens=T, eps=eps, qk_unit_rms=1)
    check(lib().b200_op_qkv_store(C.byref(a), None))
    assert rel(dq.to_numpy(np.float32, (T, Hh, D)), R.rms_unit(q, eps)) < 3e-6
    kk, vv = kc.to_numpy(np.float32, (n_cells, G, D)), vc.to_numpy(np.float32, (n_cells, G, D))
    assert rel(kk[cells], R.rms_unit(k, eps)) < 3e-6 and (vv[cells] == k.astype(np.float32)).all()
    assert (np.delete(kk, cells, 0) == 7.0).all() and (np.delete(vv, cells, 0) == 7.0).all()


# ------------------------------------------------------------------------------------------------ feed-forward pieces, tables, products
@pytest.mark.parametrize("n", [5, 4096])
def test_squared_relu(n):
    x = np.random.default_rng(n).standard_normal(n)
    dx, dy = dev(x), H.DeviceBuffer(4 * n + 256)
    tx, ty = Tensor.contiguous(dx.ptr, F32, (n,)), Tensor.contiguous(dy.ptr, F32, (n,))
    check(lib().b200_op_unary(10, C.byref(tx), C.byref(ty), 0.0, 0.0, None))
    assert rel(dy.to_numpy(np.float32, (n,)), R.relu_squared(x)) < 1e-6


@pytest.mark.parametrize("n,V,T", [(1, 9, 4), (6, 50, 3), (2052, 7, 5)])
def test_rows_of_integers_and_floats(n, V, T):
    rng = np.random.default_rng(n)
    ids = rng.integers(0, V, T)
    ti, tf = rng.integers(-2 ** 31, 2 ** 31, (V, n)), rng.standard_normal((V, n)).astype(np.float32)
    did = dev(ids, np.int32)
    for table, ty, dt in ((ti.astype(np.int32), I32, np.int32), (tf, F32, np.float32)):
        dt_, out = dev(table, dt), H.DeviceBuffer(4 * T * n + 256)
        a, b, c = Tensor.contiguous(dt_.ptr, ty, (n, V)), Tensor.contiguous(did.ptr, I32, (T,)), Tensor.contiguous(out.ptr, ty, (n, T))
        check(lib().b200_op_get_rows(C.byref(a), C.byref(b), C.byref(c), None))
        assert (out.to_numpy(dt, (T, n)) == table[ids]).all()


def bf16_bits(x):
    return (np.ascontiguousarray(R.bf16_round(x)).view(np.uint32) >> 16).astype(np.uint16)


@pytest.mark.parametrize("K,M,N", [(64, 16, 9), (64, 130, 17), (128, 100, 33), (2048, 64, 512), (4096, 300, 100), (704, 320, 70), (2112, 97, 40), (320, 520, 300)])
def test_dense_product_on_the_tensor_cores(K, M, N):
    """Few and many weight rows (tile widths 32 .. 256, K in one or two halves), ragged edges; nothing outside the result is written."""
    rng = np.random.default_rng(K + M)
    W, X = rng.standard_normal((M, K)), rng.standard_normal((N, K))
    need = int(lib().b200_mul_mat_q_workspace_bytes(BF16, K, M, N))
    ws, dw, dx, out = H.DeviceBuffer(need + 256), dev(bf16_bits(W), np.uint16), dev(X), dev(np.full((N, M + 3), 7.0))
    check(lib().b200_mul_mat_q(BF16, dw.ptr, K * 2, dx.ptr, K, out.ptr, M + 3, K, M, N, ws.ptr, need, None))
    got = out.to_numpy(np.float32, (N, M + 3))
    want = R.bf16_round(X).astype(np.float64) @ R.bf16_round(W).astype(np.float64).T
    assert rel(got[:, :M], want) < 1e-5 and (got[:, M:] == 7.0).all() and lib().b200_gemm_status() == 0


@pytest.mark.parametrize("K,M,E,top,T", [(64, 24, 5, 1, 70), (128, 200, 3, 3, 40), (320, 96, 16, 2, 150)])
def test_expert_product_on_the_tensor_cores(K, M, E, top, T):
    rng = np.random.default_rng(K + E)
    W, X = rng.standard_normal((E, M, K)), rng.standard_normal((T, K))
    ids = np.stack([rng.permutation(E)[:top] for _ in range(T)]).astype(np.int32)
    need = int(lib().b200_mul_mat_id_q_workspace_bytes(BF16, K, M, top, T, E))
    ws, dw, dx, did, out = H.DeviceBuffer(need + 512), dev(bf16_bits(W), np.uint16), dev(X), dev(ids, np.int32), H.DeviceBuffer(4 * T * top * M + 256)
    check(lib().b200_mul_mat_id_q(BF16, dw.ptr, K * 2, M * K * 2, E, did.ptr, top, dx.ptr, K, K, out.ptr, M, top * M, K, M, top, 1, T, (ws.ptr + 255) // 256 * 256, need, None))
    want = np.einsum("tsmk,tk->tsm", R.bf16_round(W).astype(np.float64)[ids], R.bf16_round(X).astype(np.float64))
    assert rel(out.to_numpy(np.float32, (T, top, M)), want) < 1e-5 and lib().b200_gemm_status() == 0


# ------------------------------------------------------------------------------------------------ whole models
from koboldcpp_b200 import mafuzen as M  # noqa: E402
from koboldcpp_b200.engine import Engine, Request  # noqa: E402

CONFIGS = {
    # every kind of layer and feed-forward; two layers read the first one's cache; a window shorter than the prompts
    "mixed": lambda: R.make_config([R.attention_layer(mlp=R.dense_cfg()), R.retention_layer(), R.attention_layer(kv_from=0), R.parallel_layer(), R.attention_layer(heads=4, kv_from=0, scale=0.4, mlp=None),
                                    R.parallel_layer(heads=2, kv_heads=2, dim=8, size=5, keep_first=0, mix_heads=1, mix_dim=20, mlp=None)]),
    # a parallel layer first, one head, one kv head, a window of one token, kept tokens beyond the window, one and all experts per token,
    # no shared expert, no rotated entries, dim != vdim, scales of exactly one, a width that is no multiple of 8, no token input
    "odd": lambda: R.make_config([R.parallel_layer(heads=1, kv_heads=1, dim=10, size=1, keep_first=9, mix_heads=5, mix_dim=6, left_scale=1.0, right_scale=1.0, mlp=R.moe_cfg(ff=40, experts=5, top=1, shared=0)),
                                  R.retention_layer(heads=1, dim=24, vdim=40, rot=0, decay=[1.0], mlp=R.moe_cfg(ff=8, experts=3, top=3, shared=10)),
                                  R.attention_layer(heads=1, kv_heads=1, dim=40, vdim=6, mlp=None), R.attention_layer(heads=1, kv_heads=1, dim=40, vdim=6, kv_from=2, mlp=R.dense_cfg(7)),
                                  R.retention_layer(heads=6, dim=10, vdim=6, rot=10, mlp=None)], width=70, vocab=70, eps=1e-6, embed_scale=1.0, side=0),
    # sizes that take the 16-byte and tensor-core paths: width, ff, head rows and the token input multiples of 64
    "aligned": lambda: R.make_config([R.attention_layer(heads=4, kv_heads=4, dim=32, vdim=32, mlp=R.moe_cfg(ff=64, experts=8, top=2, shared=128)),
                                      R.retention_layer(heads=4, dim=32, vdim=32, rot=32, base=1e5, mlp=R.dense_cfg(128)),
                                      R.parallel_layer(heads=6, kv_heads=2, dim=64, size=24, keep_first=4, mix_heads=2, mix_dim=64, mlp=R.moe_cfg(ff=64, experts=4, top=1, shared=64)),
                                      R.attention_layer(heads=4, kv_heads=4, dim=32, vdim=32, kv_from=0, mlp=R.dense_cfg(64))], width=128, vocab=96, side=64),
}


@pytest.fixture(scope="module", params=list(CONFIGS))
def model(request):
    cfg = CONFIGS[request.param]()
    W = R.random_weights(cfg, seed=len(request.param), rank=64 if request.param == "aligned" else 5)
    m = M.build(cfg, R.as_tensors(W), dtype="float32", n_ctx=768, n_seq_max=4, max_batch=400)
    yield cfg, W, m
    m.close()


def logits_err(got, want):
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return float((np.sqrt((d ** 2).mean(-1)) / want.std()).max())


def test_prompt_logits_first_tokens_and_every_position(model):
    cfg, W, m = model
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 70).tolist()
    want = R.logits(cfg, W, toks)
    eng = Engine(m)
    got = eng.step([("a", toks, range(len(toks)))])
    eng.finish("a")
    assert logits_err(got, want) < 1e-4
    one = eng.step([("b", toks[:1], [0])])  # a sequence of one token
    eng.finish("b")
    assert logits_err(one, want[:1]) < 1e-4


@pytest.mark.parametrize("portion", [2, 3, 7, 33])
def test_portions_and_decoding_match_the_whole_prompt(model, portion):
    cfg, W, m = model
    toks = np.random.default_rng(portion).integers(0, cfg["vocab"], 70).tolist()
    want = R.logits(cfg, W, toks)
    eng = Engine(m)
    rows = []
    for a in range(0, 40, portion):
        b = min(a + portion, 40)
        rows.append(eng.step([("p", toks[a:b], range(b - a))]))
    for t in range(40, 70):
        rows.append(eng.step([("p", [toks[t]], [0])]))
    eng.finish("p")
    assert logits_err(np.concatenate(rows), want) < 1e-4


def test_unequal_batch_then_decode_together_and_reuse(model):
    """Three requests of different lengths start in one batch and decode together; the shortest ends first and its cells and slot (the
    recurrent states and the previous token's input with what it left there) go to a new request that joins while the others decode."""
    cfg, W, m = model
    rng = np.random.default_rng(4)
    lens = {"a": (1, 12), "b": (23, 30), "c": (57, 70)}  # prompt length, total length
    toks = {k: rng.integers(0, cfg["vocab"], n).tolist() for k, (_, n) in lens.items()}
    toks["d"] = rng.integers(0, cfg["vocab"], 31).tolist()
    want = {k: R.logits(cfg, W, v) for k, v in toks.items()}
    eng = Engine(m)
    got = {k: [] for k in toks}
    out = eng.step([(k, toks[k][:lens[k][0]], [lens[k][0] - 1]) for k in "abc"])
    for i, k in enumerate("abc"):
        got[k].append((lens[k][0] - 1, out[i]))
    at = {k: lens[k][0] for k in "abc"}
    live, d_started = ["a", "b", "c"], False
    while live:
        out = eng.step([(k, [toks[k][at[k]]], [0]) for k in live])
        for i, k in enumerate(live):
            got[k].append((at[k], out[i])); at[k] += 1
        for k in [k for k in live if at[k] == len(toks[k])]:
            live.remove(k); eng.finish(k)
            if k == "a" and not d_started:  # "d" takes over what "a" held, as a prompt beside the decoding tokens
                d_started = True
                o = eng.step([("d", toks["d"][:20], [19])] + [(x, [toks[x][at[x]]], [0]) for x in live])
                got["d"].append((19, o[0]))
                for i, x in enumerate(live):
                    got[x].append((at[x], o[1 + i])); at[x] += 1
                at["d"] = 20; live.append("d")
    for k, rows in got.items():
        assert logits_err(np.stack([r for _, r in rows]), want[k][[p for p, _ in rows]]) < 1e-4, k
    assert m.seq_length(0) == -1  # everything was given back


def test_long_decoding_across_cache_padding(model):
    cfg, W, m = model
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], 300).tolist()
    want = R.logits(cfg, W, toks)
    eng = Engine(m)
    rows, places = [eng.step([("x", toks[:230], [0, 1, 229])])], [0, 1, 229]
    for t in range(230, 300):  # passes 256 cells
        rows.append(eng.step([("x", [toks[t]], [0])])); places.append(t)
    eng.finish("x")
    assert logits_err(np.concatenate(rows), want[places]) < 2e-4


def test_greedy_generation_through_the_engine(model):
    cfg, W, m = model
    rng = np.random.default_rng(9)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (5, 17, 1, 40)]
    eng = Engine(m, max_step_tokens=24)  # prompts are cut into portions beside decoding requests
    outs = eng.generate([Request(p, 10) for p in prompts])
    for p, out in zip(prompts, outs):
        seq = list(p)
        for tok in out:  # every generated token is the reference's argmax given what came before, or a near tie
            lg = R.logits(cfg, W, seq)[-1]
            top = np.sort(lg)[-2:]
            assert tok == int(np.argmax(lg)) or lg[tok] > top[1] - 1e-3 * (abs(top[1]) + 1), (len(seq), tok)
            seq.append(tok)
        assert len(out) == 10


@pytest.mark.parametrize("name", list(CONFIGS))
def test_bfloat16_portions_batches_and_decoding_agree_with_float32(name):
    """bf16 serving mode: prompt portions of 16 tokens or more take the tensor-core kernels (attention and expert products), over
    cells that earlier portions wrote and beside another request's tokens; shorter portions and single tokens take the f32 kernels.
    All of them must give the logits of the float64 reference up to bf16 rounding."""
    cfg = CONFIGS[name]()
    W = R.random_weights(cfg, seed=5, rank=64 if name == "aligned" else 5)
    rng = np.random.default_rng(1)
    ta, tb = rng.integers(0, cfg["vocab"], 135).tolist(), rng.integers(0, cfg["vocab"], 41).tolist()
    want = R.logits(cfg, W, ta)
    m = M.build(cfg, R.as_tensors(W), dtype="bfloat16", n_ctx=256, n_seq_max=2, max_batch=160)
    eng = Engine(m)
    whole = eng.step([("a", ta, range(135))])
    eng.finish("a")
    parts = [eng.step([("b", tb, []), ("a", ta[:33], range(33))])]  # the freed cells are used again, in another order
    parts += [eng.step([("a", ta[a:b], range(b - a))]) for a, b in ((33, 53), (53, 70), (70, 73), (73, 82), (82, 130))]
    parts += [eng.step([("a", [t], [0])]) for t in ta[130:]]
    m.close()
    for got in (whole, np.concatenate(parts)):
        d = got - want
        d = d - d.mean(-1, keepdims=True)
        e = np.sqrt((d ** 2).mean(-1)) / want.std()
        assert np.isfinite(e).all() and np.quantile(e, 0.8) < 3e-2 and e.max() < 0.12


def test_sharp_attention_far_keys_and_window_edges_through_the_model():
    """Large score scales make the attention sharp, so a wrong position, slope, window edge, kept token or cell would show in the logits;
    the window's edge passes over prompt and decoded tokens, the prompt's end is no multiple of any block size, and the decoded stretch
    crosses the cache padding.  Slow decays keep the first tokens alive in the states."""
    cfg = R.make_config([R.attention_layer(heads=2, kv_heads=1, dim=16, vdim=16, scale=2.0, mlp=None), R.retention_layer(heads=2, decay=[0.999, 0.9], mlp=None),
                         R.parallel_layer(heads=2, kv_heads=1, dim=16, size=100, keep_first=5, scale=3.0, mlp=None), R.attention_layer(heads=2, kv_heads=1, dim=16, vdim=16, scale=2.0, kv_from=0),
                         R.parallel_layer(heads=2, kv_heads=2, dim=8, size=17, keep_first=1, scale=4.0)])
    W = R.random_weights(cfg, seed=21)
    for il in (2, 4):
        W[f"l{il}.mix.right.w0"] = R.bf16_round(W[f"l{il}.mix.right.w0"] - 3.0).astype(np.float64)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 290).tolist()
    want = R.logits(cfg, W, toks)
    m = M.build(cfg, R.as_tensors(W), dtype="float32", n_ctx=512, n_seq_max=2, max_batch=300)
    eng = Engine(m)
    places = [0, 1, 2, 4, 5, 6, 16, 17, 18, 99, 100, 101, 104, 105, 106, 200, 241]
    rows = [eng.step([("a", toks[:242], places)])]
    for t in range(242, 290):
        rows.append(eng.step([("a", [toks[t]], [0])])); places.append(t)
    m.close()
    assert logits_err(np.concatenate(rows), want[places]) < 2e-4


def test_loader_refuses_what_does_not_fit():
    from koboldcpp_b200.lib import B200Error
    cfg = R.make_config([R.attention_layer(mlp=None), R.attention_layer(kv_from=0)])
    W = R.random_weights(cfg)
    bad = dict(W); bad["l1.mlp.table"] = W["l1.mlp.table"] + 5  # experts that do not exist
    with pytest.raises(B200Error, match="table"):
        M.build(cfg, R.as_tensors(bad), n_ctx=256, n_seq_max=1, max_batch=16)
    missing = {k: v for k, v in W.items() if k != "l1.side.proj"}
    with pytest.raises(B200Error, match="side.proj"):
        M.build(cfg, R.as_tensors(missing), n_ctx=256, n_seq_max=1, max_batch=16)
    later = R.make_config([R.attention_layer(kv_from=1, mlp=None), R.attention_layer(mlp=None)])
    with pytest.raises(B200Error, match="cache"):
        M.build(later, R.as_tensors(R.random_weights(later)), n_ctx=256, n_seq_max=1, max_batch=16)


# ------------------------------------------------------------------------------------------------ a model folder, the registry, the command line, the trace runner
def write_model_folder(path, cfg, W):
    import json
    import struct
    meta, blobs, at = {}, [], 0
    for name, (dt, shape, raw) in R.as_tensors(W).items():
        b = raw.tobytes()
        meta[name] = {"dtype": dt, "shape": list(shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b); at += len(b)
    head = json.dumps(meta).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    (path / "config.json").write_text(json.dumps(cfg))


def test_model_folder_command_line_and_trace_runner(tmp_path, capsys):
    import json
    import subprocess
    import sys
    from pathlib import Path
    from koboldcpp_b200 import __main__ as cli
    cfg = CONFIGS["mixed"]()
    W = R.random_weights(cfg, seed=2)
    write_model_folder(tmp_path, cfg, W)
    rng = np.random.default_rng(3)
    pa, pb = rng.integers(0, cfg["vocab"], 9).tolist(), rng.integers(0, cfg["vocab"], 4).tolist()
    # generate: greedy tokens of two prompts through registry, loader, engine and sampler
    assert cli.main(["generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6", "--prompt", ",".join(map(str, pa)), "--prompt", ",".join(map(str, pb))]) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.strip().splitlines() if x.startswith("{")]
    assert [x["prompt"] for x in lines] == [pa, pb]
    for x in lines:
        seq = list(x["prompt"])
        for tok in x["tokens"]:
            lg = R.logits(cfg, W, seq)[-1]
            top = np.sort(lg)[-2:]
            assert tok == int(np.argmax(lg)) or lg[tok] > top[1] - 1e-3 * (abs(top[1]) + 1)
            seq.append(tok)
    # the trace runner: two requests start together, decode together, the shorter one ends first
    ta, tb = rng.integers(0, cfg["vocab"], 14).tolist(), rng.integers(0, cfg["vocab"], 8).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ta[:11], "want": [0, 10]}, {"id": "y", "tokens": tb[:6], "want": [5]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ta[11:12], "want": []}, {"id": "y", "tokens": tb[6:7], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ta[12:13], "want": [0]}, {"id": "y", "tokens": tb[7:8], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": ta[13:14], "want": [0]}], "end": ["x"]}]
    out = tmp_path / "out"
    root = Path(__file__).resolve().parent.parent
    p = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
    wa, wb = R.logits(cfg, W, ta), R.logits(cfg, W, tb)
    want = {0: np.stack([wa[0], wa[10], wb[5]]), 1: wb[6:7], 2: np.stack([wa[12], wb[7]]), 3: wa[13:14]}
    for n, w in want.items():
        got = np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"])
        assert got.shape == w.shape and logits_err(got, w) < 1e-4, n
