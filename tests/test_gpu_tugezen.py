"""Tugezen on the GPU against the plain float64 statement in tugezen_ref.py: every mechanism alone through the C ABI, then whole
models through the loader, the batch step, the sequence cache and the engine (prefill against decoding, portions, mixed batches,
cells and slots that are used again, far keys and window edges, greedy generation)."""
from __future__ import annotations

import ctypes as C
import math

import numpy as np
import pytest

import koboldcpp_b200.host as H
import tugezen_ref as R
from koboldcpp_b200.lib import F32, DeltaRuleArgs, LatentAttnArgs, LinearAttnArgs, NormChainArgs, QkvStoreArgs, ShortConvArgs, SinkAttnArgs, Tensor, check, lib

pytestmark = pytest.mark.gpu


def dev(a, dtype=np.float32):
    return H.DeviceBuffer.from_numpy(np.ascontiguousarray(a, dtype=dtype), pad=256)


def rel(got, want):
    return float(np.abs(got - want).max() / (np.abs(want).max() + 1e-30))


def seq_info(runs):
    """runs: [(first token, count, slot, fresh)] -> the int32 [4][n] table the scans read."""
    return np.array(runs, dtype=np.int32).T.copy()


# ------------------------------------------------------------------------------------------------ norms, activation
@pytest.mark.parametrize("n,T", [(40, 3), (61, 4), (1030, 2), (4096, 3), (13001, 1)])
def test_residual_without_a_norm_behind_the_sublayer_then_the_next_norm(n, T):
    """x = res + y; h = x / rms(x) * w; a residual far louder than the sublayer's result must keep every digit of it."""
    rng = np.random.default_rng(n)
    row = n + (n % 4 == 0) * 4 + (n % 4 != 0) * 3
    y, res, w, eps = rng.standard_normal((T, row)) * 1e-3, rng.standard_normal((T, row)) * 30 + 100, rng.standard_normal(n), 1e-4
    dy, dr, dw, out = dev(y), dev(res), dev(w), H.DeviceBuffer(4 * 2 * T * row + 256)
    a = NormChainArgs(y=dy.ptr, y_s_slot=row, y_s_tok=row, res=dr.ptr, res_stride=row, w2=dw.ptr, x=out.ptr, x_stride=row, h=out.ptr + 4 * T * row, h_stride=row, n=n, n_tok=T, n_y=1,
                      kind1=2, kind2=1, eps=eps)
    check(lib().b200_op_norm_chain(C.byref(a), None))
    got = out.to_numpy(np.float32, (2, T, row))[:, :, :n]
    assert (got[0] == y.astype(np.float32)[:, :n] + res.astype(np.float32)[:, :n]).all()
    assert rel(got[1], R.rms_norm((y + res)[:, :n], w, eps)) < 3e-6


@pytest.mark.parametrize("V,Hh,T,gate", [(13, 4, 5, 1), (64, 3, 9, 1), (128, 2, 3, 2), (300, 3, 2, 2)])
def test_head_norm_with_one_weight_for_all_heads_and_a_gate(V, Hh, T, gate):
    rng = np.random.default_rng(V)
    x, z, w, eps = rng.standard_normal((T, Hh, V)) * 3, rng.standard_normal((T, Hh, V)) * 2, 1 + 0.3 * rng.standard_normal(V), 1e-5
    x[:, 0] *= 50.0  # a loud head must not move the others
    row = Hh * V + 5
    zbuf, dx, dw, dout = np.zeros((T, row)), dev(x), dev(w), H.DeviceBuffer(4 * T * row + 256)
    zbuf[:, 2:2 + Hh * V] = z.reshape(T, -1)
    dz = dev(zbuf)
    tx, tz, to = Tensor.contiguous(dx.ptr, F32, (V, Hh, T)), Tensor.contiguous(dz.ptr + 8, F32, (V, Hh, T)), Tensor.contiguous(dout.ptr, F32, (V, Hh, T))
    tz.nb[2] = to.nb[2] = 4 * row
    check(lib().b200_op_norm_affine(C.byref(tx), dw.ptr, 1, None, C.byref(tz), None, gate, None, C.byref(to), eps, 1, None))
    got = dout.to_numpy(np.float32, (T, row))[:, :Hh * V].reshape(T, Hh, V)
    want = R.rms_norm(x, w, eps) * (R.sigmoid(z) if gate == 1 else R.silu(z))
    for h in range(Hh):
        assert rel(got[:, h], want[:, h]) < 3e-6


@pytest.mark.parametrize("F,T,kind", [(37, 3, 1), (64, 3, 1), (1028, 2, 1), (2052, 3, 0), (36, 2, 2)])
def test_gated_activation_rows_of_four_and_others(F, T, kind):
    """The tanh form of gelu (1), and the other kinds through the same forms, over the halves of one product."""
    a, b = np.linspace(-9, 9, T * F).reshape(T, F), np.random.default_rng(0).standard_normal((T, F)) * 3
    gu, out = dev(np.concatenate([a, b], 1)), H.DeviceBuffer(4 * a.size + 256)
    ta, tb, to = Tensor.contiguous(gu.ptr, F32, (F, T)), Tensor.contiguous(gu.ptr + 4 * F, F32, (F, T)), Tensor.contiguous(out.ptr, F32, (F, T))
    ta.nb[1] = tb.nb[1] = 8 * F
    check(lib().b200_op_glu_strided(kind, C.byref(ta), C.byref(tb), C.byref(to), 5.0, 1.5, None))
    g, u = np.minimum(a, 5.0), np.clip(b, -5.0, 5.0)
    want = (R.silu(a) * b, R.gelu_tanh(a) * b, g * R.sigmoid(1.5 * g) * (u + 1.0))[kind]
    assert rel(out.to_numpy(np.float32, (T, F)), want) < 2e-6


# ------------------------------------------------------------------------------------------------ recurrences
@pytest.mark.parametrize("ch,taps,portions", [(5, 1, [7]), (130, 2, [1, 1, 3, 40, 16, 1]), (40, 4, [1, 2, 1, 30]), (33, 9, [2, 2, 20, 1])])
def test_short_convolution_whole_and_in_portions(ch, taps, portions):
    """Portions shorter than the filter, stale values in every slot, a second sequence in another slot beside it."""
    rng = np.random.default_rng(ch)
    T, slot = sum(portions), max(taps - 1, 1) * ch + 2
    x, w, other = rng.standard_normal((T, ch)), rng.standard_normal((ch, taps)), rng.standard_normal((2, ch))
    tail, dw, got, done = dev(np.full((3, slot), 9.0)), dev(w), np.zeros((T, ch)), 0
    for n in portions:
        dx, dy, info = dev(np.concatenate([other, x[done:done + n]])), H.DeviceBuffer(4 * (n + 2) * ch + 256), dev(seq_info([(0, 2, 0, 1), (2, n, 2, 1 if done == 0 else 0)]), np.int32)
        a = ShortConvArgs(x=dx.ptr, x_stride=ch, w=dw.ptr, seq_info=info.ptr, n_seq=2, tail=tail.ptr, slot_stride=slot, dst=dy.ptr, dst_stride=ch, channels=ch, taps=taps, act=1, n_tokens=n + 2)
        check(lib().b200_op_short_conv(C.byref(a), None))
        got[done:done + n] = dy.to_numpy(np.float32, (n + 2, ch))[2:]
        done += n
    assert rel(got, R.silu(R.short_conv(x, w, {}, "t"))) < 2e-6


def run_delta(q, k, v, z, b, A_log, dt_bias, portions):
    """q, k [T, G, D]; v [T, H, V]; z [T, H, D]; b [T, H]: one sequence in portions in slot 1 of 2, the other slot and this one full of stale values."""
    T, G, D = q.shape
    Hh, V = v.shape[1:]
    slot = Hh * D * V + 4
    state, dA, dt = dev(np.full((2, slot), 5.0)), dev(A_log), dev(dt_bias)
    out, done = np.zeros((T, Hh, V)), 0
    for n in portions:
        sl = slice(done, done + n)
        dq, dk, dv, dz, db = (dev(x[sl].reshape(n, -1)) for x in (q, k, v, z, b))
        dy, info = H.DeviceBuffer(4 * n * Hh * V + 256), dev(seq_info([(0, n, 1, 1 if done == 0 else 0)]), np.int32)
        a = DeltaRuleArgs(q=dq.ptr, k=dk.ptr, v=dv.ptr, q_stride=G * D, k_stride=G * D, v_stride=Hh * V, a=dz.ptr, b=db.ptr, a_stride=Hh * D, b_stride=Hh, a_log=dA.ptr, dt_bias=dt.ptr,
                          seq_info=info.ptr, n_seq=1, state=state.ptr, slot_stride=slot, dst=dy.ptr, dst_stride=Hh * V, heads=Hh, kv_heads=G, dim=D, vdim=V, unit_qk=1, unit_eps=1e-6,
                          q_scale=D ** -0.5, channel_decay=1)
        check(lib().b200_op_delta_rule_scan(C.byref(a), None))
        out[sl] = dy.to_numpy(np.float32, (n, Hh, V))
        done += n
    assert (state.to_numpy(np.float32, (2, slot))[0] == 5.0).all()
    return out


def delta_reference(q, k, v, z, b, A_log, dt_bias):
    T, G, D = q.shape
    Hh, V = v.shape[1:]
    g, beta, q, k = R.delta_decay(z, A_log, dt_bias), R.sigmoid(b), R.unit(q) * D ** -0.5, R.unit(k)
    S, out = np.zeros((Hh, D, V)), np.zeros((T, Hh, V))
    for t in range(T):
        for h in range(Hh):
            S[h], out[t, h] = R.delta_step(S[h], q[t, h // (Hh // G)], k[t, h // (Hh // G)], v[t, h], g[t, h], beta[t, h])
    return out


@pytest.mark.parametrize("Hh,G,D,V,portions", [(4, 2, 9, 13, [1, 1, 2, 17, 16, 1]), (3, 3, 32, 40, [37]), (6, 1, 64, 20, [20, 3, 16]), (2, 2, 128, 70, [33, 1, 1]), (2, 1, 200, 33, [19, 1]),
                                               (1, 1, 1, 1, [5, 2])])
def test_delta_rule_with_a_decay_per_channel_whole_and_in_portions(Hh, G, D, V, portions):
    rng = np.random.default_rng(D + V)
    T = sum(portions)
    q, k, v, z, b = (rng.standard_normal(s) for s in ((T, G, D), (T, G, D), (T, Hh, V), (T, Hh, D), (T, Hh)))
    A_log, dt_bias = rng.uniform(-3, 0.5, Hh), rng.uniform(-4, 1, (Hh, D))
    want = delta_reference(q, k, v, z, b, A_log, dt_bias)
    assert rel(run_delta(q, k, v, z, b, A_log, dt_bias, portions), want) < 2e-5
    assert rel(run_delta(q, k, v, z, b, A_log, dt_bias, [T]), want) < 2e-5


def test_delta_rule_keeps_one_channel_and_loses_another():
    """Two values written along two key channels; hundreds of tokens later (which write nothing) the channel without decay still gives its
    value, the other one gives none, and a channel written again holds the new value only."""
    D, V, T = 8, 8, 400
    q, k, v, z, b = np.zeros((T, 1, D)), np.zeros((T, 1, D)), np.zeros((T, 1, V)), np.full((T, 1, D), -60.0), np.full((T, 1), -200.0)
    z[:, 0, 5] = 1.0
    k[0, 0, 2], k[1, 0, 5], b[:2] = 1.0, 1.0, 200.0
    v[0, 0], v[1, 0] = np.arange(V), 1.0 + np.arange(V)
    k[2:, 0, 7] = 1.0
    q[:, 0, 7] = 1.0
    q[390], q[391] = 0.0, 0.0
    q[390, 0, 2], q[391, 0, 5] = 1.0, 1.0
    k[392], b[392], v[392], q[392] = k[0], 200.0, -3.0, q[390]
    got = run_delta(q, k, v, z, b, np.zeros(1), np.zeros((1, D)), [150, 1, T - 151]) * math.sqrt(D)
    assert np.abs(got[390, 0] - np.arange(V)).max() < 1e-4 and np.abs(got[391, 0]).max() < 1e-4 and np.abs(got[392, 0] + 3.0).max() < 1e-4


def run_gla(q, k, v, z, bias, tau, portions):
    T, Hh, D = q.shape
    V = v.shape[2]
    slot = Hh * D * V + 8
    state, db = dev(np.full((2, slot), 5.0)), dev(bias)
    out, done = np.zeros((T, Hh, V)), 0
    for n in portions:
        sl = slice(done, done + n)
        dq, dk, dv, dz = (dev(x[sl].reshape(n, -1)) for x in (q, k, v, z))
        dy, info = H.DeviceBuffer(4 * n * Hh * V + 256), dev(seq_info([(0, n, 1, 1 if done == 0 else 0)]), np.int32)
        a = LinearAttnArgs(q=dq.ptr, k=dk.ptr, v=dv.ptr, q_stride=Hh * D, k_stride=Hh * D, v_stride=Hh * V, z=dz.ptr, z_stride=Hh * D, z_bias=db.ptr, tau=tau, seq_info=info.ptr, n_seq=1,
                           state=state.ptr, slot_stride=slot, dst=dy.ptr, dst_stride=Hh * V, heads=Hh, dim=D, vdim=V, k_scale=D ** -0.5)
        check(lib().b200_op_linear_attn_scan(C.byref(a), None))
        out[sl] = dy.to_numpy(np.float32, (n, Hh, V))
        done += n
    assert (state.to_numpy(np.float32, (2, slot))[0] == 5.0).all()
    return out


@pytest.mark.parametrize("Hh,D,V,tau,portions", [(3, 11, 8, 4.0, [1, 1, 2, 17, 16, 1]), (2, 32, 40, 16.0, [37]), (1, 64, 20, 1.0, [20, 3]), (2, 128, 70, 8.0, [33, 1, 1]), (2, 200, 9, 2.0, [19, 1, 9])])
def test_gated_linear_attention_whole_and_in_portions(Hh, D, V, tau, portions):
    rng = np.random.default_rng(D + V)
    T = sum(portions)
    q, k, v, z, bias = (rng.standard_normal(s) for s in ((T, Hh, D), (T, Hh, D), (T, Hh, V), (T, Hh, D), (Hh, D)))
    z, bias = z * 4, bias * 3  # fast and slow channels; |z| far beyond where a sigmoid rounds to one
    alpha = R.sigmoid(z + bias) ** (1.0 / tau)
    S, want = np.zeros((Hh, D, V)), np.zeros((T, Hh, V))
    for t in range(T):
        for h in range(Hh):
            S[h], want[t, h] = R.gla_step(S[h], q[t, h] * D ** -0.5, k[t, h], v[t, h], alpha[t, h])
    assert rel(run_gla(q, k, v, z, bias, tau, portions), want) < 2e-5
    assert rel(run_gla(q, k, v, z, bias, tau, [T]), want) < 2e-5


def test_gated_linear_attention_slow_channel_remembers_the_first_token():
    """exp(-softplus(-z) / tau) with z = 9 forgets 1 - 1e-4 / tau per token: 500 tokens on, the first value is damped by exactly that power;
    a pre-activation of -400 forgets at once without turning into NaN."""
    D, V, T, tau = 4, 3, 501, 2.0
    q, k, v, z = np.zeros((T, 1, D)), np.zeros((T, 1, D)), np.zeros((T, 1, V)), np.full((T, 1, D), 9.0)
    z[:, 0, 1] = -400.0
    k[0, 0, :2], v[0, 0], q[-1, 0, 0], q[-2, 0, 1] = 1.0, [1.0, 2.0, -3.0], 2.0, 1.0
    got = run_gla(q, k, v, z, np.zeros((1, D)), tau, [300, 201])
    assert rel(got[-1, 0], np.array([1.0, 2.0, -3.0]) * R.sigmoid(9.0) ** (500 / tau)) < 1e-4 and (got[-2] == 0.0).all()


# ------------------------------------------------------------------------------------------------ attention
def scattered_cache(rng, n_cells, lens, *widths):
    """Sequences of the given lengths shuffled into one cache; free cells hold NaN."""
    total = sum(lens)
    order = rng.permutation(n_cells)[:total]
    cell_seq, cell_pos = np.full(n_cells, -1), np.full(n_cells, -1)
    at = 0
    for s, n in enumerate(lens):
        cell_seq[order[at:at + n]], cell_pos[order[at:at + n]] = s, np.arange(n)
        at += n
    caches = []
    for w in widths:
        c = np.full((n_cells, w), np.nan)
        c[order] = rng.standard_normal((total, w))
        caches.append(c)
    return cell_seq, cell_pos, *caches


def rows_of_sequence(cell_seq, cell_pos, s, n):
    return [int(np.where((cell_seq == s) & (cell_pos == j))[0][0]) for j in range(n)]


def run_attn(q, kc, vc, cell_seq, cell_pos, tok_seq, tok_pos, scale, G, softcap=0.0, out_scale=0.0, bf16=0):
    T, Hh, D = q.shape
    V = vc.shape[1] // G
    bufs = [dev(q), dev(kc), dev(vc), dev(cell_seq, np.int32), dev(cell_pos, np.int32), dev(tok_seq, np.int32), dev(tok_pos, np.int32)]
    row = Hh * V + 3
    out = dev(np.full((T, row), 7.0))
    a = SinkAttnArgs(q=bufs[0].ptr, q_stride=Hh * D, k_cache=bufs[1].ptr, k_cache_stride=kc.shape[1], v_cache=bufs[2].ptr, v_cache_stride=vc.shape[1], cell_seq=bufs[3].ptr,
                     cell_pos=bufs[4].ptr, tok_seq=bufs[5].ptr, tok_pos=bufs[6].ptr, dst=out.ptr, dst_stride=row, n_head=Hh, n_head_kv=G, dim=D, vdim=V, n_tokens=T, n_kv=len(cell_seq),
                     scale=scale, bf16_products=bf16, out_scale=out_scale, softcap=softcap)
    need = int(lib().b200_sink_attn_workspace_bytes(C.byref(a)))
    ws = H.DeviceBuffer(need + 256) if need else None
    check(lib().b200_op_sink_attn_ws(C.byref(a), ws.ptr if ws else None, need, None))
    full = out.to_numpy(np.float32, (T, row))
    assert (full[:, Hh * V:] == 7.0).all()
    return full[:, :Hh * V].reshape(T, Hh, V)


@pytest.mark.parametrize("Hh,G,D,V,cap", [(4, 2, 16, 24, 3.0), (6, 3, 40, 40, 0.5), (1, 1, 200, 33, 30.0), (3, 1, 32, 32, 0.0)])
@pytest.mark.parametrize("n_cells", [96, 2304])
def test_soft_capped_attention_single_tokens_scattered_cells_two_sequences(Hh, G, D, V, cap, n_cells):
    """The decode form (split over CTAs at 2304 cells), scores far beyond the cap."""
    rng = np.random.default_rng(Hh + D)
    lens = (41, 52)
    cell_seq, cell_pos, kc, vc = scattered_cache(rng, n_cells, lens, G * D, G * V)
    toks = [(0, 40), (1, 51), (0, 0), (1, 7), (0, 2), (1, 20)]
    q, scale, f = rng.standard_normal((len(toks), Hh, D)), 4.0 / math.sqrt(D), 0.6
    for sel in ([0], list(range(len(toks)))):
        got = run_attn(q[sel], kc, vc, cell_seq, cell_pos, [toks[i][0] for i in sel], [toks[i][1] for i in sel], scale, G, cap, f)
        for r, i in enumerate(sel):
            s, p = toks[i]
            idx = rows_of_sequence(cell_seq, cell_pos, s, p + 1)
            want = R.softmax_attention(q[i:i + 1], kc[idx].reshape(-1, G, D), vc[idx].reshape(-1, G, V), [p], np.arange(p + 1), scale, cap)[0]
            assert rel(got[r], want * f) < 2e-5, (i, s, p)


@pytest.mark.parametrize("Hh,G,D,V,T,cap", [(4, 2, 16, 24, 70, 2.0), (2, 2, 64, 64, 129, 8.0), (3, 1, 40, 72, 33, 0.7), (1, 1, 128, 128, 64, 50.0), (2, 1, 150, 20, 40, 5.0)])
@pytest.mark.parametrize("bf16", [0, 1])
def test_soft_capped_attention_prompt_batches_behind_cached_tokens(Hh, G, D, V, T, cap, bf16):
    rng = np.random.default_rng(T)
    P0, Lb = 23, 30
    cell_seq, cell_pos, kc, vc = scattered_cache(rng, 256, [Lb, P0 + T], G * D, G * V)
    q, scale = rng.standard_normal((T, Hh, D)), 3.0 / math.sqrt(D)
    pos = list(range(P0, P0 + T))
    got = run_attn(q, kc, vc, cell_seq, cell_pos, [1] * T, pos, scale, G, cap, 1.5, bf16)
    idx = rows_of_sequence(cell_seq, cell_pos, 1, P0 + T)
    src = (lambda a: R.bf16_round(a).astype(np.float64)) if bf16 else (lambda a: a)
    want = R.softmax_attention(src(q), src(kc[idx]).reshape(-1, G, D), src(vc[idx]).reshape(-1, G, V), pos, np.arange(P0 + T), scale, cap) * 1.5
    assert rel(got, want) < (1e-2 if bf16 else 2e-5)


@pytest.mark.parametrize("T,bf16", [(1, 0), (40, 0), (40, 1)])
@pytest.mark.parametrize("score", [1e-3, 40.0, -40.0, 1e4])
def test_cap_against_one_loud_key(T, bf16, score):
    """One far key of 700 with a score from tiny to absurd: its weight follows from the capped score, not from the score."""
    rng = np.random.default_rng(5)
    D, V, n, cap = 32, 16, 700, 9.0
    q, k, v, p = np.zeros((T, 1, D)), np.zeros((n, D)), rng.standard_normal((n, V)), n - 1
    q[:, 0, 3], k[37, 3] = 1.0, score
    v[37] *= 30
    got = run_attn(q, k, v, np.zeros(n, dtype=np.int64), np.arange(n), [0] * T, [p] * T, 1.0, 1, cap, bf16=bf16)
    e = np.where(np.arange(n) == 37, math.exp(cap * math.tanh(score / cap)), 1.0)
    want = (e / e.sum()) @ v
    assert np.abs(got[:, 0] - want).max() < (0.2 if bf16 else 1e-4)


@pytest.mark.parametrize("Hh,G,D,V,dims,scaling,pos0", [(4, 2, 12, 10, 8, R.YARN, 0), (2, 1, 64, 16, 64, {"factor": 3.0, "original": 100, "fast": 20.0, "slow": 1.5}, 1500), (3, 3, 20, 7, 20, None, 9)])
def test_store_with_interleaved_rotation_and_a_factor(Hh, G, D, V, dims, scaling, pos0):
    rng = np.random.default_rng(D)
    T, n_cells = 5, 16
    q, k, v = rng.standard_normal((T, Hh, D)), rng.standard_normal((T, G, D)), rng.standard_normal((T, G, V))
    pos, cells = np.arange(T) + pos0, np.array([5, 0, 15, 7, 2])
    freqs, mag = R.yarn_frequencies(dims, 300.0, scaling)
    dq, dk, dv, dp, dc, df = dev(q), dev(k), dev(v), dev(pos, np.int32), dev(cells, np.int32), dev(freqs)
    kc, vc = dev(np.full((n_cells, G * D), 7.0)), dev(np.full((n_cells, G * V), 7.0))
    a = QkvStoreArgs(q=dq.ptr, q_stride=Hh * D, k=dk.ptr, k_stride=G * D, v=dv.ptr, v_stride=G * V, pos=dp.ptr, cells=dc.ptr, freqs=df.ptr, k_cache=kc.ptr, k_cache_stride=G * D,
                     v_cache=vc.ptr, v_cache_stride=G * V, n_head=Hh, n_head_kv=G, dim=D, vdim=V, n_dims=dims, n_tokens=T, rope_mscale=mag if scaling else 0.0)
    check(lib().b200_op_qkv_store(C.byref(a), None))
    tol = 2e-6 + 2e-7 * pos0  # the angle is a 32-bit product
    assert rel(dq.to_numpy(np.float32, (T, Hh, D)), R.rotate_pairs(q, pos, dims, freqs, mag)) < tol
    kk, vv = kc.to_numpy(np.float32, (n_cells, G, D)), vc.to_numpy(np.float32, (n_cells, G, V))
    assert rel(kk[cells], R.rotate_pairs(k, pos, dims, freqs, mag)) < tol and (vv[cells] == v.astype(np.float32)).all()
    assert (np.delete(kk, cells, 0) == 7.0).all() and (np.delete(vv, cells, 0) == 7.0).all()


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("KR,QR,T", [(18, 20, 3), (64, 7, 100), (300, 500, 1), (513, 128, 70)])
def test_latent_store_norms_both_latents(KR, QR, T):
    rng = np.random.default_rng(KR)
    row, n_cells, eps, lead = KR + QR + 9, T + 20, 1e-4, 3
    x, w, wq = rng.standard_normal((T, row)) * 5, rng.standard_normal(KR), rng.standard_normal(QR)
    cells = rng.permutation(n_cells)[:T]
    dx, dw, dwq, dc, cache = dev(x), dev(w), dev(wq), dev(cells, np.int32), dev(np.full((n_cells, KR + 4), 7.0))
    check(lib().b200_op_latent_store(dx.ptr + 4 * (lead + QR), row, dw.ptr, None, None, dc.ptr, cache.ptr, KR + 4, KR, 0, 0, 1.0, eps, dx.ptr + 4 * lead, row, dwq.ptr, QR, T, None))
    c, y = cache.to_numpy(np.float32, (n_cells, KR + 4)), dx.to_numpy(np.float32, (T, row))
    assert rel(c[cells, :KR], R.rms_norm(x[:, lead + QR:lead + QR + KR], w, eps)) < 3e-6 and rel(y[:, lead:lead + QR], R.rms_norm(x[:, lead:lead + QR], wq, eps)) < 3e-6
    y[:, lead:lead + QR] = x[:, lead:lead + QR]
    assert (y == x.astype(np.float32)).all() and (np.delete(c, cells, 0) == 7.0).all() and (c[:, KR:] == 7.0).all()


def run_latent(q, cache, cell_seq, cell_pos, tok_seq, tok_pos, scale, window, gate, bf16=0):
    """q [T, H, KR] against the latent rows; returns [T, H, KR]."""
    T, Hh, KR = q.shape
    bufs = [dev(q), dev(cache), dev(cell_seq, np.int32), dev(cell_pos, np.int32), dev(tok_seq, np.int32), dev(tok_pos, np.int32)]
    row = Hh + 3
    gbuf = np.zeros((T, row)); gbuf[:, 1:1 + Hh] = gate
    dg, out = dev(gbuf), H.DeviceBuffer(4 * T * Hh * KR + 256)
    a = LatentAttnArgs(q_lat=bufs[0].ptr, q_lat_s_head=KR, q_lat_s_tok=Hh * KR, cache=bufs[1].ptr, cache_stride=KR, cell_seq=bufs[2].ptr, cell_pos=bufs[3].ptr, tok_seq=bufs[4].ptr,
                       tok_pos=bufs[5].ptr, dst=out.ptr, dst_s_head=T * KR, dst_s_tok=KR, kv_rank=KR, rot_dim=0, n_head=Hh, n_tokens=T, n_kv=len(cell_seq), window=window, scale=scale,
                       bf16_products=bf16, gate=dg.ptr + 4, gate_stride=row)
    check(lib().b200_op_latent_attn(C.byref(a), None))
    return out.to_numpy(np.float32, (Hh, T, KR)).transpose(1, 0, 2)


@pytest.mark.parametrize("KR,Hh,T,window,bf16", [(18, 3, 1, 9, 0), (18, 3, 100, 9, 0), (64, 5, 50, 33, 0), (64, 5, 50, 33, 1), (128, 2, 77, 1, 1), (80, 8, 130, 16, 1), (512, 2, 20, 0, 1), (130, 9, 40, 17, 0),
                                                  (64, 40, 60, 20, 0)])
def test_latent_attention_with_window_and_head_gate(KR, Hh, T, window, bf16):
    """A portion of T tokens behind cached ones, beside a second sequence in the same cache, free cells hold NaN."""
    rng = np.random.default_rng(KR + T)
    P0 = 23
    cell_seq, cell_pos, cache = scattered_cache(rng, 256, [30, P0 + T], KR)
    q, gate, scale = rng.standard_normal((T, Hh, KR)), rng.standard_normal((T, Hh)) * 2, 1.5 / math.sqrt(KR)
    pos = list(range(P0, P0 + T))
    got = run_latent(q, cache, cell_seq, cell_pos, [1] * T, pos, scale, window, gate, bf16)
    rows = cache[rows_of_sequence(cell_seq, cell_pos, 1, P0 + T)]
    if bf16:
        q, rows = (R.bf16_round(x).astype(np.float64) for x in (q, rows))
    want = R.softmax_attention(q, rows[:, None], rows[:, None], pos, np.arange(P0 + T), scale, window=window or None) * R.sigmoid(gate)[:, :, None]
    assert rel(got, want) < (1e-2 if bf16 else 2e-5)


@pytest.mark.parametrize("T,bf16", [(1, 0), (40, 0), (40, 1)])
def test_latent_attention_one_loud_key_at_the_window_edges(T, bf16):
    """One latent stands out: at the own position and just inside the window it is the result, one token further back it is not seen."""
    KR, n, window = 32, 700, 50
    p = n - 1
    q = np.zeros((T, 1, KR)); q[:, 0, 3] = 1.0
    base = np.random.default_rng(1).standard_normal((n, KR)); base[:, 3] = 0.0
    for loud, seen in ((p, True), (p - 1, True), (p - window + 1, True), (p - window, False), (0, False), (300, False)):
        cache = base.copy(); cache[loud, 3] = 60.0
        got = run_latent(q, cache, np.zeros(n, dtype=np.int64), np.arange(n), [0] * T, [p] * T, 1.0, window, np.zeros((T, 1)), bf16)
        want = 0.5 * (cache[loud] if seen else base[p - window + 1:].mean(0))
        assert np.abs(got[:, 0] - want).max() < (2e-2 if bf16 else 1e-4), loud


# ------------------------------------------------------------------------------------------------ whole models
from koboldcpp_b200 import tugezen as M  # noqa: E402
from koboldcpp_b200.engine import Engine, Request  # noqa: E402

CONFIGS = {
    # every kind of layer, with and without a feed-forward, a window shorter than the prompts, partial rotation
    "mixed": lambda: R.make_config([R.latent_layer(), R.parallel_layer(), R.gla_layer(mlp=None), R.parallel_layer(heads=2, kv_heads=2, d_heads=2, d_kv=2, scaling=None, conv=2, mlp=None),
                                    R.latent_layer(heads=2, size=33, mlp=None)]),
    # a parallel layer first; one head, one kv head, a window of one token, no window, a convolution of one tap and a long one, no rotated entries, tau
    # and scales of exactly one, no soft cap, a ramp that no pair lies on, sizes of one, a width that is no multiple of 8
    "odd": lambda: R.make_config([R.parallel_layer(heads=1, kv_heads=1, dim=10, vdim=3, rot=0, softcap=None, d_heads=5, d_kv=1, d_dim=1, d_vdim=6, conv=1, left_scale=1.0, right_scale=1.0, mlp=R.dense_cfg(7)),
                                  R.latent_layer(heads=1, dim=7, vdim=1, q_rank=5, kv_rank=3, size=1, mlp=None), R.gla_layer(heads=1, dim=24, vdim=40, tau=1.0),
                                  R.parallel_layer(heads=6, kv_heads=3, dim=6, rot=6, scaling={"factor": 1.0, "original": 7, "fast": 1.0, "slow": 1.0}, d_heads=1, d_kv=1, d_dim=20, d_vdim=1, conv=9, mlp=None),
                                  R.latent_layer(heads=9, dim=4, vdim=5, q_rank=33, kv_rank=40, size=0)], width=70, vocab=70, eps=1e-6, logit_scale=1.0),
    # sizes that take the 16-byte and tensor-core paths
    "aligned": lambda: R.make_config([R.parallel_layer(heads=4, kv_heads=2, dim=32, vdim=64, rot=32, base=1e4, softcap=4.0, d_heads=4, d_kv=2, d_dim=32, d_vdim=64, mlp=R.dense_cfg(128)),
                                      R.gla_layer(heads=4, dim=64, vdim=32, tau=8.0, mlp=R.dense_cfg(64)),
                                      R.latent_layer(heads=4, dim=64, vdim=64, q_rank=64, kv_rank=128, size=24, scale=0.25, mlp=R.dense_cfg(192)),
                                      R.parallel_layer(heads=2, kv_heads=1, dim=128, vdim=32, rot=64, d_heads=2, d_kv=2, d_dim=64, d_vdim=32, conv=3, mlp=R.dense_cfg(64))], width=128, vocab=96, logit_scale=0.5),
}


@pytest.fixture(scope="module", params=list(CONFIGS))
def model(request):
    cfg = CONFIGS[request.param]()
    W = R.random_weights(cfg, seed=len(request.param), rank_a=32 if request.param == "aligned" else 5)
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
    recurrent states and the last inputs of the convolutions with what it left there) go to a new request that joins while the others decode."""
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
    """bf16 serving mode: prompt portions of 16 tokens or more take the tensor-core kernels (attention and dense products), over
    cells that earlier portions wrote and beside another request's tokens; shorter portions and single tokens take the f32 kernels.
    All of them must give the logits of the float64 reference up to bf16 rounding."""
    cfg = CONFIGS[name]()
    W = R.random_weights(cfg, seed=5, rank_a=32 if name == "aligned" else 5)
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
    """Large score scales make the attention sharp, so a wrong position, frequency, window edge or cell would show in the logits; the
    windows' edges pass over prompt and decoded tokens, the prompt's end is no multiple of any block size, and the decoded stretch crosses
    the cache padding.  Slow decays keep the first tokens alive in the states."""
    cfg = R.make_config([R.latent_layer(heads=2, dim=16, size=100, scale=2.0, mlp=None), R.parallel_layer(heads=2, kv_heads=1, dim=16, rot=16, base=5e3, scale=2.5, softcap=20.0, mlp=None),
                         R.latent_layer(heads=2, size=17, scale=3.0), R.gla_layer(heads=2, tau=64.0, mlp=None), R.parallel_layer(heads=2, kv_heads=2, dim=8, rot=4, scale=3.0, softcap=30.0)])
    W = R.random_weights(cfg, seed=21)
    for il in (1, 4):
        W[f"l{il}.mix.right.dt_bias"] = R.bf16_round(W[f"l{il}.mix.right.dt_bias"] - 4.0).astype(np.float64)
    toks = np.random.default_rng(2).integers(0, cfg["vocab"], 290).tolist()
    want = R.logits(cfg, W, toks)
    m = M.build(cfg, R.as_tensors(W), dtype="float32", n_ctx=512, n_seq_max=2, max_batch=300)
    eng = Engine(m)
    places = [0, 1, 2, 3, 4, 15, 16, 17, 18, 98, 99, 100, 101, 200, 241]
    rows = [eng.step([("a", toks[:242], places)])]
    for t in range(242, 290):
        rows.append(eng.step([("a", [toks[t]], [0])])); places.append(t)
    m.close()
    assert logits_err(np.concatenate(rows), want[places]) < 2e-4


def test_a_changed_first_token_reaches_the_last_logits():
    """Windows end after a few tokens, so only the full attention and the states can carry the first token 300 positions; all of it must
    arrive, in the prompt and in decoding."""
    cfg = R.make_config([R.latent_layer(size=3, mlp=None), R.gla_layer(tau=500.0, mlp=None), R.parallel_layer(scale=0.02, mlp=None)])
    W = R.random_weights(cfg, seed=8)
    W["l1.mix.a2.b"][:] = 4.0
    W["l2.mix.right.dt_bias"][:] = -8.0
    toks = np.random.default_rng(3).integers(1, cfg["vocab"], 300).tolist()
    other = [0] + toks[1:]
    m = M.build(cfg, R.as_tensors(W), dtype="float32", n_ctx=512, n_seq_max=2, max_batch=300)
    eng = Engine(m)
    got = {}
    for name, t in (("p", toks), ("o", other)):
        eng.step([(name, t[:290], [])])
        got[name] = np.concatenate([eng.step([(name, [x], [0])]) for x in t[290:]])
        eng.finish(name)
    m.close()
    wp, wo = R.logits(cfg, W, toks)[290:], R.logits(cfg, W, other)[290:]
    assert np.abs(wp - wo).max() > 1e-3  # the two differ by far more than rounding ...
    assert np.abs((got["p"] - got["o"]) - (wp - wo)).max() < 2e-2 * np.abs(wp - wo).max()  # ... and by the right amount


def test_tensors_in_any_order():
    cfg = CONFIGS["mixed"]()
    W = R.random_weights(cfg, seed=4)
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 12).tolist()
    rng = np.random.default_rng(0)
    t = R.as_tensors(W)
    for _ in range(2):
        names = [list(t)[i] for i in rng.permutation(len(t))]
        m = M.build(cfg, {n: t[n] for n in names}, dtype="float32", n_ctx=256, n_seq_max=1, max_batch=16)
        got = Engine(m).step([("a", toks, range(12))])
        m.close()
        assert logits_err(got, R.logits(cfg, W, toks)) < 1e-4


def test_loader_refuses_what_does_not_fit():
    from koboldcpp_b200.lib import B200Error
    cfg = R.make_config([R.latent_layer(mlp=None), R.parallel_layer(), R.gla_layer(mlp=None)])
    W = R.random_weights(cfg)
    for name in ("l0.mix.dq.norm", "l0.mix.g", "l1.mix.right.q.conv", "l1.mix.right.g2", "l1.mix.left.o", "l1.mix.right.norm", "l1.mlp.gate", "l2.mix.a2.b", "l2.norm1", "final.norm", "head"):
        with pytest.raises(B200Error, match=name.split(".", 1)[-1]):
            M.build(cfg, R.as_tensors({k: v for k, v in W.items() if k != name}), n_ctx=256, n_seq_max=1, max_batch=16)
    bad = dict(W); bad["l1.mix.right.k"] = W["l1.mix.right.k"][:-1]
    with pytest.raises(B200Error, match="right.k"):
        M.build(cfg, R.as_tensors(bad), n_ctx=256, n_seq_max=1, max_batch=16)
    odd = R.make_config([R.parallel_layer(heads=4, kv_heads=3)])
    with pytest.raises(B200Error, match="kv heads"):
        M.build(odd, R.as_tensors(R.random_weights(odd)), n_ctx=256, n_seq_max=1, max_batch=16)


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
