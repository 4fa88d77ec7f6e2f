"""Mafuzen without a GPU: configuration -> layer parameters, the registry, and the oracle's own consistency (a continued sequence
against the whole one, window and kept first tokens, slopes, rotation of halves, the recurrences as explicit sums)."""
from __future__ import annotations

import numpy as np
import pytest

import mafuzen_ref as R
from koboldcpp_b200 import mafuzen
from koboldcpp_b200.lib import B200Error
from koboldcpp_b200.models import ARCHITECTURES


def test_registry_knows_the_architecture():
    assert ARCHITECTURES["Mafuzen"] is mafuzen.load


def test_layer_parameters_from_the_configuration():
    a = mafuzen.layer_params(R.attention_layer(heads=6, kv_heads=3, dim=24, vdim=8, scale=0.3, mlp=R.dense_cfg(50)), token_side=7)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.kv_from, a.window, a.token_side) == (mafuzen.MIXER_ATTENTION, 6, 3, 24, 8, -1, 0, 7)
    assert (a.mlp, a.ff, a.glu_kind, a.dist_slope_exp) == (mafuzen.MLP_DENSE_GATED, 50, mafuzen.GLU_SILU, 8.0) and abs(a.scale - 0.3) < 1e-7
    b = mafuzen.layer_params(R.attention_layer(kv_from=0, mlp=None))
    assert (b.kv_from, b.mlp, b.token_side) == (0, mafuzen.MLP_NONE, 0)
    r = mafuzen.layer_params(R.retention_layer(heads=2, dim=18, vdim=30, rot=10, base=500.0, mlp=R.moe_cfg(ff=44, experts=9, top=4, shared=0)))
    assert (r.mixer, r.heads, r.dim, r.vdim, r.rope_dims, r.rope_base, r.rope_halves) == (mafuzen.MIXER_RETENTION, 2, 18, 30, 10, 500.0, 1)
    assert (r.mlp, r.ff, r.n_expert, r.n_expert_used, r.shared_ff) == (mafuzen.MLP_MOE_TABLE, 44, 9, 4, 0)
    p = mafuzen.layer_params(R.parallel_layer(heads=2, kv_heads=1, dim=20, size=9, keep_first=2, mix_heads=5, mix_dim=14, left_scale=0.25, right_scale=1.5, mlp=R.moe_cfg(shared=33)))
    assert (p.mixer, p.heads, p.kv_heads, p.dim, p.vdim, p.window, p.keep_first) == (mafuzen.MIXER_WINDOW_ATTENTION_TIME_MIX, 2, 1, 20, 20, 9, 2)
    assert (p.mix_heads, p.mix_dim, p.left_scale, p.right_scale, p.shared_ff, p.dist_slope_exp) == (5, 14, 0.25, 1.5, 33, 0.0)


def test_configurations_that_do_not_fit_are_refused():
    with pytest.raises(B200Error):
        mafuzen.layer_params(R.retention_layer(heads=3, decay=[0.5, 0.5]))
    bad = R.parallel_layer()
    bad["mixer"]["left"]["vdim"] = 8
    with pytest.raises(B200Error):
        mafuzen.layer_params(bad)
    with pytest.raises(B200Error):
        mafuzen.layer_params(dict(R.attention_layer(), type="something"))


def test_window_and_kept_first_tokens():
    see = [j for j in range(12) if R.visible(9, j, 4, 2)]
    assert see == [0, 1, 6, 7, 8, 9]  # 9 - 6 = 3 < 4 is inside, 9 - 5 = 4 is not
    assert [j for j in range(5) if R.visible(2, j, 1, 0)] == [2] and [j for j in range(5) if R.visible(2, j, None, 0)] == [0, 1, 2]


def test_slopes_halve_between_heads_of_a_set_of_eight():
    assert [R.slope(h, 8) for h in range(8)] == [2.0 ** -(h + 1) for h in range(8)]
    assert R.slope(0, 1) == 2.0 ** -8 and abs(R.slope(1, 3) - 2.0 ** (-16 / 3)) < 1e-15


def test_rotation_keeps_lengths_and_depends_on_differences():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 1, 12)), rng.standard_normal((1, 1, 12))
    dot = lambda i, j: float((R.rotate_halves(q, [i], 8, 100.0) * R.rotate_halves(k, [j], 8, 100.0)).sum())
    assert abs(dot(7, 3) - dot(24, 20)) < 1e-9 and abs(dot(7, 3) - dot(7, 4)) > 1e-3
    assert np.allclose(R.rotate_halves(q, [5], 8, 100.0)[..., 8:], q[..., 8:])


def test_retention_and_time_mix_as_explicit_sums():
    rng = np.random.default_rng(1)
    T, D, V = 7, 4, 3
    q, k, v, w, u = (rng.standard_normal(s) for s in ((T, D), (T, D), (T, V), (T, D), (D,)))
    w = 1.0 / (1.0 + np.exp(-w))
    S = np.zeros((D, V))
    for t in range(T):
        S, o = R.retention_step(S, q[t], k[t], v[t], 0.8)
        assert np.allclose(o, sum(0.8 ** (t - j) * (q[t] @ k[j]) * v[j] for j in range(t + 1)))
    S = np.zeros((D, V))
    for t in range(T):
        S, o = R.time_mix_step(S, q[t], k[t], v[t], w[t], u)
        want = (q[t] @ (u * k[t])) * v[t] + sum((q[t] @ (np.prod(w[j + 1:t], axis=0) * k[j])) * v[j] for j in range(t))
        assert np.allclose(o, want)


def test_table_experts_have_equal_weights():
    rng = np.random.default_rng(2)
    mlp = R.moe_cfg(ff=6, experts=4, top=3, shared=0)
    W = {f"e{e}.{n}": rng.standard_normal(s) for e in range(4) for n, s in (("up", (6, 5)), ("down", (5, 6)))}
    W["table"] = np.array([[0, 1, 2], [3, 1, 0]], dtype=np.int32)
    h = rng.standard_normal((2, 5))
    got = R.moe(h, W, mlp, [1, 0])
    assert np.allclose(got[0], sum(R.expert(h[0], W[f"e{e}.up"], W[f"e{e}.down"]) for e in (3, 1, 0)) / 3)


def test_continued_sequence_equals_the_whole_one():
    cfg = R.make_config([R.attention_layer(), R.retention_layer(mlp=R.dense_cfg()), R.parallel_layer(size=4, keep_first=1), R.attention_layer(kv_from=0, mlp=None)])
    W = R.random_weights(cfg, seed=3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 17).tolist()
    whole = R.logits(cfg, W, toks)
    a, st = R.forward(cfg, W, toks[:5])
    b, st = R.forward(cfg, W, toks[5:6], st)
    c, st = R.forward(cfg, W, toks[6:], st)
    assert np.allclose(np.concatenate([a, b, c]), whole, atol=1e-9)
