"""Tugezen without a GPU: configuration -> layer parameters, the registry, and the oracle's own consistency (a continued sequence
against the whole one, windows, YaRN's two ends, the recurrences as explicit sums)."""
from __future__ import annotations

import math

import numpy as np
import pytest

import tugezen_ref as R
from koboldcpp_b200 import tugezen
from koboldcpp_b200.lib import B200Error
from koboldcpp_b200.models import ARCHITECTURES


def test_registry_knows_the_architecture():
    assert ARCHITECTURES["Tugezen"] is tugezen.load


def test_layer_parameters_from_the_configuration():
    a = tugezen.layer_params(R.latent_layer(heads=6, dim=24, vdim=8, q_rank=30, kv_rank=22, size=77, scale=0.3, mlp=R.dense_cfg(50)))
    assert (a.mixer, a.heads, a.dim, a.vdim, a.q_rank, a.kv_rank, a.rot_dim, a.window, a.head_gate) == (tugezen.MIXER_LATENT_ATTENTION, 6, 24, 8, 30, 22, 0, 77, 1)
    assert (a.mlp, a.ff, a.glu_kind) == (tugezen.MLP_DENSE_GATED, 50, tugezen.GLU_GELU_TANH) and abs(a.scale - 0.3) < 1e-7
    assert tugezen.layer_params(R.latent_layer(size=0)).window == 0
    g = tugezen.layer_params(R.gla_layer(heads=2, dim=18, vdim=30, tau=12.0, mlp=None), decay_rank=9)
    assert (g.mixer, g.heads, g.dim, g.vdim, g.decay_tau, g.decay_rank, g.mlp) == (tugezen.MIXER_GATED_LINEAR_ATTENTION, 2, 18, 30, 12.0, 9, tugezen.MLP_NONE)
    p = tugezen.layer_params(R.parallel_layer(heads=6, kv_heads=3, dim=20, vdim=14, rot=10, base=500.0, softcap=7.5, d_heads=8, d_kv=4, d_dim=9, d_vdim=11, conv=5, left_scale=0.25,
                                              right_scale=1.5), decay_rank=3, gate_rank=4)
    assert (p.mixer, p.heads, p.kv_heads, p.dim, p.vdim, p.rope_dims, p.rope_base, p.attn_softcap) == (tugezen.MIXER_ATTENTION_DELTA, 6, 3, 20, 14, 10, 500.0, 7.5)
    assert (p.rope_scaling, p.yarn_factor, p.yarn_original, p.yarn_fast, p.yarn_slow, p.window) == (tugezen.ROPE_SCALING_YARN, 5.0, 40, 9.0, 0.5, 0)
    assert (p.mix_heads, p.mix_kv_heads, p.mix_dim, p.mix_vdim, p.conv_taps, p.left_scale, p.right_scale, p.decay_rank, p.gate_rank) == (8, 4, 9, 11, 5, 0.25, 1.5, 3, 4)
    q = tugezen.layer_params(R.parallel_layer(scaling=None, softcap=None))
    assert (q.rope_scaling, q.attn_softcap) == (tugezen.ROPE_SCALING_NONE, 0.0)


def test_unknown_kinds_are_refused():
    with pytest.raises(B200Error):
        tugezen.layer_params(dict(R.gla_layer(), type="something"))
    with pytest.raises(B200Error):
        tugezen.layer_params(R.gla_layer(mlp={"kind": "moe"}))


def test_window_counts_the_token_itself():
    assert [j for j in range(12) if R.visible(9, j, 4)] == [6, 7, 8, 9] and [j for j in range(5) if R.visible(2, j, 1)] == [2] and [j for j in range(5) if R.visible(2, j)] == [0, 1, 2]


def test_yarn_keeps_fast_pairs_and_divides_slow_ones():
    f, mag = R.yarn_frequencies(32, 1e4, {"factor": 4.0, "original": 256, "fast": 16.0, "slow": 1.0})
    plain, one = R.yarn_frequencies(32, 1e4, None)
    # a pair turns original f / (2 pi) times within the original length
    turns = [256 * p / (2 * math.pi) for p in plain]
    assert all(abs(a - b) < 1e-15 for a, b, t in zip(f, plain, turns) if t > 30) and all(abs(a - b / 4) < 1e-15 for a, b, t in zip(f, plain, turns) if t < 0.5)
    assert all(b / 4 - 1e-15 <= a <= b + 1e-15 for a, b in zip(f, plain)) and (mag, one) == (0.1 * math.log(4.0) + 1.0, 1.0)


def test_soft_cap_bounds_scores_and_leaves_small_ones():
    s = np.array([-1e6, -0.01, 0.0, 0.01, 1e6])
    assert np.allclose(R.capped(s, 5.0), [-5.0, -0.01, 0.0, 0.01, 5.0], atol=1e-6) and (R.capped(s, None) == s).all()


def test_gated_linear_attention_as_an_explicit_sum():
    rng = np.random.default_rng(1)
    T, D, V = 7, 4, 3
    q, k, v, a = (rng.standard_normal(s) for s in ((T, D), (T, D), (T, V), (T, D)))
    a = R.sigmoid(a)
    S = np.zeros((D, V))
    for t in range(T):
        S, o = R.gla_step(S, q[t], k[t], v[t], a[t])
        assert np.allclose(o, sum((q[t] @ (np.prod(a[j + 1:t + 1], axis=0) * k[j])) * v[j] for j in range(t + 1)))


def test_delta_rule_writes_what_is_missing():
    """With strength one and a unit key the state gives the value back at that key, whatever it held; strength zero writes nothing."""
    rng = np.random.default_rng(2)
    S, k, v = rng.standard_normal((5, 3)), R.unit(rng.standard_normal(5)), rng.standard_normal(3)
    S1, o = R.delta_step(S, k, k, v, np.ones(5), 1.0)
    assert np.allclose(o, v, atol=1e-5)
    g = rng.uniform(0, 1, 5)
    S2, _ = R.delta_step(S1, k, k, v, g, 0.0)
    assert np.allclose(S2, g[:, None] * S1)


def test_convolution_looks_back_only():
    w = np.array([[1.0, 10.0, 100.0]])
    x = np.array([[1.0], [2.0], [3.0], [4.0]])
    st = {}
    assert R.short_conv(x[:1], w, st, "t").ravel().tolist() == [100.0] and R.short_conv(x[1:], w, st, "t").ravel().tolist() == [210.0, 321.0, 432.0]


def test_continued_sequence_equals_the_whole_one():
    cfg = R.make_config([R.latent_layer(size=4), R.parallel_layer(), R.gla_layer(mlp=None), R.parallel_layer(conv=1, mlp=None)])
    W = R.random_weights(cfg, seed=3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 17).tolist()
    whole = R.logits(cfg, W, toks)
    a, st = R.forward(cfg, W, toks[:5])
    b, st = R.forward(cfg, W, toks[5:6], st)
    c, st = R.forward(cfg, W, toks[6:], st)
    assert np.allclose(np.concatenate([a, b, c]), whole, atol=1e-9)
