"""Tugezen: the reader of its config.json and weights behind the shared decoder (include/b200_llama.h).

A Tugezen model folder holds config.json ("architecture": "Tugezen", "width", "vocab", "norm": {"eps"}, "logit_scale", and "layers": a
list of {"type", "mixer": {...}, "mlp": {...} or null}) and model.safetensors (bfloat16 matrices named "embed", "head", "final.norm"
and "l<i>.<leaf>").  Three layer types: "latent_attention" (keys and values from one cached latent per token, a window, a gate per
head), "parallel" (soft-capped attention with YaRN rotation beside the gated delta rule with a decay per key channel) and "gla" (gated
linear attention).  The feed-forward is dense and gated.  The graph and the kernels live in the library (csrc/host_tugezen.cu); this
module translates the configuration into b200_layer_params and uploads the tensors under their own names.
"""
from __future__ import annotations

import json
from pathlib import Path

from .genesun import SequenceModel, read_safetensors, to_f32, upload
from .lib import BF16, F32, B200Error
from .llama import LayerParams

ARCH_TUGEZEN = 6
MIXER_LATENT_ATTENTION, MIXER_GATED_LINEAR_ATTENTION, MIXER_ATTENTION_DELTA = 1, 9, 10
MLP_NONE, MLP_DENSE_GATED = 0, 3
GLU_GELU_TANH = 1
ROPE_SCALING_NONE, ROPE_SCALING_YARN = 0, 1
# 2-D tensors that the library reads in f32 whatever the matrix type: convolution taps
F32_LEAVES = (".conv",)


def layer_params(layer: dict, decay_rank: int = 0, gate_rank: int = 0) -> LayerParams:
    """decay_rank, gate_rank: rows of the first matrices of the low-rank projections (the shapes of "a1" and "g1")."""
    mx = layer["mixer"]
    lp = LayerParams(kv_from=-1, decay_rank=decay_rank, gate_rank=gate_rank)
    kind = layer["type"]
    if kind == "latent_attention":
        lp.mixer = MIXER_LATENT_ATTENTION
        lp.heads, lp.dim, lp.vdim = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"])
        lp.q_rank, lp.kv_rank, lp.scale = int(mx["q_rank"]), int(mx["kv_rank"]), float(mx["scale"])
        lp.window, lp.head_gate = int((mx.get("mask") or {}).get("size", 0)), 1
    elif kind == "parallel":
        a, r = mx["left"], mx["right"]
        lp.mixer = MIXER_ATTENTION_DELTA
        lp.heads, lp.kv_heads, lp.dim, lp.vdim = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
        lp.scale, lp.attn_softcap = float(a["scale"]), float(a.get("softcap") or 0.0)
        rot = a.get("rot") or {}
        lp.rope_dims, lp.rope_base = int(rot.get("dims", 0)), float(rot.get("base", 1.0))
        sc = rot.get("scaling")
        if sc:
            lp.rope_scaling = ROPE_SCALING_YARN
            lp.yarn_factor, lp.yarn_original = float(sc["factor"]), int(sc["original"])
            lp.yarn_fast, lp.yarn_slow = float(sc["fast"]), float(sc["slow"])
        lp.mix_heads, lp.mix_kv_heads, lp.mix_dim, lp.mix_vdim = int(r["heads"]), int(r["kv_heads"]), int(r["dim"]), int(r["vdim"])
        lp.conv_taps = int(r["conv"])
        lp.left_scale, lp.right_scale = float(mx["left_scale"]), float(mx["right_scale"])
    elif kind == "gla":
        lp.mixer = MIXER_GATED_LINEAR_ATTENTION
        lp.heads, lp.dim, lp.vdim, lp.decay_tau = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"]), float(mx["tau"])
    else:
        raise B200Error(f"Tugezen: unknown layer type {kind!r}")
    mlp = layer.get("mlp")
    if mlp is None:
        lp.mlp, lp.ff = MLP_NONE, 0
    elif mlp.get("kind", "dense") == "dense":
        lp.mlp, lp.ff, lp.glu_kind = MLP_DENSE_GATED, int(mlp["ff"]), GLU_GELU_TANH
    else:
        raise B200Error(f"Tugezen: unknown feed-forward kind {mlp.get('kind')!r}")
    return lp


def build(config: dict, tensors, dtype: str = "bfloat16", n_ctx: int = 4096, n_seq_max: int = 16, max_batch: int = 512, device: int = 0) -> SequenceModel:
    """config: the parsed config.json; tensors: name -> (dtype, shape, raw bytes)."""
    if dtype not in ("bfloat16", "float32"):
        raise B200Error(f"dtype {dtype!r}: bfloat16 or float32")

    def rows(*names):
        return next((int(tensors[n][1][0]) for n in names if n in tensors), 0)

    layers = [layer_params(x, rows(f"l{i}.mix.a1", f"l{i}.mix.right.a1"), rows(f"l{i}.mix.right.g1")) for i, x in enumerate(config["layers"])]
    model = SequenceModel(ARCH_TUGEZEN, int(config["width"]), int(config["vocab"]), layers, float(config["norm"]["eps"]), n_ctx, n_seq_max, max_batch, device,
                          logit_scale=float(config.get("logit_scale", 1.0)))
    matrix_type = BF16 if dtype == "bfloat16" else F32
    for name, (dt, shape, raw) in tensors.items():
        if name.endswith(F32_LEAVES):
            model.set_tensor(name, F32, shape, to_f32(dt, raw))
        else:
            upload(model, name, dt, shape, raw, matrix_type)
    model.finalize()
    return model


def load(path, **kw) -> SequenceModel:
    path = Path(path)
    config = json.loads((path / "config.json").read_text())
    return build(config, read_safetensors(path / "model.safetensors"), **kw)
