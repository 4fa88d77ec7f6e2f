"""Mafuzen: the reader of its config.json and weights behind the shared decoder (include/b200_llama.h).

A Mafuzen model folder holds config.json ("architecture": "Mafuzen", "width", "vocab", "norm": {"eps"}, "embedding": {"scale"},
"token_side": {"dim"} or null, and "layers": a list of {"type", "mixer": {...}, "mlp": {...} or null}) and model.safetensors
(bfloat16 matrices named "embed", "final.norm", "side.embed" and "l<i>.<leaf>", int32 tables).  Three layer types: "attention" (a
score penalty that grows with the distance; a layer may read an earlier layer's cache), "retention" (linear attention with a fixed
decay per head) and "parallel" (windowed attention whose values are its keys, beside time mixing).  The feed-forward is dense and
gated, or a mixture of experts that a table names by token id, plus a shared expert.  The output head is the embedding table.  The
graph and the kernels live in the library (csrc/host_mafuzen.cu); this module translates the configuration into b200_layer_params
and uploads the tensors under their own names.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np

from .genesun import SequenceModel, read_safetensors, to_f32, upload
from .lib import BF16, F32, I32, B200Error
from .llama import LayerParams

ARCH_MAFUZEN = 5
MIXER_ATTENTION, MIXER_RETENTION, MIXER_WINDOW_ATTENTION_TIME_MIX = 3, 7, 8
MLP_NONE, MLP_DENSE_GATED, MLP_MOE_TABLE = 0, 3, 4
GLU_SILU = 0
DIST_SLOPE_EXP = 8.0  # head h of H takes 2^(-8 (h + 1) / H) per position of distance off its scores
# 2-D tensors that the library reads in f32 whatever the matrix type
F32_LEAVES = (".right.u", "side.embed")


def layer_params(layer: dict, token_side: int = 0) -> LayerParams:
    mx = layer["mixer"]
    lp = LayerParams(kv_from=-1, token_side=token_side)
    kind = layer["type"]
    if kind == "attention":
        lp.mixer = MIXER_ATTENTION
        lp.heads, lp.kv_heads, lp.dim, lp.vdim = int(mx["heads"]), int(mx["kv_heads"]), int(mx["dim"]), int(mx["vdim"])
        lp.scale, lp.dist_slope_exp = float(mx["scale"]), DIST_SLOPE_EXP
        lp.kv_from = -1 if mx.get("kv_from") is None else int(mx["kv_from"])
    elif kind == "retention":
        lp.mixer = MIXER_RETENTION
        lp.heads, lp.dim, lp.vdim = int(mx["heads"]), int(mx["dim"]), int(mx["vdim"])
        rot = mx.get("rot") or {}
        lp.rope_dims, lp.rope_base, lp.rope_halves = int(rot.get("dims", 0)), float(rot.get("base", 1.0)), 1
        if len(mx["decay"]) != lp.heads:
            raise B200Error(f"Mafuzen: {len(mx['decay'])} decays for {lp.heads} heads")
    elif kind == "parallel":
        a, r = mx["left"], mx["right"]
        lp.mixer = MIXER_WINDOW_ATTENTION_TIME_MIX
        lp.heads, lp.kv_heads, lp.dim, lp.vdim = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a.get("vdim", a["dim"]))
        if lp.vdim != lp.dim:
            raise B200Error(f"Mafuzen: the values of a parallel layer are its keys, so vdim {lp.vdim} must be dim {lp.dim}")
        mask = a.get("mask") or {}
        lp.scale, lp.window, lp.keep_first = float(a["scale"]), int(mask.get("size", 0)), int(mask.get("keep_first", 0))
        lp.mix_heads, lp.mix_dim = int(r["heads"]), int(r["dim"])
        lp.left_scale, lp.right_scale = float(mx["left_scale"]), float(mx["right_scale"])
    else:
        raise B200Error(f"Mafuzen: unknown layer type {kind!r}")
    mlp = layer.get("mlp")
    if mlp is None:
        lp.mlp, lp.ff = MLP_NONE, 0
    elif mlp.get("kind", "dense") == "dense":
        lp.mlp, lp.ff, lp.glu_kind = MLP_DENSE_GATED, int(mlp["ff"]), GLU_SILU
    elif mlp["kind"] == "moe":
        lp.mlp, lp.ff = MLP_MOE_TABLE, int(mlp["expert"]["ff"])
        lp.n_expert, lp.n_expert_used = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
        lp.shared_ff = int((mlp.get("shared") or {}).get("ff", 0))
    else:
        raise B200Error(f"Mafuzen: unknown feed-forward kind {mlp.get('kind')!r}")
    return lp


def build(config: dict, tensors, dtype: str = "bfloat16", n_ctx: int = 4096, n_seq_max: int = 16, max_batch: int = 512, device: int = 0) -> SequenceModel:
    """config: the parsed config.json; tensors: name -> (dtype, shape, raw bytes)."""
    if dtype not in ("bfloat16", "float32"):
        raise B200Error(f"dtype {dtype!r}: bfloat16 or float32")
    side = int((config.get("token_side") or {}).get("dim", 0))
    layers = [layer_params(x, side) for x in config["layers"]]
    model = SequenceModel(ARCH_MAFUZEN, int(config["width"]), int(config["vocab"]), layers, float(config["norm"]["eps"]), n_ctx, n_seq_max, max_batch, device,
                          embed_scale=float((config.get("embedding") or {}).get("scale", 1.0)))
    matrix_type = BF16 if dtype == "bfloat16" else F32
    for i, layer in enumerate(config["layers"]):
        if layer["type"] == "retention":
            decay = np.asarray(layer["mixer"]["decay"], dtype=np.float32)
            model.set_tensor(f"l{i}.mix.decay", F32, decay.shape, decay)
    for name, (dt, shape, raw) in tensors.items():
        if name.endswith(".table"):
            if dt != "I32":
                raise B200Error(f"Mafuzen: {name} must hold int32 expert numbers, not {dt}")
            model.set_tensor(name, I32, shape, raw.view(np.int32))
        elif name.endswith(F32_LEAVES):
            model.set_tensor(name, F32, shape, to_f32(dt, raw))
        else:
            upload(model, name, dt, shape, raw, matrix_type)
            if name == "embed":  # the output head is the table as stored (the library multiplies its own copy by the embedding scale)
                upload(model, "head", dt, shape, raw, matrix_type)
    model.finalize()
    return model


def load(path, **kw) -> SequenceModel:
    path = Path(path)
    config = json.loads((path / "config.json").read_text())
    return build(config, read_safetensors(path / "model.safetensors"), **kw)
