"""Mafuzen in plain float64 numpy, one function per mechanism, written from the equations and sharing no code with the product
path.  Everything is token by token or dense and slow on purpose.

Notation: x is the residual stream [T, W]; N a layer norm with weight and bias.  A layer is
    x <- x + N1b(mixer(N1(x)));   x <- x + N2b(ff(N2(x)));   x <- x + rms(proj(gelu(gate x) * e)) * w_side
with e the layer's slice of a second embedding of the token.  The stream starts as scale * embed[token]; the logits are
embed (unscaled) times the final norm of the stream.

A `state` dict carries what a sequence needs to go on: per layer the cached keys and values, the recurrent states, the previous
token's input of a time-mixing layer, and the number of tokens seen.  forward() with a state continues that sequence.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def rms_unit(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    mean = x.mean(-1, keepdims=True)
    var = ((x - mean) ** 2).mean(-1, keepdims=True)
    return (x - mean) / np.sqrt(var + eps) * w + b


# ------------------------------------------------------------------------------------------------ retention
def rotate_halves(x, pos, dims, base):
    """x [T, heads, dim]: entry i turns with entry i + dims / 2 by the angle pos * base^(-2 i / dims); entries from dims on stay."""
    y = x.copy()
    half = dims // 2
    for t, p in enumerate(pos):
        for i in range(half):
            a = p * base ** (-2.0 * i / dims)
            u, v = x[t, :, i], x[t, :, i + half]
            y[t, :, i] = u * math.cos(a) - v * math.sin(a)
            y[t, :, i + half] = v * math.cos(a) + u * math.sin(a)
    return y


def retention_step(S, q, k, v, decay):
    """One token of one head, S [dim, vdim]: forget, write, read."""
    S = decay * S + np.outer(k, v)
    return S, S.T @ q


def retention_mixer(h, W, mx, eps, pos, st):
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = rotate_halves((h @ W["q"].T).reshape(T, H, D), pos, mx["rot"]["dims"], mx["rot"]["base"])
    k = rotate_halves((h @ W["k"].T).reshape(T, H, D), pos, mx["rot"]["dims"], mx["rot"]["base"]) * D ** -0.5
    v = (h @ W["v"].T).reshape(T, H, V)
    S = st.get("S", np.zeros((H, D, V))).copy()
    o = np.zeros((T, H, V))
    for t in range(T):
        for hh in range(H):
            S[hh], o[t, hh] = retention_step(S[hh], q[t, hh], k[t, hh], v[t, hh], mx["decay"][hh])
    st["S"] = S
    o = rms_unit(o, eps).reshape(T, H * V)
    return (o * silu(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ softmax attention
def slope(hh, H):
    return 2.0 ** (-8.0 * (hh + 1) / H)


def visible(i, j, window, keep_first):
    return j <= i and (window is None or i - j < window or j < keep_first)


def softmax_attention(q, k, v, pos_q, pos_k, scale, distance_bias=False, window=None, keep_first=0):
    """q [T, H, D]; k [N, G, D], v [N, G, V] everything cached including the new tokens.  Head h reads key / value head h // (H / G);
    with distance_bias the score of a key n positions back is lowered by slope_h * n."""
    T, H, _ = q.shape
    G = k.shape[1]
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        see = [n for n in range(k.shape[0]) if visible(pos_q[t], pos_k[n], window, keep_first)]
        for hh in range(H):
            kv = hh // (H // G)
            s = np.array([scale * (q[t, hh] @ k[n, kv]) - (slope(hh, H) * (pos_q[t] - pos_k[n]) if distance_bias else 0.0) for n in see])
            p = np.exp(s - s.max())
            p /= p.sum()
            for n, pn in zip(see, p):
                o[t, hh] += pn * v[n, kv]
    return o


def cached(st, name, new):
    st[name] = np.concatenate([st[name], new], 0) if name in st else new
    return st[name]


def attention_mixer(h, W, mx, pos, st, shared_from=None):
    """shared_from: the state of the layer whose keys and values this layer reads (it has none of its own then)."""
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = (h @ W["q"].T).reshape(T, H, D)
    if shared_from is None:
        cached(st, "k", (h @ W["k"].T).reshape(T, G, D))
        cached(st, "v", (h @ W["v"].T).reshape(T, G, V))
        cached(st, "pos", np.asarray(pos))
    src = st if shared_from is None else shared_from
    o = softmax_attention(q, src["k"], src["v"], pos, src["pos"], mx["scale"], distance_bias=True)
    return o.reshape(T, H * V) @ W["o"].T


def windowed_side(h, W, mx, eps, pos, st):
    """Keys and queries are unit-RMS per head; the values are the keys as projected; window with kept first tokens; output gate."""
    H, G, D = mx["heads"], mx["kv_heads"], mx["dim"]
    T = h.shape[0]
    q = rms_unit((h @ W["q"].T).reshape(T, H, D), eps)
    raw = (h @ W["k"].T).reshape(T, G, D)
    k, v, pk = cached(st, "k", rms_unit(raw, eps)), cached(st, "v", raw), cached(st, "pos", np.asarray(pos))
    o = softmax_attention(q, k, v, pos, pk, mx["scale"], window=mx["mask"]["size"], keep_first=mx["mask"]["keep_first"])
    return (o.reshape(T, H * D) * sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ time mixing
def token_shift(h, prev):
    """The previous token's row for every token: [prev, h_0, h_1, ...]."""
    return np.concatenate([prev[None], h[:-1]], 0)


def time_mix_step(S, r, k, v, w, u):
    """One token of one head, S [dim, vdim]: read with the bonus u on the current token, then forget per key channel and write."""
    o = (S + np.outer(u * k, v)).T @ r
    return w[:, None] * S + np.outer(k, v), o


def time_mix_side(h, W, mx, eps, st):
    H, D = mx["heads"], mx["dim"]
    T = h.shape[0]
    back = token_shift(h, st.get("prev", np.zeros(h.shape[1])))
    st["prev"] = h[-1].copy()
    mix = {s: h + (back - h) * W["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[s].T).reshape(T, H, D) for s in "rkv")
    gate = silu(mix["g"] @ W["g"].T)
    w = np.exp(-np.exp(np.tanh(mix["w"] @ W["w1"].T) @ W["w2"].T + W["w0"])).reshape(T, H, D)
    S = st.get("S", np.zeros((H, D, D))).copy()
    o = np.zeros((T, H, D))
    for t in range(T):
        for hh in range(H):
            S[hh], o[t, hh] = time_mix_step(S[hh], r[t, hh], k[t, hh], v[t, hh], w[t, hh], W["u"].reshape(H, D)[hh])
    st["S"] = S
    o = rms_unit(o, eps).reshape(T, H * D) * W["norm"] * gate
    return o @ W["o"].T


def parallel_mixer(h, W, mx, eps, pos, st):
    left = windowed_side(h, sub(W, "left."), mx["left"], eps, pos, st.setdefault("left", {}))
    right = time_mix_side(h, sub(W, "right."), mx["right"], eps, st.setdefault("right", {}))
    return mx["left_scale"] * left + mx["right_scale"] * right


# ------------------------------------------------------------------------------------------------ feed-forward
def dense(h, W):
    return (silu(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def expert(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def moe(h, W, mlp, tokens):
    """A table names every token id's experts; each has the weight 1 / top.  A shared expert runs for every token."""
    top = mlp["router"]["top"]
    out = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in np.asarray(W["table"])[tok]:
            out[t] += expert(h[t], W[f"e{int(e)}.up"], W[f"e{int(e)}.down"]) / top
    if mlp.get("shared"):
        out += expert(h, W["shared.up"], W["shared.down"])
    return out


# ------------------------------------------------------------------------------------------------ per-layer token input
def side_input(x, e, W, eps):
    y = (gelu_tanh(x @ W["gate"].T) * e) @ W["proj"].T
    return rms_unit(y, eps) * W["norm"]


# ------------------------------------------------------------------------------------------------ the model
def sub(W, prefix):
    return {k[len(prefix):]: v for k, v in W.items() if k.startswith(prefix)}


def layer(x, W, il, cfg, tokens, pos, states, side_embed):
    lc, eps = cfg["layers"][il], cfg["norm"]["eps"]
    mx, st = lc["mixer"], states.setdefault(il, {})
    h, mixW = layer_norm(x, W["norm1"], W["norm1.b"], eps), sub(W, "mix.")
    if lc["type"] == "attention":
        src = mx.get("kv_from")
        y = attention_mixer(h, mixW, mx, pos, st, None if src is None else states[src])
    elif lc["type"] == "retention":
        y = retention_mixer(h, mixW, mx, eps, pos, st)
    elif lc["type"] == "parallel":
        y = parallel_mixer(h, mixW, mx, eps, pos, st)
    else:
        raise ValueError(lc["type"])
    x = x + layer_norm(y, W["norm1b"], W["norm1b.b"], eps)
    mlp = lc.get("mlp")
    if mlp:
        h = layer_norm(x, W["norm2"], W["norm2.b"], eps)
        y = dense(h, sub(W, "mlp.")) if mlp["kind"] == "dense" else moe(h, sub(W, "mlp."), mlp, tokens)
        x = x + layer_norm(y, W["norm2b"], W["norm2b.b"], eps)
    if side_embed is not None:
        n = cfg["token_side"]["dim"]
        x = x + side_input(x, side_embed[np.asarray(tokens), il * n:(il + 1) * n], sub(W, "side."), eps)
    return x


def forward(cfg, weights, tokens, state=None, want_layers=False):
    """tokens: the next tokens of one sequence.  Returns logits [T, vocab] (and the stream after every layer) and the state."""
    W = {k: np.asarray(v) if k.endswith(".table") else np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    state = state if state is not None else {"n": 0, "layers": {}}
    pos = list(range(state["n"], state["n"] + len(tokens)))
    state["n"] += len(tokens)
    x = W["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    streams = []
    for il in range(len(cfg["layers"])):
        x = layer(x, sub(W, f"l{il}."), il, cfg, tokens, pos, state["layers"], W.get("side.embed") if cfg.get("token_side") else None)
        streams.append(x)
    logits = layer_norm(x, W["final.norm"], W["final.norm.b"], cfg["norm"]["eps"]) @ W["embed"].T
    if want_layers:
        return logits, np.stack(streams), state
    return logits, state


def logits(cfg, weights, tokens):
    return forward(cfg, weights, tokens)[0]


# ------------------------------------------------------------------------------------------------ small random models for the tests
def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16
    return u.astype(np.uint32).view(np.float32)


def dense_cfg(ff=40):
    return {"kind": "dense", "ff": ff}


def moe_cfg(ff=24, experts=6, top=2, shared=16):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def attention_layer(heads=4, kv_heads=2, dim=16, vdim=24, scale=None, kv_from=None, mlp="moe"):
    mx = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "attention", "mixer": mx, "mlp": moe_cfg() if mlp == "moe" else mlp}


def retention_layer(heads=3, dim=16, vdim=20, rot=8, base=1000.0, decay=None, mlp="moe"):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base},
                                           "decay": decay or [1.0 - 2.0 ** (-2 - i) for i in range(heads)]}, "mlp": moe_cfg() if mlp == "moe" else mlp}


def parallel_layer(heads=4, kv_heads=2, dim=16, size=11, keep_first=3, scale=None, mix_heads=3, mix_dim=12, left_scale=0.7, right_scale=1.3, mlp="moe"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size, "keep_first": keep_first}, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": left_scale, "right": {"heads": mix_heads, "dim": mix_dim}, "right_scale": right_scale},
            "mlp": moe_cfg() if mlp == "moe" else mlp}


def make_config(layers, width=40, vocab=61, eps=1e-5, embed_scale=3.0, side=12):
    return {"architecture": "Mafuzen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "token_side": {"dim": side} if side else None, "layers": layers}


def random_weights(cfg, seed=0, rank=5):
    """name -> float64 arrays whose values bfloat16 holds exactly (tables: int32), so that the served (bf16) and the exact (f32) modes
    read the same model."""
    rng = np.random.default_rng(seed)
    Wd, Vc = cfg["width"], cfg["vocab"]
    W = {}

    def mat(name, rows, cols, g=1.0):
        W[name] = bf16_round(rng.standard_normal((rows, cols)) * g / math.sqrt(cols)).astype(np.float64)

    def vec(name, n, mean=0.0, spread=0.3):
        W[name] = bf16_round(mean + spread * rng.standard_normal(n)).astype(np.float64)

    def norm(name):
        vec(name, Wd, 1.0, 0.2)
        vec(name + ".b", Wd, 0.0, 0.2)

    W["embed"] = bf16_round(rng.standard_normal((Vc, Wd)) / math.sqrt(Wd) * 3.0).astype(np.float64)
    norm("final.norm")
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        W["side.embed"] = bf16_round(rng.standard_normal((Vc, side * len(cfg["layers"])))).astype(np.float64)
    for il, L in enumerate(cfg["layers"]):
        p, mx = f"l{il}.", L["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if L["type"] == "attention":
            H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
            mat(p + "mix.q", H * D, Wd, 1.5)
            if mx.get("kv_from") is None:
                mat(p + "mix.k", G * D, Wd, 1.5)
                mat(p + "mix.v", G * V, Wd, 1.5)
            mat(p + "mix.o", Wd, H * V)
        elif L["type"] == "retention":
            H, D, V = mx["heads"], mx["dim"], mx["vdim"]
            for leaf, rows in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V)):
                mat(p + "mix." + leaf, rows, Wd, 1.5)
            mat(p + "mix.o", Wd, H * V)
        else:
            a, HR, DR = mx["left"], mx["right"]["heads"], mx["right"]["dim"]
            H, G, D = a["heads"], a["kv_heads"], a["dim"]
            mat(p + "mix.left.q", H * D, Wd, 1.5)
            mat(p + "mix.left.k", G * D, Wd, 1.5)
            mat(p + "mix.left.g", H * D, Wd, 1.5)
            mat(p + "mix.left.o", Wd, H * D)
            for s in "rkvgw":
                vec(p + "mix.right.mu." + s, Wd, 0.5, 0.3)
            for s in "rkvg":
                mat(p + "mix.right." + s, HR * DR, Wd, 1.5)
            mat(p + "mix.right.w1", rank, Wd, 1.0)
            mat(p + "mix.right.w2", HR * DR, rank, 1.0)
            vec(p + "mix.right.w0", HR * DR, -2.0, 1.5)
            W[p + "mix.right.u"] = bf16_round(rng.standard_normal((HR, DR))).astype(np.float64)
            vec(p + "mix.right.norm", HR * DR, 1.0, 0.3)
            mat(p + "mix.right.o", Wd, HR * DR)
        if side:
            mat(p + "side.gate", side, Wd, 1.5)
            mat(p + "side.proj", Wd, side)
            vec(p + "side.norm", Wd, 0.7, 0.3)
        mlp = L.get("mlp")
        if mlp is None:
            continue
        norm(p + "norm2")
        norm(p + "norm2b")
        if mlp["kind"] == "dense":
            mat(p + "mlp.gate", mlp["ff"], Wd, 1.5)
            mat(p + "mlp.up", mlp["ff"], Wd, 1.5)
            mat(p + "mlp.down", Wd, mlp["ff"])
            continue
        F, E, top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
        W[p + "mlp.table"] = np.stack([rng.permutation(E)[:top] for _ in range(Vc)]).astype(np.int32)
        for e in range(E):
            mat(p + f"mlp.e{e}.up", F, Wd, 1.5)
            mat(p + f"mlp.e{e}.down", Wd, F, 1.5)
        if mlp.get("shared"):
            mat(p + "mlp.shared.up", mlp["shared"]["ff"], Wd, 1.5)
            mat(p + "mlp.shared.down", Wd, mlp["shared"]["ff"], 1.5)
    return W


def as_tensors(W):
    """name -> (dtype, shape, raw bytes), the form the loader takes: matrices and vectors as bf16 bits, tables as int32."""
    out = {}
    for name, a in W.items():
        if a.dtype == np.int32:
            out[name] = ("I32", tuple(a.shape), np.ascontiguousarray(a).reshape(-1).view(np.uint8))
            continue
        bits = (np.ascontiguousarray(a, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)
        out[name] = ("BF16", tuple(a.shape), bits.view(np.uint8).reshape(-1))
    return out
