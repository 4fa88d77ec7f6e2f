"""Tugezen in plain float64 numpy, one function per mechanism, written from the equations and sharing no code with the product
path.  Everything is token by token or dense and slow on purpose.

Notation: x is the residual stream [T, W]; N(z) = z / sqrt(mean(z^2) + eps) * w.  A layer is
    x <- x + mixer(N1(x));   x <- x + down(gelu(gate h) * up h) with h = N2(x)   (the second step may be absent)
The stream starts as embed[token]; the logits are logit_scale * head N_final(x).

A `state` dict carries what a sequence needs to go on: per layer the cached keys and values (or latents), the recurrent states, the last
inputs of the convolutions, and the number of tokens seen.  forward() with a state continues that sequence.
"""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def keep(st, name, new):
    """Append to what the state holds under this name; returns everything."""
    st[name] = np.concatenate([st[name], new], 0) if name in st else new
    return st[name]


# ------------------------------------------------------------------------------------------------ rotation
def yarn_frequencies(dims, base, scaling):
    """Per pair base^(-2 i / dims), blended with the same divided by the factor: pairs that turn often within the original length keep
    theirs, pairs that turn rarely take the divided one.  Returns the frequencies and the factor on sine and cosine."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    s, orig = scaling["factor"], scaling["original"]

    def place(turns):
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s * ramp + fi * (1.0 - ramp))
    return out, 0.1 * math.log(s) + 1.0


def rotate_pairs(x, pos, dims, freqs, magnitude):
    """x [T, heads, dim]: entries 2 i and 2 i + 1 turn by pos * freqs[i] and are multiplied by the magnitude; entries from dims on stay."""
    y = x.copy()
    for t, p in enumerate(pos):
        for i in range(dims // 2):
            c, s = math.cos(p * freqs[i]) * magnitude, math.sin(p * freqs[i]) * magnitude
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            y[t, :, 2 * i] = u * c - v * s
            y[t, :, 2 * i + 1] = v * c + u * s
    return y


# ------------------------------------------------------------------------------------------------ softmax attention
def capped(s, cap):
    return cap * np.tanh(s / cap) if cap else s


def visible(i, j, window=None):
    return j <= i and (window is None or i - j < window)


def softmax_attention(q, k, v, pos_q, pos_k, scale, softcap=None, window=None):
    """q [T, H, D]; k [N, G, D], v [N, G, V] everything cached including the new tokens.  Head h reads key / value head h // (H / G)."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        see = [n for n in range(k.shape[0]) if visible(pos_q[t], pos_k[n], window)]
        for hh in range(H):
            s = capped(scale * (k[see, hh // group] @ q[t, hh]), softcap)
            p = np.exp(s - s.max())
            o[t, hh] = (p / p.sum()) @ v[see, hh // group]
    return o


def attention_side(h, W, mx, pos, st):
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    rot = mx.get("rot") or {"dims": 0, "base": 1.0}
    freqs, mag = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    q = rotate_pairs((h @ W["q"].T).reshape(T, H, D), pos, rot["dims"], freqs, mag)
    k = keep(st, "k", rotate_pairs((h @ W["k"].T).reshape(T, G, D), pos, rot["dims"], freqs, mag))
    v = keep(st, "v", (h @ W["v"].T).reshape(T, G, V))
    return softmax_attention(q, k, v, pos, np.arange(len(k)), mx["scale"], mx.get("softcap")).reshape(T, H * V) @ W["o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def latent_attention_mixer(h, W, mx, eps, pos, st):
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q = (rms_norm(h @ W["dq"].T, W["dq.norm"], eps) @ W["uq"].T).reshape(T, H, D)
    c = keep(st, "c", rms_norm(h @ W["dkv"].T, W["dkv.norm"], eps))
    k, v = (c @ W["uk"].T).reshape(-1, H, D), (c @ W["uv"].T).reshape(-1, H, V)
    o = softmax_attention(q, k, v, pos, np.arange(len(c)), mx["scale"], window=(mx.get("mask") or {}).get("size"))
    return (o * sigmoid(h @ W["g"].T)[:, :, None]).reshape(T, H * V) @ W["o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule
def short_conv(x, w, st, name):
    """x [T, channels], w [channels, taps] (the last column meets the current token): zeros stand before the start, the last taps - 1
    inputs stay in the state."""
    taps = w.shape[1]
    past = st.get(name, np.zeros((taps - 1, x.shape[1])))
    full = np.concatenate([past, x], 0)
    st[name] = full[len(full) - (taps - 1):]
    return np.stack([(full[t:t + taps] * w.T).sum(0) for t in range(len(x))])


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_decay(z, A_log, dt_bias):
    """z, dt_bias [.., heads, dim], A_log [heads]: the factor each key channel's row of the state is multiplied by."""
    return np.exp(-np.exp(A_log)[:, None] * softplus(z + dt_bias))


def delta_step(S, q, k, v, g, beta):
    """One token of one head, S [dim, vdim]: forget per key channel, correct towards v along k, read."""
    S = g[:, None] * S
    u = beta * (v - S.T @ k)
    S = S + np.outer(k, u)
    return S, S.T @ q


def delta_side(h, W, mx, eps, st):
    H, G, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ W[n].T, W[n + ".conv"], st, n + ".tail")) for n in "qkv")
    q, k, v = unit(q.reshape(T, G, D)) * D ** -0.5, unit(k.reshape(T, G, D)), v.reshape(T, H, V)
    beta = sigmoid(h @ W["b"].T)
    g = delta_decay((h @ W["a1"].T @ W["a2"].T).reshape(T, H, D), W["A_log"], W["dt_bias"].reshape(H, D))
    S = st.get("S", np.zeros((H, D, V))).copy()
    o = np.zeros((T, H, V))
    for t in range(T):
        for hh in range(H):
            S[hh], o[t, hh] = delta_step(S[hh], q[t, hh // (H // G)], k[t, hh // (H // G)], v[t, hh], g[t, hh], beta[t, hh])
    st["S"] = S
    o = rms_norm(o, W["norm"], eps) * sigmoid(h @ W["g1"].T @ W["g2"].T).reshape(T, H, V)
    return o.reshape(T, H * V) @ W["o"].T


def sub(W, prefix):
    return {n[len(prefix):]: w for n, w in W.items() if n.startswith(prefix)}


def parallel_mixer(h, W, mx, eps, pos, st):
    return (mx["left_scale"] * attention_side(h, sub(W, "left."), mx["left"], pos, st.setdefault("left", {})) +
            mx["right_scale"] * delta_side(h, sub(W, "right."), mx["right"], eps, st.setdefault("right", {})))


# ------------------------------------------------------------------------------------------------ gated linear attention
def gla_step(S, q, k, v, alpha):
    """One token of one head, S [dim, vdim]: forget per key channel, write, read."""
    S = alpha[:, None] * S + np.outer(k, v)
    return S, S.T @ q


def gla_mixer(h, W, mx, eps, st):
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    T = h.shape[0]
    q, k, v = ((h @ W[n].T).reshape(T, H, -1) for n in "qkv")
    alpha = (sigmoid(h @ W["a1"].T @ W["a2"].T + W["a2.b"]) ** (1.0 / mx["tau"])).reshape(T, H, D)
    S = st.get("S", np.zeros((H, D, V))).copy()
    o = np.zeros((T, H, V))
    for t in range(T):
        for hh in range(H):
            S[hh], o[t, hh] = gla_step(S[hh], q[t, hh] * D ** -0.5, k[t, hh], v[t, hh], alpha[t, hh])
    st["S"] = S
    return (rms_norm(o, W["norm"], eps).reshape(T, H * V) * silu(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------------------------------------ the model
def feed_forward(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def forward(cfg, W, tokens, state=None, want_layers=False):
    """Logits of every token, (the stream after every layer,) and the state behind them."""
    eps = cfg["norm"]["eps"]
    state = state if state is not None else {"n": 0, "layers": [{} for _ in cfg["layers"]]}
    pos = np.arange(state["n"], state["n"] + len(tokens))
    state["n"] += len(tokens)
    x = W["embed"][np.asarray(tokens)].astype(np.float64)
    streams = []
    for i, L in enumerate(cfg["layers"]):
        Wl, mx, st = sub(W, f"l{i}."), L["mixer"], state["layers"][i]
        Wm = sub(Wl, "mix.")
        h = rms_norm(x, Wl["norm1"], eps)
        if L["type"] == "latent_attention":
            x = x + latent_attention_mixer(h, Wm, mx, eps, pos, st)
        elif L["type"] == "gla":
            x = x + gla_mixer(h, Wm, mx, eps, st)
        else:
            x = x + parallel_mixer(h, Wm, mx, eps, pos, st)
        if L["mlp"]:
            x = x + feed_forward(rms_norm(x, Wl["norm2"], eps), sub(Wl, "mlp."))
        streams.append(x)
    logits = cfg["logit_scale"] * (rms_norm(x, W["final.norm"], eps) @ W["head"].T)
    return (logits, np.stack(streams), state) if want_layers else (logits, state)


def logits(cfg, W, tokens):
    return forward(cfg, W, tokens)[0]


# ------------------------------------------------------------------------------------------------ small configurations and random weights
def dense_cfg(ff=44):
    return {"kind": "dense", "ff": ff}


def latent_layer(heads=3, dim=10, vdim=14, q_rank=20, kv_rank=18, size=9, scale=0.4, mlp="dense"):
    mixer = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if size:
        mixer["mask"] = {"size": size}
    return {"type": "latent_attention", "mixer": mixer, "mlp": dense_cfg() if mlp == "dense" else mlp}


YARN = {"factor": 5.0, "original": 40, "fast": 9.0, "slow": 0.5}


def parallel_layer(heads=4, kv_heads=2, dim=12, vdim=10, rot=8, base=300.0, scaling=YARN, scale=0.35, softcap=6.0, d_heads=4, d_kv=2, d_dim=9, d_vdim=13, conv=4,
                   left_scale=0.7, right_scale=1.3, mlp="dense"):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot, "scaling": scaling}, "scale": scale, "softcap": softcap}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": left_scale, "right": {"heads": d_heads, "kv_heads": d_kv, "dim": d_dim, "vdim": d_vdim, "conv": conv},
                                          "right_scale": right_scale}, "mlp": dense_cfg() if mlp == "dense" else mlp}


def gla_layer(heads=3, dim=11, vdim=8, tau=4.0, mlp="dense"):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": dense_cfg() if mlp == "dense" else mlp}


def make_config(layers, width=48, vocab=60, eps=1e-4, logit_scale=1.7):
    return {"architecture": "Tugezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def bf16_round(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).view(np.float32)


def tensor_shapes(cfg, rank_a=5, rank_g=7):
    Wd, V = cfg["width"], cfg["vocab"]
    t = {"embed": (V, Wd), "final.norm": (Wd,), "head": (V, Wd)}
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        m = p + "mix."
        t[p + "norm1"] = (Wd,)
        if L["type"] == "latent_attention":
            H, D, Vd, QR, KR = mx["heads"], mx["dim"], mx["vdim"], mx["q_rank"], mx["kv_rank"]
            t.update({m + "dq": (QR, Wd), m + "dq.norm": (QR,), m + "uq": (H * D, QR), m + "dkv": (KR, Wd), m + "dkv.norm": (KR,), m + "uk": (H * D, KR), m + "uv": (H * Vd, KR),
                      m + "g": (H, Wd), m + "o": (Wd, H * Vd)})
        elif L["type"] == "gla":
            H, D, Vd = mx["heads"], mx["dim"], mx["vdim"]
            t.update({m + "q": (H * D, Wd), m + "k": (H * D, Wd), m + "v": (H * Vd, Wd), m + "g": (H * Vd, Wd), m + "o": (Wd, H * Vd), m + "norm": (Vd,), m + "a1": (rank_a, Wd),
                      m + "a2": (H * D, rank_a), m + "a2.b": (H * D,)})
        else:
            a, r = mx["left"], mx["right"]
            H, G, D, Vd = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            t.update({m + "left.q": (H * D, Wd), m + "left.k": (G * D, Wd), m + "left.v": (G * Vd, Wd), m + "left.o": (Wd, H * Vd)})
            H, G, D, Vd, taps = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
            m += "right."
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Vd)):
                t.update({m + n: (rows, Wd), m + n + ".conv": (rows, taps)})
            t.update({m + "b": (H, Wd), m + "A_log": (H,), m + "norm": (Vd,), m + "a1": (rank_a, Wd), m + "a2": (H * D, rank_a), m + "dt_bias": (H * D,), m + "g1": (rank_g, Wd),
                      m + "g2": (H * Vd, rank_g), m + "o": (Wd, H * Vd)})
        if L["mlp"]:
            F = L["mlp"]["ff"]
            t.update({p + "norm2": (Wd,), p + "mlp.gate": (F, Wd), p + "mlp.up": (F, Wd), p + "mlp.down": (Wd, F)})
    return t


def random_weights(cfg, seed=0, rank_a=5, rank_g=7):
    """bf16-representable values; decays spread over fast and slow channels, norm weights away from one."""
    rng = np.random.default_rng(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, rank_a, rank_g).items():
        leaf = name.split(".")[-1]
        if leaf == "A_log":
            w = rng.uniform(-3.0, 0.5, shape)
        elif leaf == "dt_bias":
            w = rng.uniform(-4.0, 1.0, shape)
        elif name.endswith("a2.b"):
            w = rng.uniform(-1.0, 5.0, shape)
        elif leaf.startswith("norm"):
            w = 1.0 + 0.3 * rng.standard_normal(shape)
        elif leaf == "conv":
            w = rng.standard_normal(shape) * 0.6
        elif leaf == "embed":
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) / math.sqrt(shape[-1]) * (1.5 if leaf in ("a2", "g2", "b", "g") else 1.0)
        W[name] = bf16_round(w).astype(np.float64)
    return W


def as_tensors(W):
    """name -> (dtype, shape, raw bytes), as the loader takes them."""
    return {n: ("BF16", w.shape, (np.ascontiguousarray(w, dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16).reshape(-1).view(np.uint8)) for n, w in W.items()}
