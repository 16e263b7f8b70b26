"""Plain float64 NumPy implementation of the Fafelix design, one function per mechanism, written from its equations.

It shares nothing with the library: whole sequences at once, explicit loops over positions and heads, every matrix as the
checkpoint stores it (out, in).  `forward(cfg, w, tokens)` returns the logits of every position and the residual stream
after every layer run; `make_config` / `make_weights` build small random checkpoints (tests choose their own sizes) and
`write_checkpoint` stores one as config.json + model.safetensors.

Notation: T positions t = 0 .. T-1, width W, eps = norm.eps, rms(z) = z / sqrt(mean(z^2) + eps).  A layer is
    h = LN(x) * w + b;   x <- x + mixer(h) + W_down (silu(W_gate h) * (W_up h))
and a span of layers may run several times in a row, the embedding output being added to x before every pass but the first.
"""
import json
import math
import os
import struct

import numpy as np


# ---- norms and activations ----------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


# ---- embedding with a bigram table --------------------------------------------------------------------------------------
def bigram_row(prev, token, big):
    """Row of the bigram table for a token and the one before it (prev None: the sequence's first token)."""
    if prev is None:
        return int(big["buckets"])
    return (int(prev) * int(big["mul_prev"]) + int(token) * int(big["mul_cur"])) % int(big["buckets"])


def embedding(tokens, cfg, w):
    x = w["embed"][tokens].copy()
    big = (cfg.get("embedding") or {}).get("bigram")
    if big:
        for t in range(len(tokens)):
            x[t] += w["bigram"][bigram_row(tokens[t - 1] if t else None, tokens[t], big)]
    return x


# ---- rotary positions, interleaved pairs, frequencies rescaled by wavelength ------------------------------------------------
def rotary_freqs(rot):
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return np.array(f)
    factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for fi in f:
        wave = 2 * math.pi / fi
        if wave < orig / high:
            out.append(fi)
        elif wave > orig / low:
            out.append(fi / factor)
        else:
            s = (orig / wave - low) / (high - low)
            out.append((1 - s) * fi / factor + s * fi)
    return np.array(out)


def rotate_pairs(x, pos, freqs):
    """x (..., >= dims) at position pos: channel 2 i pairs with 2 i + 1; the rest passes."""
    n = len(freqs)
    out = np.array(x, dtype=np.float64)
    c, s = np.cos(pos * freqs), np.sin(pos * freqs)
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    out[..., 0:2 * n:2] = u * c - v * s
    out[..., 1:2 * n:2] = v * c + u * s
    return out


# ---- attention with a sink ----------------------------------------------------------------------------------------------
def softmax_with_sink(s, sink):
    """Weights over the keys when the denominator also holds exp(sink): no key, no value, counted once."""
    top = max(s.max(), sink)
    e = np.exp(s - top)
    return e / (e.sum() + math.exp(sink - top))


def attention(h, m, w, p, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, d)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    f = rotary_freqs(m["rot"])
    for t in range(T):
        q[t], k[t] = rms(rotate_pairs(q[t], t, f), eps), rms(rotate_pairs(k[t], t, f), eps)
    out = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        for t in range(T):
            s = (k[:t + 1, g] @ q[t, a]) * float(m["scale"])
            out[t, a] = softmax_with_sink(s, float(w[p + "sink"][a])) @ v[:t + 1, g]
    return out.reshape(T, H * dv) @ w[p + "o"].T


# ---- gated delta rule, one decay per head ----------------------------------------------------------------------------------
def short_conv(z, c):
    """z (T, C), c (C, taps), last tap on the current position, zeros before the sequence."""
    T, taps = z.shape[0], c.shape[1]
    out = np.zeros_like(z)
    for t in range(T):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                out[t] += c[:, j] * z[t - (taps - 1) + j]
    return out


def delta_rule(q, k, v, g, beta):
    """q, k (T, D), v (T, P), g, beta (T): one head's recurrence from a zero state."""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        S = S + np.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out[t] = S.T @ q[t]
    return out


def delta(h, m, w, p, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = unit(silu(short_conv(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, d)) * d ** -0.5
    k = unit(silu(short_conv(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, d))
    v = silu(short_conv(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = np.stack([delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], g[:, a], beta[:, a]) for a in range(H)], 1)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, dv)
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- time mixing with a decay per key channel and a bonus for the current token ----------------------------------------------
def wkv_rule(r, k, v, dec, u):
    """r, k, dec (T, D), v (T, P), u (D): one head's recurrence from a zero state; the read-out comes before the decay."""
    S = np.zeros((k.shape[1], v.shape[1]))
    out = np.zeros_like(v)
    for t in range(k.shape[0]):
        out[t] = (S + np.outer(u * k[t], v[t])).T @ r[t]
        S = dec[t][:, None] * S + np.outer(k[t], v[t])
    return out


def wkv_mixes(h, w, p):
    prev = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])
    return {s: h + (prev - h) * w[p + "mu." + s] for s in "rkvgw"}


def wkv(h, m, w, p, eps):
    T = h.shape[0]
    H, d = int(m["heads"]), int(m["dim"])
    x = wkv_mixes(h, w, p)
    r, k, v = ((x[s] @ w[p + s].T).reshape(T, H, d) for s in "rkv")
    dec = np.exp(-np.exp(np.tanh(x["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(T, H, d)
    o = np.stack([wkv_rule(r[:, a], k[:, a], v[:, a], dec[:, a], w[p + "u"][a]) for a in range(H)], 1)
    o = rms(o, eps).reshape(T, H * d) * w[p + "norm"] * silu(x["g"] @ w[p + "g"].T)
    return o @ w[p + "o"].T


# ---- feed-forward, the order of layers, the model ---------------------------------------------------------------------------
def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer_runs(cfg):
    """(layer, first layer of a repeated pass?) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    out = [(i, False) for i in range(a)]
    for times in range(int(loop["times"])):
        out += [(i, times > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


MIXERS = {"delta": delta, "attention": attention, "wkv": wkv}


def forward(cfg, w, tokens):
    """Logits (T, vocab) and the residual stream after every layer run (runs, T, W)."""
    tokens = [int(t) for t in tokens]
    eps = float(cfg["norm"]["eps"])
    x = x0 = embedding(tokens, cfg, w)
    after = []
    for i, again in layer_runs(cfg):
        L, p = cfg["layers"][i], "l%d." % i
        if again:
            x = x + x0
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        y = MIXERS[L["type"]](h, L["mixer"], w, p + "mix.", eps)
        if L.get("mlp"):
            y = y + dense_ff(h, w, p + "mlp.")
        x = x + y
        after.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T, np.stack(after)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, w, toks)[0][-1])))
    return toks[len(prompt):]


def bf16_round(a):
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64)


# ---- small random checkpoints -------------------------------------------------------------------------------------------
def delta_mixer(heads=4, kv_heads=2, dim=16, vdim=24, conv=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attention_mixer(heads=6, kv_heads=3, dim=16, vdim=24, rot_dims=8, base=300.0, scaling=True, scale=None):
    rot = {"dims": rot_dims, "base": base}
    if scaling:   # the four wavelengths at base 300 lie on both sides of, and between, the two bounds
        rot["scaling"] = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot,
                                           "scale": scale if scale is not None else 0.3}}


def wkv_mixer(heads=3, dim=12, rank=5):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "rank": rank}


def make_config(layers, width=48, vocab=96, ff=80, loop=None, eps=1e-5, buckets=53, mul_prev=31, mul_cur=5):
    out = []
    for L in layers:
        L = dict(L)
        L.setdefault("mlp", {"kind": "dense", "ff": ff} if ff else None)
        out.append(L)
    cfg = {"architecture": "Fafelix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": out}
    if buckets:
        cfg["embedding"] = {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def make_weights(cfg, seed=0, gain=1.0):
    """Random weights, rounded to bf16 (what a checkpoint stores)."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, o, i, g=1.0):
        w[name] = bf16_round(rng.standard_normal((o, i)) * g * gain / math.sqrt(i))

    def vec(name, n, around=1.0, spread=0.2):
        w[name] = bf16_round(around + spread * rng.standard_normal(n))

    w["embed"] = bf16_round(rng.standard_normal((V, W)))
    big = (cfg.get("embedding") or {}).get("bigram")
    if big:
        w["bigram"] = bf16_round(0.7 * rng.standard_normal((big["buckets"] + 1, W)))
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        q = p + "mix."
        vec(p + "norm1", W)
        vec(p + "norm1.b", W, 0.0, 0.3)
        if L["type"] == "delta":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                mat(q + n, c, W, 1.5)
                vec(q + n + ".conv", (c, m["conv"]), 0.2, 0.6)
            mat(q + "b", H, W, 2.0)
            mat(q + "a", H, W)
            vec(q + "A_log", H, -0.5, 0.8)
            vec(q + "dt_bias", H, -1.0, 1.0)
            vec(q + "norm", dv)
            mat(q + "g", H * dv, W)
            mat(q + "o", W, H * dv)
        elif L["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, c in (("q", H * d), ("k", G * d), ("v", G * dv)):
                mat(q + n, c, W, 1.5)
                vec(q + n + ".b", c, 0.0, 0.4)
            vec(q + "sink", H, 0.5, 1.0)
            mat(q + "o", W, H * dv)
        else:
            H, d = m["heads"], m["dim"]
            for s in "rkvgw":
                vec(q + "mu." + s, W, 0.5, 0.3)
            for s in "rkvg":
                mat(q + s, H * d, W)
            mat(q + "w1", L["rank"], W)
            mat(q + "w2", H * d, L["rank"], 1.5)
            vec(q + "w0", H * d, -1.5, 0.8)
            vec(q + "u", (H, d), 0.5, 0.5)
            vec(q + "norm", H * d)
            mat(q + "o", W, H * d)
        if L.get("mlp"):
            f = L["mlp"]["ff"]
            mat(p + "mlp.gate", f, W)
            mat(p + "mlp.up", f, W)
            mat(p + "mlp.down", W, f)
    vec("final.norm", W)
    vec("final.norm.b", W, 0.0, 0.3)
    mat("head", V, W)
    return w


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (bf16).  The decay's inner size is given by the tensors alone."""
    os.makedirs(folder, exist_ok=True)
    stored = dict(cfg, layers=[{k: v for k, v in L.items() if k != "rank"} for L in cfg["layers"]])
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(stored, f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        b = (np.asarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    hj = json.dumps(header).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
