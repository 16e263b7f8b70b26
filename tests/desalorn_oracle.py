"""Plain float64 NumPy implementation of the Desalorn design, one function per mechanism, written from its equations.

It shares nothing with the library: whole sequences at once, explicit loops over positions for everything that has a
window or a state.  `forward(cfg, w, tokens)` returns the logits of every position and the residual stream after every
layer; `make_config` / `make_weights` build small random checkpoints (tests choose their own sizes) and `write_checkpoint`
stores one as config.json + model.safetensors.

Notation: T positions t = 0 .. T-1, width W.  A layer is x <- x + m (mixer(h) + ff(h)) with ONE norm h = N(x), an RMS norm
of every one of `groups` equal parts of the vector.
"""
import json
import math
import os
import struct

import numpy as np


# ---- norms --------------------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def group_norm(x, w, groups, eps):
    """Every one of `groups` equal neighbouring parts over its own root mean square; then the weight."""
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    return rms(parts, eps).reshape(x.shape) * w


# ---- rotary positions ---------------------------------------------------------------------------------------------------
def rotary_freqs(rot):
    d = int(rot["dims"])
    return np.array([float(rot["base"]) ** (-2.0 * i / d) for i in range(d // 2)])


def rotate(x, pos, freqs, interleaved):
    """The first 2 len(freqs) channels of x (..., D) at position pos, pair i turned by pos * freqs[i]."""
    n = len(freqs)
    out = np.array(x, dtype=np.float64)
    c, s = np.cos(pos * freqs), np.sin(pos * freqs)
    a, b = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    u, v = x[..., a], x[..., b]
    out[..., a] = u * c - v * s
    out[..., b] = v * c + u * s
    return out


# ---- distance bias ------------------------------------------------------------------------------------------------------
def bucket(n, rows, far):
    """Row of the distance table for distance n: one each below rows / 2, then logarithmic up to `far`, then the last."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


# ---- attention ----------------------------------------------------------------------------------------------------------
def softmax(s):
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def mixed_scores(q_t, k, m, rel, talk):
    """Scores (H, j) of one query position t = len(k) - 1: q_t (H, dim), k (t + 1, G, dim)."""
    H, G = q_t.shape[0], k.shape[1]
    t = k.shape[0] - 1
    rows = rel.shape[0]
    dist = [bucket(t - j, rows, float(m["bias_max"])) for j in range(t + 1)]
    s = np.zeros((H, t + 1))
    for h in range(H):
        z = (k[:, h // (H // G)] @ q_t[h]) * float(m["scale"])
        cap = float(m["softcap"])
        s[h] = cap * np.tanh(z / cap) + rel[dist, h]
    return talk @ s


def attention(h, m, w, p, eps):
    """h (T, W) -> (T, W)."""
    T = h.shape[0]
    H, G, D, P = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, P)
    q, k = q.reshape(T, H, D), k.reshape(T, G, D)
    o = np.zeros((T, H, P))
    for t in range(T):
        a = softmax(mixed_scores(q[t], k[:t + 1], m, w[p + "rel"], w[p + "talk"]))
        for hh in range(H):
            o[t, hh] = a[hh] @ v[:t + 1, hh // (H // G)]
    o *= 1.0 / (1.0 + np.exp(-(h @ w[p + "g"].T)))[:, :, None]
    return o.reshape(T, H * P) @ w[p + "o"].T + w[p + "o.b"]


# ---- retention ----------------------------------------------------------------------------------------------------------
def retention_scan(q, k, v, decay):
    """Per head S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t.  q, k (T, H, D), v (T, H, P)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    o = np.zeros(v.shape)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdp,hd->hp", S, q[t])
    return o


def retention(h, m, w, p, eps):
    T = h.shape[0]
    H, D, P = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    f = rotary_freqs(m["rot"])
    q, k = (h @ w[p + "q"].T).reshape(T, H, D), (h @ w[p + "k"].T).reshape(T, H, D)
    v = (h @ w[p + "v"].T).reshape(T, H, P)
    q = np.stack([rotate(q[t], t, f, False) for t in range(T)])
    k = np.stack([rotate(k[t], t, f, False) for t in range(T)]) * D ** -0.5
    o = rms(retention_scan(q, k, v, np.array(m["decay"], dtype=np.float64)), eps).reshape(T, H * P)
    return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- latent attention ---------------------------------------------------------------------------------------------------
def latent_attention(h, m, w, p, eps):
    T = h.shape[0]
    H, dn, dr, dv, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    f = rotary_freqs(m["rot"])
    q = ((rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]) @ w[p + "uq"].T).reshape(T, H, dn + dr)
    ckr = h @ w[p + "dkv"].T
    c = rms(ckr[:, :r], eps) * w[p + "dkv.norm"]
    kr = np.stack([rotate(ckr[t, r:], t, f, True) for t in range(T)])
    kn, val = (c @ w[p + "uk"].T).reshape(T, H, dn), (c @ w[p + "uv"].T).reshape(T, H, dv)
    win = int(m["mask"]["size"])
    o = np.zeros((T, H, dv))
    for t in range(T):
        lo = max(0, t - win + 1)
        qr = rotate(q[t, :, dn:], t, f, True)
        for hh in range(H):
            s = (kn[lo:t + 1, hh] @ q[t, hh, :dn] + kr[lo:t + 1] @ qr[hh]) * float(m["scale"])
            o[t, hh] = softmax(s) @ val[lo:t + 1, hh]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def silu(z):
    return z / (1.0 + np.exp(-z))


def glu(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(choice, top, count, keep):
    """Indices of the `top` largest choice scores (E,) among the `keep` groups of neighbours whose two largest add up highest."""
    E = choice.shape[0]
    g = choice.reshape(count, E // count)
    score = np.sort(g, -1)[:, -2:].sum(-1)
    best = np.argsort(-score, kind="stable")[:keep]
    open_ = np.zeros(count, dtype=bool)
    open_[best] = True
    c = np.where(np.repeat(open_, E // count), choice, -np.inf)
    return np.argsort(-c, kind="stable")[:top]


def route(h, f, w, p):
    """Chosen experts (T, top) and their weights."""
    r = f["router"]
    s = 1.0 / (1.0 + np.exp(-(h @ w[p + "router"].T)))
    gr = r.get("groups") or {"count": 1, "keep": 1}
    ids = np.stack([choose(s[t] + w[p + "correction"], int(r["top"]), int(gr["count"]), int(gr["keep"])) for t in range(h.shape[0])])
    return ids, np.take_along_axis(s, ids, -1)


def moe(h, f, w, p):
    ids, ws = route(h, f, w, p)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t], ws[t]):
            out[t] += wt * glu(h[t:t + 1], w, "%se%d." % (p, e))[0]
    if f.get("shared"):
        out = out + glu(h, w, p + "shared.")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention, "retention": retention, "latent_attention": latent_attention}


def forward(cfg, w, tokens):
    """-> logits (T, vocab), residual stream after every layer (L, T, W); all float64."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in w.items()}
    eps, groups, mult = float(cfg["norm"]["eps"]), int(cfg["norm"]["groups"]), float(cfg["residual_mult"])
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    after = []
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        h = group_norm(x, w[p + "norm1"], groups, eps)
        y = MIXERS[L["type"]](h, L["mixer"], w, p + "mix.", eps)
        if L.get("mlp"):
            y = y + moe(h, L["mlp"], w, p + "mlp.")
        x = x + mult * y
        after.append(x)
    return group_norm(x, w["final.norm"], groups, eps) @ w["head"].T, np.stack(after)


def greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(forward(cfg, w, toks)[0][-1])))
    return toks[len(prompt):]


# ---- small random checkpoints -------------------------------------------------------------------------------------------
def bf16_round(a):
    """float -> nearest bfloat16 (ties to even), as float32."""
    u = np.asarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32)


def attention_mixer(heads=4, kv_heads=2, dim=16, vdim=24, bias_max=40, softcap=6.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "softcap": softcap,
            "scale": scale if scale is not None else dim ** -0.5}


def retention_mixer(heads=3, dim=24, vdim=40, rot_dims=16, base=20000.0, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims},
            "decay": list(decay) if decay is not None else [1.0 - 2.0 ** -(3 + i) for i in range(heads)]}


def latent_mixer(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=32, q_rank=48, window=12, base=10000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
            "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}


def moe_mlp(ff=24, experts=6, top=2, count=3, keep=2, shared=40):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def make_config(layers, width=48, vocab=96, groups=3, eps=1e-5, embed_scale=4.0, residual_mult=0.6):
    """layers: list of (type, mixer dict, mlp dict or None)."""
    return {"architecture": "Desalorn", "embedding": {"scale": embed_scale}, "layers": [{"type": t, "mixer": m, "mlp": f} for t, m, f in layers],
            "norm": {"eps": eps, "groups": groups}, "residual_mult": residual_mult, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, rel_rows=12, router_gain=1.0):
    """Random weights, rounded to bfloat16 values (float32 arrays)."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def lin(name, out, inp, gain=1.0):
        w[name] = rng.standard_normal((out, inp)) * gain / math.sqrt(inp)

    def near(name, shape, mean, spread):
        w[name] = mean + spread * rng.standard_normal(shape)

    w["embed"] = rng.standard_normal((V, W)) / cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p, m, f = "l%d." % i, L["mixer"], L["mlp"]
        near(p + "norm1", W, 1.0, 0.2)
        q = p + "mix."
        if L["type"] == "attention":
            H, G, D, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, n in (("q", H * D), ("k", G * D), ("v", G * P)):
                lin(q + name, n, W), near(q + name + ".b", n, 0.0, 0.3)
            near(q + "q.norm", H * D, 1.5, 0.2), near(q + "k.norm", G * D, 1.5, 0.2)
            near(q + "rel", (rel_rows, H), 0.0, 0.5)
            w[q + "talk"] = np.eye(H) + rng.standard_normal((H, H)) * 0.4 / math.sqrt(H)
            lin(q + "g", H, W, 2.0), lin(q + "o", W, H * P), near(q + "o.b", W, 0.0, 0.3)
        elif L["type"] == "retention":
            H, D, P = m["heads"], m["dim"], m["vdim"]
            lin(q + "q", H * D, W), lin(q + "k", H * D, W), lin(q + "v", H * P, W), lin(q + "g", H * P, W), lin(q + "o", W, H * P)
        else:
            H, dn, dr, dv, r, qr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            lin(q + "dq", qr, W), near(q + "dq.norm", qr, 1.0, 0.2), lin(q + "uq", H * (dn + dr), qr, 2.0)
            lin(q + "dkv", r + dr, W, 2.0), near(q + "dkv.norm", r, 1.0, 0.2)
            lin(q + "uk", H * dn, r, 2.0), lin(q + "uv", H * dv, r), lin(q + "o", W, H * dv)
        if f:
            q, r = p + "mlp.", f["router"]
            for e in ["e%d" % e for e in range(r["experts"])] + (["shared"] if f.get("shared") else []):
                ff = f["shared"]["ff"] if e == "shared" else f["expert"]["ff"]
                lin(q + e + ".gate", ff, W), lin(q + e + ".up", ff, W), lin(q + e + ".down", W, ff)
            lin(q + "router", r["experts"], W, router_gain)
            near(q + "correction", r["experts"], -0.5, 0.3)
    near("final.norm", W, 1.0, 0.2)
    lin("head", V, W)
    return {k: bf16_round(v) for k, v in w.items()}


def write_checkpoint(folder, cfg, w):
    """config.json + model.safetensors (bfloat16 tensors)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, a in w.items():
        b = (np.asarray(a, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    hj = json.dumps(head).encode()
    hj += b" " * (-len(hj) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
