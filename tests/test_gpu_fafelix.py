"""-m gpu: the Fafelix design on the layered executor against the plain float64 statement in fafelix_oracle.py.

The new row ops alone (device arrays through the C ABI): the bigram embedding and its carried token; the layer norm with a bias
(far from zero mean, with an addition before it, into 16-bit operands); the blends with the previous token; short convolutions,
unit vectors, decay and beta; the time mixing's decay; both recurrences with a key that stands out hundreds of positions back,
in portions and as fused decode rows; biases + rotation + weightless norm + cache append; causal attention with a far key and
sinks that outweigh all keys or none; the output product's input; the decode products with the norm, the blends, the
activation and the residual add inside; the tensor-core product with one input per segment.  Then small models with random weights
whose sizes differ from layer to layer: every mechanism through the residual after its layer run; repeated passes; whole
prompts against token-by-token decoding and portions down to two tokens; caches given back and used again; long decoding;
tensor-core prompt routes and serving precision; greedy generation through the library's entry points, the command line and the
trace runner.
"""
import ctypes as C
import json
import math
import os
import re
import subprocess
import sys

import numpy as np
import pytest
import torch

import fafelix_oracle as O
from yalm_b200 import api

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 3e-4
vp, i32, f32, i64 = C.c_void_p, C.c_int, C.c_float, C.c_longlong
DTYPES = [(api.F32, torch.float32), (api.BF16, torch.bfloat16)]


def dev(a, dtype=torch.float32):
    return torch.as_tensor(np.ascontiguousarray(a), dtype=dtype).cuda().contiguous()


def zeros(*shape, dtype=torch.float32):
    return torch.zeros(shape, dtype=dtype, device="cuda")


def ptr(t, offset=0):
    return vp(t.data_ptr() + offset * t.element_size()) if t is not None else None


def ok(rc, what):
    torch.cuda.synchronize()
    assert rc == 0, "%s returned %d" % (what, rc)


def close_enough(got, want, tol=F32_TOL):
    scale = max(1.0, float(np.abs(want).max()))
    err = float(np.abs(np.asarray(got, np.float64) - want).max())
    assert err <= tol * scale, f"max |delta| {err:.3e} > {tol * scale:.3e}"


def portions(T, sizes):
    at, k = 0, 0
    while at < T:
        n = min(sizes[k % len(sizes)], T - at)
        yield at, n
        at, k = at + n, k + 1


def L():
    lib = api.lib()
    lib.yalm_attn_window_pool_workspace.restype = C.c_size_t
    return lib


PORTIONS = [[1], [2], [3, 1, 7], [64]]


# ---- embedding ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("sizes", PORTIONS)
@pytest.mark.parametrize("dt,tt", DTYPES)
def test_bigram_embedding(dt, tt, sizes):
    rng = np.random.default_rng(1)
    V, W, T = 50, 36, 23
    big = {"buckets": 17, "mul_prev": 2000000011, "mul_cur": 1999999973}      # the products pass 2^31: the sum is formed in 64 bits
    cfg = {"embedding": {"bigram": big}}
    w = {"embed": O.bf16_round(rng.standard_normal((V, W))), "bigram": O.bf16_round(rng.standard_normal((18, W)))}
    table, btab, prev = dev(w["embed"], tt), dev(w["bigram"], tt), zeros(1, dtype=torch.int32)
    for seed in (2, 3):                                              # the second sequence starts over the first one's carried token
        toks = np.random.default_rng(seed).integers(0, V, T)
        x, x0, tk = zeros(T, W), zeros(T, W), dev(toks, torch.int32)
        for at, n in portions(T, sizes):
            ok(L().yalm_embed_bigram_rows(ptr(x[at:]), ptr(x0[at:]), ptr(table), ptr(btab), dt, ptr(tk[at:]), big["buckets"], i64(big["mul_prev"]), i64(big["mul_cur"]),
                                          ptr(prev), n, W, at, None, None), "embed_bigram_rows")
        want = O.embedding(toks, cfg, w)
        close_enough(x.cpu().numpy(), want, 1e-6)
        close_enough(x0.cpu().numpy(), want, 1e-6)
        assert int(prev[0]) == toks[-1]


# ---- norm and blends --------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W", [48, 50, 2048])
def test_layer_norm_rows(W):
    rng = np.random.default_rng(W)
    n, eps = 5, 1e-5
    x, a = 40.0 + rng.standard_normal((n, W)), rng.standard_normal((n, W))     # the mean is far larger than the spread
    w, b = 1 + 0.3 * rng.standard_normal(W), rng.standard_normal(W)
    wd, bd, ad = dev(w), dev(b), dev(a)
    xd, out, o16 = dev(x), zeros(n, W), zeros(n, W, dtype=torch.bfloat16)
    ok(L().yalm_layer_norm_rows(ptr(out), ptr(o16), 1, ptr(xd), ptr(ad), None, ptr(wd), ptr(bd), f32(eps), n, W, None), "layer_norm_rows")
    want = O.layer_norm(np.float32(x).astype(np.float64) + np.float32(a), w, b, eps)
    close_enough(out.cpu().numpy(), want)
    close_enough(o16.float().cpu().numpy(), want, 5e-3)
    close_enough(xd.cpu().numpy(), x + a, 1e-6)
    rows = dev([3, 1], torch.int32)
    two = zeros(2, W)
    ok(L().yalm_layer_norm_rows(ptr(two), None, 0, ptr(xd), None, ptr(rows), ptr(wd), None, f32(eps), 2, W, None), "layer_norm_rows gathered")
    close_enough(two.cpu().numpy(), want[[3, 1]] - b)
    assert np.abs(O.rms(x + a, eps) * w + b - want).max() > 1.0               # not an RMS norm


@pytest.mark.parametrize("sizes", PORTIONS)
def test_blends_with_the_previous_token(sizes):
    rng = np.random.default_rng(4)
    W, T, S = 37, 20, 4
    h, mu = rng.standard_normal((T, W)), rng.standard_normal((S, W))
    prev = np.concatenate([np.zeros((1, W)), h[:-1]])
    want = np.stack([h if s == 2 else h + (prev - h) * mu[s] for s in range(S)])
    hd, md, state = dev(h), dev(mu), dev(rng.standard_normal((2, W)))          # what an earlier sequence left is not read
    got, got16 = np.zeros((S, T, W)), np.zeros((S, T, W))
    for at, n in portions(T, sizes):
        out, o16 = zeros(S, n, W), zeros(S, n, W, dtype=torch.bfloat16)
        ok(L().yalm_mix_rows(ptr(out), ptr(o16), 1, ptr(hd[at:]), ptr(md), S, 1 << 2, ptr(state), n, W, at, None, None), "mix_rows")
        got[:, at:at + n], got16[:, at:at + n] = out.cpu().numpy(), o16.float().cpu().numpy()
    close_enough(got, want)
    close_enough(got16, want, 1e-2)


# ---- the delta rule ------------------------------------------------------------------------------------------------------------------
def delta_case(T, H, G, D, P, taps, seed=0):
    """Raw projection rows [q | k | v | gate | beta | decay] and weights; row T - 1 asks for what row 3 wrote (decays near 1)."""
    rng = np.random.default_rng(seed)
    c = {"H": H, "G": G, "D": D, "P": P, "taps": taps, "C": 2 * G * D + H * P}
    c["ld"] = c["C"] + H * P + 2 * H + 3
    c["rows"] = rng.standard_normal((T, c["ld"]))
    c["conv"] = rng.standard_normal((c["C"], taps)) / math.sqrt(taps)
    c["A_log"], c["dt_bias"], c["norm"] = rng.standard_normal(H) - 4.0, rng.standard_normal(H) - 2.0, 1 + 0.3 * rng.standard_normal(P)
    c["o_gate"], c["o_beta"], c["o_decay"] = c["C"], c["C"] + H * P, c["C"] + H * P + H
    return c


def delta_plain(c, eps=1e-5):
    z, H, G, D, P, C = c["rows"], c["H"], c["G"], c["D"], c["P"], c["C"]
    T = len(z)
    y = O.silu(O.short_conv(z[:, :C], c["conv"]))
    q, k, v = O.unit(y[:, :G * D].reshape(T, G, D)) * D ** -0.5, O.unit(y[:, G * D:2 * G * D].reshape(T, G, D)), y[:, 2 * G * D:].reshape(T, H, P)
    beta = O.sigmoid(z[:, c["o_beta"]:c["o_beta"] + H])
    g = np.exp(-np.exp(c["A_log"]) * O.softplus(z[:, c["o_decay"]:c["o_decay"] + H] + c["dt_bias"]))
    o = np.stack([O.delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], g[:, a], beta[:, a]) for a in range(H)], 1)
    out = O.rms(o, eps) * c["norm"] * O.silu(z[:, c["o_gate"]:c["o_gate"] + H * P]).reshape(T, H, P)
    return dict(q=q, k=k, v=v, beta=beta, g=g, o=o.reshape(T, -1), out=out.reshape(T, -1))


DELTA_SIZES = [(4, 2, 16, 24, 3), (3, 3, 64, 32, 4), (2, 1, 10, 7, 1), (4, 1, 128, 40, 2), (2, 2, 200, 72, 5)]


@pytest.mark.parametrize("sizes", PORTIONS)
@pytest.mark.parametrize("H,G,D,P,taps", DELTA_SIZES)
def test_delta_rule_rows(H, G, D, P, taps, sizes):
    T = 70
    c = delta_case(T, H, G, D, P, taps, seed=D)
    want = delta_plain(c)
    C_, ld = c["C"], c["ld"]
    z, conv, al, dtb, nw = dev(c["rows"]), dev(c["conv"]), dev(c["A_log"]), dev(c["dt_bias"]), dev(c["norm"])
    ring, state = dev(np.full((taps, C_), 7.0)), dev(np.full((H, P, D), 3.0))      # left by another sequence: not read
    y, gates, o, out = zeros(T, C_), zeros(T, 2 * H), zeros(T, H * P), zeros(T, H * P)
    scale = f32(D ** -0.5)
    for at, n in portions(T, sizes):
        ok(L().yalm_delta_in_rows(ptr(y[at:]), ptr(gates[at:]), ptr(z[at:]), ptr(z[at:], c["o_beta"]), ld, ptr(conv), ptr(ring), ptr(al), ptr(dtb), n, H, G, D, P, taps,
                                  f32(1e-6), scale, at, None, None), "delta_in_rows")
        ya, ga = y[at:], gates[at:]
        ok(L().yalm_state_scan_rows(ptr(o[at:]), H * P, ptr(ya, G * D), C_, ptr(ya), C_, ptr(ya, 2 * G * D), C_, ptr(ga), 2 * H, 0, None, 0, ptr(ga, H), 2 * H, None,
                                    ptr(state), n, H, H // G, D, P, at, None, None), "state_scan_rows")
    ok(L().yalm_block_out_rows(ptr(out), None, 0, H * P, ptr(o), H * P, ptr(z, c["o_gate"]), None, ld, ptr(nw), 0, f32(1e-5), T, H, P, 0, 1, None), "block_out_rows")
    g = y.cpu().numpy()
    close_enough(g[:, :G * D].reshape(T, G, D), want["q"])
    close_enough(g[:, G * D:2 * G * D].reshape(T, G, D), want["k"])
    close_enough(g[:, 2 * G * D:].reshape(T, H, P), want["v"])
    close_enough(gates.cpu().numpy(), np.concatenate([want["g"], want["beta"]], 1))
    close_enough(o.cpu().numpy(), want["o"])
    close_enough(out.cpu().numpy(), want["out"])


@pytest.mark.parametrize("first", [0, 1, 2, 30])
@pytest.mark.parametrize("H,G,D,P,taps", DELTA_SIZES)
def test_delta_rule_decode_rows_in_one_launch(H, G, D, P, taps, first):
    """A portion of `first` rows through the separate ops, then one fused launch per row, over state another sequence left."""
    T = 45
    c = delta_case(T, H, G, D, P, taps, seed=D + 1)
    want = delta_plain(c)
    C_, ld = c["C"], c["ld"]
    z, conv, al, dtb, nw = dev(c["rows"]), dev(c["conv"]), dev(c["A_log"]), dev(c["dt_bias"]), dev(c["norm"])
    ring, state = dev(np.full((taps, C_), 7.0)), dev(np.full((H, P, D), 3.0))
    if first:
        y, gates, o = zeros(first, C_), zeros(first, 2 * H), zeros(first, H * P)
        ok(L().yalm_delta_in_rows(ptr(y), ptr(gates), ptr(z), ptr(z, c["o_beta"]), ld, ptr(conv), ptr(ring), ptr(al), ptr(dtb), first, H, G, D, P, taps, f32(1e-6),
                                  f32(D ** -0.5), 0, None, None), "delta_in_rows")
        ok(L().yalm_state_scan_rows(ptr(o), H * P, ptr(y, G * D), C_, ptr(y), C_, ptr(y, 2 * G * D), C_, ptr(gates), 2 * H, 0, None, 0, ptr(gates, H), 2 * H, None, ptr(state),
                                    first, H, H // G, D, P, 0, None, None), "state_scan_rows")
    out = zeros(T, H * P)
    for t in range(first, T):
        ok(L().yalm_delta_step(ptr(out[t:]), ptr(state), ptr(z[t:]), 0, c["o_gate"], c["o_beta"], c["o_decay"], ptr(conv), ptr(ring), ptr(al), ptr(dtb), ptr(nw), H, G, D, P,
                               taps, f32(1e-6), f32(D ** -0.5), f32(1e-5), t, None, None), "delta_step")
    close_enough(out.cpu().numpy()[first:], want["out"][first:])


@pytest.mark.parametrize("sizes", [[1], [37, 2], [600]])
def test_delta_rule_recalls_a_far_key(sizes):
    """Six hundred positions with orthogonal-ish keys and no decay: the last query is row 5's key and must return row 5's value;
    without that row's write the result is another."""
    T, D, P = 600, 64, 16
    rng = np.random.default_rng(9)
    k = O.unit(rng.standard_normal((T, D)))
    k[6:] -= np.outer(k[6:] @ k[5], k[5])                    # nothing later writes along row 5's key
    q, v = O.unit(rng.standard_normal((T, D))), rng.standard_normal((T, P))
    q[-1] = k[5]
    g, beta = np.ones(T), np.full(T, 0.9)
    beta[5] = 1.0
    want = O.delta_rule(q, k, v, g, beta)
    np.testing.assert_allclose(want[-1], v[5], atol=1e-5)
    assert np.abs(O.delta_rule(q, k, v, g, np.where(np.arange(T) == 5, 0.0, beta))[-1] - want[-1]).max() > 0.5
    kd, qd, vd, gd, bd = dev(k), dev(q), dev(v), dev(g[:, None]), dev(beta[:, None])
    out, state = zeros(T, P), zeros(1, P, D)
    for at, n in portions(T, sizes):
        ok(L().yalm_state_scan_rows(ptr(out[at:]), P, ptr(kd[at:]), D, ptr(qd[at:]), D, ptr(vd[at:]), P, ptr(gd[at:]), 1, 0, None, 0, ptr(bd[at:]), 1, None, ptr(state), n, 1, 1,
                                    D, P, at, None, None), "state_scan_rows")
    close_enough(out.cpu().numpy(), want)


# ---- time mixing ----------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rank", [5, 16, 64])
@pytest.mark.parametrize("dt,tt", DTYPES)
def test_time_mixing_decay(dt, tt, rank):
    rng = np.random.default_rng(rank)
    n, ch, ld = 37, 70, rank + 3
    t, w2, w0 = 2 * rng.standard_normal((n, ld)), O.bf16_round(rng.standard_normal((ch, rank))), rng.standard_normal(ch) - 1.0
    out, td, wd, bd = zeros(n, ch + 2), dev(t), dev(w2, tt), dev(w0)
    ok(L().yalm_wkv_decay_rows(ptr(out), ch + 2, ptr(td), ld, ptr(wd), ptr(bd), dt, n, ch, rank, None), "wkv_decay_rows")
    close_enough(out.cpu().numpy()[:, :ch], np.exp(-np.exp(np.tanh(t[:, :rank]) @ w2.T + w0)))


def wkv_case(T, H, D, seed=0):
    rng = np.random.default_rng(seed)
    r, k, v = (rng.standard_normal((T, H, D)) for _ in range(3))
    dec = 1.0 - 0.05 * rng.random((T, H, D))
    dec[:, :, 0] = 1.0                                        # one channel per head never forgets
    return r, k, v, dec, rng.standard_normal((H, D))


@pytest.mark.parametrize("sizes", [[1], [2], [33, 1, 7], [300]])
@pytest.mark.parametrize("H,D", [(3, 12), (2, 64), (1, 130), (4, 8)])
def test_time_mixing_recurrence(H, D, sizes):
    T = 300
    r, k, v, dec, u = wkv_case(T, H, D, seed=D)
    k[:, :, 0] *= 0.01
    k[4, :, 0], r[-1, :, 0] = 5.0, 8.0                        # the last row reads what row 4 wrote into the channel that never forgets
    want = np.stack([O.wkv_rule(r[:, a], k[:, a], v[:, a], dec[:, a], u[a]) for a in range(H)], 1)
    k2 = k.copy()
    k2[4, :, 0] = 0.0
    assert np.abs(np.stack([O.wkv_rule(r[:, a], k2[:, a], v[:, a], dec[:, a], u[a]) for a in range(H)], 1)[-1] - want[-1]).max() > 5.0
    rd, kd, vd, dd, ud = dev(r), dev(k), dev(v), dev(dec), dev(u)
    out, state, w = zeros(T, H * D), dev(np.full((H, D, D), 3.0)), H * D
    for at, n in portions(T, sizes):
        ok(L().yalm_state_scan_bonus_rows(ptr(out[at:]), w, ptr(kd[at:]), w, ptr(rd[at:]), w, ptr(vd[at:]), w, ptr(dd[at:]), w, ptr(ud), ptr(state), n, H, D, D, at, None, None),
           "state_scan_bonus_rows")
    close_enough(out.cpu().numpy().reshape(T, H, D), want)


@pytest.mark.parametrize("dt,tt", DTYPES)
@pytest.mark.parametrize("H,D,rank", [(3, 12, 5), (2, 64, 16), (1, 130, 64), (4, 8, 40), (1, 24, 90)])
def test_time_mixing_decode_rows_in_one_launch(H, D, rank, dt, tt):
    T, hd, eps = 40, H * D, 1e-5
    rng = np.random.default_rng(rank)
    z = rng.standard_normal((T, 4 * hd + rank + 2))
    w2, w0, u, nw = O.bf16_round(rng.standard_normal((hd, rank)) / math.sqrt(rank)), rng.standard_normal(hd) - 2.0, rng.standard_normal((H, D)), 1 + 0.3 * rng.standard_normal(hd)
    r, k, v = (z[:, i * hd:(i + 1) * hd].reshape(T, H, D) for i in range(3))
    dec = np.exp(-np.exp(np.tanh(z[:, 4 * hd:4 * hd + rank]) @ w2.T + w0)).reshape(T, H, D)
    o = np.stack([O.wkv_rule(r[:, a], k[:, a], v[:, a], dec[:, a], u[a]) for a in range(H)], 1)
    want = O.rms(o, eps).reshape(T, hd) * nw * O.silu(z[:, 3 * hd:4 * hd])
    zd, wd, bd, ud, nd = dev(z), dev(w2, tt), dev(w0), dev(u), dev(nw)
    out, state = zeros(T, hd), dev(np.full((H, D, D), 3.0))
    for t in range(T):
        ok(L().yalm_wkv_step(ptr(out[t:]), ptr(state), ptr(zd[t:]), 0, hd, 2 * hd, 3 * hd, 4 * hd, ptr(wd), ptr(bd), ptr(ud), ptr(nd), dt, H, D, rank, f32(eps), t, None, None), "wkv_step")
    close_enough(out.cpu().numpy(), want)


# ---- attention ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cache_f32", [1, 0])
@pytest.mark.parametrize("dk,dv,rot_dims", [(16, 24, 8), (48, 40, 48), (20, 8, 0), (72, 96, 24), (10, 7, 6)])
def test_bias_rotation_norm_append(dk, dv, rot_dims, cache_f32):
    rng = np.random.default_rng(dk)
    nq, nk, T, ring, eps = 6, 3, 23, 32, 1e-2                 # an eps that matters
    ld, o_k, o_v = (nq + nk) * dk + nk * dv + 3, nq * dk, (nq + nk) * dk
    P, b = 0.3 * rng.standard_normal((T, ld)), rng.standard_normal(ld - 3)
    f = O.rotary_freqs({"dims": rot_dims, "base": 50.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 16}}) if rot_dims else np.zeros(0)
    z = P[:, :ld - 3] + b
    turn = lambda x: np.stack([O.rms(O.rotate_pairs(x[t], t, f), eps) for t in range(T)])
    want_q, want_k, want_v = turn(z[:, :o_k].reshape(T, nq, dk)), turn(z[:, o_k:o_v].reshape(T, nk, dk)), z[:, o_v:].reshape(T, nk, dv)
    ct = torch.float32 if cache_f32 else torch.bfloat16
    Pd, bd, fd = dev(P), dev(b), dev(f) if rot_dims else None
    kr, vr = zeros(nk, ring, dk, dtype=ct), zeros(nk, ring, dv, dtype=ct)
    for at, n in portions(T, [1, 2, 7, 5]):
        ok(L().yalm_head_bias_rope_norm_append_rows(ptr(Pd[at:]), ld, 0, o_k, o_v, nq, nk, nk, dk, dv, ptr(bd), ptr(bd, o_k), ptr(bd, o_v), ptr(fd), f32(1.0), rot_dims, 1,
                                                    f32(eps), ptr(kr), ptr(vr), ring, cache_f32, n, at, None, None), "head_bias_rope_norm_append_rows")
    tol = F32_TOL if cache_f32 else 1e-2
    close_enough(Pd.cpu().numpy()[:, :o_k].reshape(T, nq, dk), want_q)
    close_enough(kr.float().cpu().numpy()[:, :T], want_k.transpose(1, 0, 2), tol)
    close_enough(vr.float().cpu().numpy()[:, :T], want_v.transpose(1, 0, 2), tol)


@pytest.mark.parametrize("sizes,mma", [([1], 0), ([2, 3], 0), ([400], 0), ([400], 1), ([70, 16, 33], 1)])
def test_far_keys_and_sinks(sizes, mma):
    """Four hundred unit-RMS keys; every query asks, with a score far above the rest, for one key: position 0, 1, its own, or hundreds
    back.  One head has a heavy sink, one a negligible one."""
    T, H, G, d, dv, scale, cache_f32 = 400, 4, 2, 64, 32, 0.5, 0
    rng = np.random.default_rng(7)
    k, v = O.bf16_round(O.rms(rng.standard_normal((T, G, d)), 1e-6)), O.bf16_round(rng.standard_normal((T, G, dv)))
    q = np.zeros((T, H, d))
    for t in range(T):
        for h in range(H):
            q[t, h] = k[[0, min(1, t), t, t // 3][(h + t) % 4], h // 2]          # score d * scale = 32; others around +-4
    q = O.bf16_round(q)
    sink = np.array([-50.0, 40.0, 2.0, 31.0])
    want = np.zeros((T, H, dv))
    for t in range(T):
        for h in range(H):
            want[t, h] = O.softmax_with_sink((k[:t + 1, h // 2] @ q[t, h]) * scale, sink[h]) @ v[:t + 1, h // 2]
    assert np.abs(want[:, 1]).max() < 0.01 and np.abs(want[8, 0] - v[0, 0]).max() < 0.05
    kr, vr = dev(k.transpose(1, 0, 2), torch.bfloat16), dev(v.transpose(1, 0, 2), torch.bfloat16)
    qd, sk, out = dev(q.reshape(T, -1)), dev(sink), zeros(T, H * dv)
    ws = zeros(int(L().yalm_attn_window_pool_workspace(dv)))
    for at, n in portions(T, sizes):
        if mma:
            ok(L().yalm_attn_window_pool_mma_sink(ptr(out[at:]), H * dv, ptr(qd[at:]), H * d, ptr(kr), ptr(vr), None, None, n, H, G, d, dv, T, 0, 0, 0, f32(scale), at, None, ptr(sk),
                                                  G, None), "attn_window_pool_mma_sink")
        else:
            ok(L().yalm_attn_window_pool_sink(ptr(out[at:]), H * dv, ptr(qd[at:]), H * d, ptr(kr), d, ptr(vr), dv, None, None, ptr(ws), n, H, G, d, dv, T, 0, 0, 0, f32(scale),
                                              cache_f32, T, at, None, ptr(sk), G, None), "attn_window_pool_sink")
    close_enough(out.cpu().numpy().reshape(T, H, dv), want, 1e-2)


# ---- the block's products ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("per_channel", [0, 1, None])
def test_output_products_input(per_channel):
    rng = np.random.default_rng(3)
    n, H, P, ff, ld = 5, 3, 20, 37, 150
    o, z = rng.standard_normal((n, H * P)), rng.standard_normal((n, ld))
    nw = 1 + 0.3 * rng.standard_normal(H * P if per_channel else P)
    K = H * P + ff
    left = o
    if per_channel is not None:
        left = (O.rms(o.reshape(n, H, P), 1e-2) * (nw.reshape(H, P) if per_channel else nw)).reshape(n, -1) * O.silu(z[:, 2:2 + H * P])
    want = np.concatenate([left, O.silu(z[:, 70:70 + ff]) * z[:, 70 + ff:70 + 2 * ff]], 1)
    od, zd, nd = dev(o), dev(z), dev(nw)
    out, o16 = zeros(n, K + 1), zeros(n, K + 1, dtype=torch.bfloat16)
    norm = ptr(nd) if per_channel is not None else None
    ok(L().yalm_block_out_rows(ptr(out), ptr(o16), 1, K + 1, ptr(od), H * P, ptr(zd, 2), ptr(zd, 70), ld, norm, P if per_channel else 0, f32(1e-2), n, H, P, ff, 1, None), "block_out_rows")
    close_enough(out.cpu().numpy()[:, :K], want)
    close_enough(o16.float().cpu().numpy()[:, :K], want, 1e-2)


@pytest.mark.parametrize("dt,tt", DTYPES)
@pytest.mark.parametrize("W,segs,plain", [(96, [17, 40, 41, 90], 0b0010), (48, [7], 1), (2048, [300, 700, 1500, 1516], 0b0100), (320, [3000], 1)])
def test_decode_product_with_the_norm_and_the_blends_inside(W, segs, plain, dt, tt):
    rng = np.random.default_rng(W)
    T, d, eps = 4, segs[-1], 1e-5
    x, g, b, mu = 3.0 + rng.standard_normal((T, W)), 1 + 0.3 * rng.standard_normal(W), rng.standard_normal(W), rng.standard_normal((len(segs), W))
    w = O.bf16_round(rng.standard_normal((d, W)) / math.sqrt(W))
    h = O.layer_norm(x, g, b, eps)
    prev = np.concatenate([np.zeros((1, W)), h[:-1]])
    want, at = np.zeros((T, d)), 0
    for s, end in enumerate(segs):
        want[:, at:end] = (h if plain >> s & 1 else h + (prev - h) * mu[s]) @ w[at:end].T
        at = end
    wd, gd, bd, md, state = dev(w, tt), dev(g), dev(b), dev(mu), dev(np.full((2, W), 9.0))
    ends = (C.c_int * len(segs))(*segs)
    out = zeros(T, d)
    for t in range(T):
        xd = dev(x[t])
        ok(L().yalm_gemv_block_in(ptr(out[t:]), ptr(xd), ptr(wd), W, d, dt, ptr(gd), ptr(bd), f32(eps), len(segs), ends, ptr(md), plain, ptr(state), t, None, None), "gemv_block_in")
    close_enough(out.cpu().numpy(), want)
    close_enough(state.cpu().numpy()[(T - 1) & 1], h[T - 1])


@pytest.mark.parametrize("dt,tt", DTYPES)
@pytest.mark.parametrize("n1,ff,d", [(64, 40, 96), (24, 0, 50), (512, 3000, 2048)])
def test_decode_product_with_the_activation_and_the_residual_inside(n1, ff, d, dt, tt):
    rng = np.random.default_rng(d)
    x1, gu, res, add = rng.standard_normal(n1), rng.standard_normal(2 * ff), rng.standard_normal(d), rng.standard_normal(d)
    w = O.bf16_round(rng.standard_normal((d, n1 + ff)) / math.sqrt(n1 + ff))
    want = res + w @ np.concatenate([x1, O.silu(gu[:ff]) * gu[ff:]])
    x1d, gud, wd, ad = dev(x1), dev(gu), dev(w, tt), dev(add)
    for a, extra in ((None, 0.0), (ad, add)):
        rd = dev(res)
        ok(L().yalm_gemv_block_out(ptr(rd), ptr(x1d), n1, ptr(gud) if ff else None, ff, 1, ptr(wd), d, dt, ptr(a), None), "gemv_block_out")
        close_enough(rd.cpu().numpy(), want + extra)


@pytest.mark.parametrize("M,K,segs", [(40, 64, [128, 132, 400, 405]), (200, 320, [256, 512, 768, 1024, 1536, 1552]), (128, 72, [60])])
def test_tensor_core_product_with_one_input_per_segment(M, K, segs):
    rng = np.random.default_rng(M)
    N, S = segs[-1], len(segs)
    a, w = O.bf16_round(rng.standard_normal((S, M, K))), O.bf16_round(rng.standard_normal((N, K)) / math.sqrt(K))
    want, at = np.zeros((M, N)), 0
    for s, end in enumerate(segs):
        want[:, at:end], at = a[s] @ w[at:end].T, end
    ldc = (N + 11) // 4 * 4
    c, ad, wd = dev(np.full((M, ldc), 5.0)), dev(a, torch.bfloat16), dev(w, torch.bfloat16)
    ok(L().yalm_gemm_16_segments(ptr(c), ldc, ptr(ad), ptr(wd), M, N, K, S, (C.c_int * S)(*segs), 1, None), "gemm_16_segments")
    got = c.cpu().numpy()
    close_enough(got[:, :N], want)
    assert (got[:, N:] == 5.0).all()


# ---- small models -----------------------------------------------------------------------------------------------------------------
def open_model(folder, dtype=api.F32, chunk=None, context=0):
    old = os.environ.get("YALM_STACK_CHUNK")
    if chunk is not None:
        os.environ["YALM_STACK_CHUNK"] = str(chunk)
    try:
        m = api.Model(folder, context, dtype).cuda(0)
    finally:
        if chunk is not None:
            if old is None:
                del os.environ["YALM_STACK_CHUNK"]
            else:
                os.environ["YALM_STACK_CHUNK"] = old
    return m, api.InferenceState(m)


def close(m, s):
    s.close()
    m.close()


def checkpoint(tmp_path, cfg, seed=0, **kw):
    W = O.make_weights(cfg, seed, **kw)
    folder = str(tmp_path / ("m%d" % seed))
    O.write_checkpoint(folder, cfg, W)
    return folder, W


_oracle_runs = {}


def oracle_forward(cfg, W, toks):
    key = (json.dumps(cfg, sort_keys=True), float(sum(np.abs(v).sum() for v in W.values())), tuple(toks))
    if key not in _oracle_runs:
        _oracle_runs[key] = O.forward(cfg, W, toks)
    return _oracle_runs[key]


def tokens_for(cfg, n, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def five_layers(**kw):
    kw.setdefault("loop", (1, 4, 2))
    return O.make_config([
        O.attention_mixer(),
        O.wkv_mixer(),
        O.delta_mixer(),
        dict(O.attention_mixer(heads=4, kv_heads=1, dim=24, vdim=8, rot_dims=24, scaling=False), mlp=None),
        O.delta_mixer(heads=3, kv_heads=3, dim=8, vdim=40, conv=5),
    ], **kw)


ONE_LAYER = {
    "delta rule": [O.delta_mixer()],
    "delta rule, one head, one tap, no feed-forward": [dict(O.delta_mixer(heads=1, kv_heads=1, dim=16, vdim=16, conv=1), mlp=None)],
    "delta rule, one key head, two taps": [O.delta_mixer(heads=6, kv_heads=1, dim=40, vdim=8, conv=2)],
    "attention": [O.attention_mixer()],
    "attention, one key head, whole heads rotated without scaling": [O.attention_mixer(heads=3, kv_heads=1, dim=12, vdim=40, rot_dims=12, scaling=False)],
    "attention, every head its own keys, sharp scores, no feed-forward": [dict(O.attention_mixer(heads=2, kv_heads=2, scale=1.2), mlp=None)],
    "attention, nothing rotated": [O.attention_mixer(heads=4, kv_heads=2, dim=8, vdim=8, rot_dims=0, scaling=False)],
    "time mixing": [O.wkv_mixer()],
    "time mixing, one head, no feed-forward": [dict(O.wkv_mixer(heads=1, dim=40, rank=16), mlp=None)],
    "time mixing, many small heads, a rank of one": [O.wkv_mixer(heads=8, dim=4, rank=1)],
}


@pytest.mark.parametrize("name", list(ONE_LAYER))
@pytest.mark.parametrize("buckets,loop", [(53, None), (0, (0, 1, 3)), (1, (0, 1, 2))])
def test_one_layer_models(tmp_path, name, buckets, loop):
    cfg = O.make_config(ONE_LAYER[name], buckets=buckets, loop=loop)
    folder, W = checkpoint(tmp_path, cfg, seed=3)
    T = 40
    toks = tokens_for(cfg, T)
    want, after = O.forward(cfg, W, toks)
    m, s = open_model(folder, context=64)
    buf = np.zeros((len(after), T, cfg["width"]), np.float32)
    m.stack_tap(buf)
    got = s.forward_rows(toks, 0, range(T))
    m.stack_tap(None)
    s.end_sequence()
    dec = np.concatenate([s.forward_rows(toks[t:t + 1], t, [0]) for t in range(T)])
    close(m, s)
    close_enough(buf, after)
    close_enough(got, want)
    close_enough(dec, want)


@pytest.mark.parametrize("loop", [None, (1, 4, 2), (0, 5, 2), (2, 3, 4), (4, 5, 3)])
def test_every_layer_run_of_a_mixed_model(tmp_path, loop):
    cfg = five_layers(loop=loop)
    folder, W = checkpoint(tmp_path, cfg, seed=5)
    T = 50
    toks = tokens_for(cfg, T)
    want, after = oracle_forward(cfg, W, toks)
    m, s = open_model(folder, context=64)
    buf = np.zeros((len(after), T, cfg["width"]), np.float32)
    m.stack_tap(buf)
    got = s.forward_rows(toks, 0, range(T))
    s.end_sequence()
    for t in range(T):                                          # the taps of decode rows too: the pass's addition comes after the tap
        one = np.zeros((len(after), 1, cfg["width"]), np.float32)
        m.stack_tap(one)
        s.forward_rows(toks[t:t + 1], t, [])
        close_enough(one[:, 0], after[:, t])
    m.stack_tap(None)
    close(m, s)
    for i in range(len(after)):
        close_enough(buf[i], after[i])
    close_enough(got, want)


@pytest.mark.parametrize("dtype,tol", [(api.F32, F32_TOL), (api.BF16, 5e-2)])
def test_sizes_that_are_no_vector_multiple(tmp_path, dtype, tol):
    """Nothing here is a multiple of 8 (some not of 4): every op takes its scalar route, rows of caches and weights start at odd offsets."""
    cfg = O.make_config([
        O.delta_mixer(heads=3, kv_heads=1, dim=10, vdim=14, conv=4),
        O.attention_mixer(heads=3, kv_heads=1, dim=10, vdim=6, rot_dims=4),
        O.wkv_mixer(heads=3, dim=7, rank=3),
        O.attention_mixer(heads=5, kv_heads=5, dim=6, vdim=11, rot_dims=6, scaling=False),
    ], width=54, vocab=51, ff=37, loop=(1, 3, 2))
    folder, W = checkpoint(tmp_path, cfg, seed=12)
    T = 45
    toks = tokens_for(cfg, T)
    want, _ = O.forward(cfg, W, toks)
    m, s = open_model(folder, dtype, context=64)
    whole = s.forward_rows(toks, 0, range(T))
    s.end_sequence()
    parts = np.concatenate([s.forward_rows(toks[at:at + n], at, range(n)) for at, n in portions(T, [1, 2, 33, 1, 5])])
    close(m, s)
    close_enough(whole, want, tol)
    close_enough(parts, want, tol)


def edited(cfg, **path):
    out = json.loads(json.dumps(cfg))
    for k, v in path.items():
        at = out
        keys = k.split("__")
        for p in keys[:-1]:
            at = at[int(p[1:])] if p[0] == "_" else at[p]
        at[keys[-1]] = v
    return out


def test_what_is_left_out_would_show(tmp_path):
    """The random weights are such that the mechanisms matter: the oracle with one of them changed differs from the library by far
    more than the tolerance."""
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=6)
    T = 60
    toks = tokens_for(cfg, T)
    m, s = open_model(folder, context=64)
    got = s.forward_rows(toks, 0, range(T))
    close(m, s)
    close_enough(got, O.forward(cfg, W, toks)[0])

    def differs(c, w, least=0.02):
        assert np.abs(O.forward(c, w, toks)[0] - got).max() > least
    differs(cfg, dict(W, **{"l0.mix.sink": np.full(6, -80.0)}))
    differs(cfg, dict(W, **{"l0.mix.v.b": W["l0.mix.v.b"] * 0}))
    differs(cfg, dict(W, **{"l0.norm1.b": W["l0.norm1.b"] * 0}))
    differs(cfg, dict(W, **{"l1.mix.u": np.ones((3, 12))}))
    differs(cfg, dict(W, **{"l1.mix.mu.w": W["l1.mix.mu.w"] * 0}))
    differs(cfg, dict(W, **{"l2.mix.q.conv": np.roll(W["l2.mix.q.conv"], 1, 1)}))
    differs(cfg, dict(W, **{"l2.mix.A_log": W["l2.mix.A_log"] + 0.5}))
    differs(edited(cfg, loop__times=1), W)
    differs(edited(cfg, loop__times=3), W)
    differs(edited(cfg, embedding__bigram__mul_cur=6), W)
    differs(edited(cfg, layers___0__mixer__rot__scaling__factor=1.0), W)
    differs(edited(cfg, layers___0__mixer__rot__base=310.0), W)
    differs(edited(cfg, norm__eps=1e-1), W)


@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 11, 2, 5], [17, 64]])
def test_whole_prompt_equals_decoding_equals_portions(tmp_path, sizes):
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=7)
    T = 90
    toks = tokens_for(cfg, T)
    want, _ = oracle_forward(cfg, W, toks)
    m, s = open_model(folder, context=96)
    whole = s.forward_rows(toks, 0, range(T))
    s.end_sequence()
    parts = np.concatenate([s.forward_rows(toks[at:at + n], at, range(n)) for at, n in portions(T, sizes)])
    close(m, s)
    close_enough(whole, want)
    close_enough(parts, want)
    close_enough(parts, whole.astype(np.float64))


@pytest.mark.parametrize("decode", [False, True])
def test_caches_and_states_given_back_and_used_again(tmp_path, decode):
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=8)
    a, b = tokens_for(cfg, 70, 2), tokens_for(cfg, 33, 3)

    def run(s):
        if decode:
            return np.concatenate([s.forward_rows(b[t:t + 1], t, [0]) for t in range(len(b))])
        return s.forward_rows(b, 0, range(len(b)))
    m, s = open_model(folder, chunk=16, context=96)
    s.forward_rows(a, 0, [])
    s.end_sequence()
    second = run(s)
    s.end_sequence()
    m2, s2 = open_model(folder, chunk=16, context=96)
    alone = run(s2)
    close(m2, s2)
    close(m, s)
    np.testing.assert_array_equal(second, alone)                 # nothing of the earlier sequence is read
    close_enough(second, oracle_forward(cfg, W, b)[0])


@pytest.mark.parametrize("chunk", [1, 4, 16])
def test_long_decoding(tmp_path, chunk):
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=9)
    T = 230
    toks = tokens_for(cfg, T)
    want, _ = oracle_forward(cfg, W, toks)
    m, s = open_model(folder, chunk=chunk, context=T)             # the last position fills the rings exactly
    rows = sorted(set(list(range(0, T, 7)) + [T - 1]))
    close_enough(s.forward_rows(toks, 0, rows), want[rows])
    s.end_sequence()
    s.forward_rows(toks[:20], 0, [])
    dec = np.concatenate([s.forward_rows(toks[i:i + 1], i, [0]) for i in range(20, T)])
    with pytest.raises(api.YalmError):
        s.forward_rows(toks[:1], T, [0])                          # past the context
    close(m, s)
    close_enough(dec, want[20:])


def test_prompt_portions_on_the_tensor_cores_and_serving_precision(tmp_path):
    """Head sizes and portions that take the tensor-core products and attention kernels; bf16 against the float64 run, and
    whole = decoded in bf16."""
    cfg = O.make_config([
        O.delta_mixer(heads=4, kv_heads=2, dim=32, vdim=48, conv=4),
        O.attention_mixer(heads=4, kv_heads=2, dim=64, vdim=64, rot_dims=32, base=5000.0, scale=0.1),
        O.wkv_mixer(heads=3, dim=64, rank=24),
        O.attention_mixer(heads=2, kv_heads=1, dim=128, vdim=32, rot_dims=64, base=5000.0, scale=0.08),
    ], width=136, vocab=160, ff=264, loop=(1, 4, 2))
    folder, W = checkpoint(tmp_path, cfg, seed=10)
    T = 150
    toks = tokens_for(cfg, T)
    want, _ = O.forward(cfg, W, toks)
    m, s = open_model(folder, api.F32, context=192)
    close_enough(s.forward_rows(toks, 0, range(T)), want)
    close(m, s)
    m, s = open_model(folder, api.BF16, context=192)
    whole = s.forward_rows(toks, 0, range(T))
    s.end_sequence()
    cut = np.concatenate([s.forward_rows(toks[at:at + n], at, range(n)) for at, n in portions(T, [70, 2, 33, 45])])
    s.end_sequence()
    s.forward_rows(toks[:100], 0, [])
    dec = np.concatenate([s.forward_rows(toks[i:i + 1], i, [0]) for i in range(100, T)])
    close(m, s)

    def rows_close(got, ref):
        e = np.abs(got - ref).max(1) / max(1.0, np.abs(ref).max())
        assert np.median(e) < 2e-2 and e.max() < 6e-2, (float(np.median(e)), float(e.max()))
    rows_close(whole, want)
    rows_close(cut, want)
    rows_close(dec, want[100:])


def test_decode_rows_with_and_without_the_fused_launches(tmp_path):
    """The same decode rows through the separate ops (YALM_STACK_FUSE=0, in a process of its own) and the fused ones."""
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=13)
    toks = tokens_for(cfg, 30)
    want, _ = oracle_forward(cfg, W, toks)
    code = ("import sys, numpy as np; sys.path.insert(0, %r); from yalm_b200 import api; m = api.Model(%r, 64, api.F32).cuda(0); s = api.InferenceState(m); toks = %r; "
            "np.save(%r, np.concatenate([s.forward_rows(toks[t:t + 1], t, [0]) for t in range(len(toks))]))") % (ROOT, folder, toks, str(tmp_path / "o.npy"))
    for fuse in ("0", "1"):
        r = subprocess.run([sys.executable, "-c", code], env=dict(os.environ, YALM_STACK_FUSE=fuse, YALM_B200_LIB=api.LIB_PATH), capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        close_enough(np.load(tmp_path / "o.npy"), want)


def test_generation_through_the_entry_points(tmp_path):
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=11)
    prompt, n = tokens_for(cfg, 21), 14
    want = O.greedy(cfg, W, prompt, n)
    m, s = open_model(folder, context=128)
    assert s.generate(prompt, n) == want
    s.end_sequence()
    s.forward_batch(prompt[:-1], 0)
    assert s.generate_greedy(prompt[-1], len(prompt) - 1, n) == want      # the captured decode step, replayed
    s.end_sequence()
    s.forward_batch(prompt[:-1], 0)
    toks, lg = s.generate_greedy(prompt[-1], len(prompt) - 1, n, keep_logits=True)
    assert toks == want
    close_enough(lg, O.forward(cfg, W, prompt + want)[0][len(prompt) - 1:-1])
    s.end_sequence()
    s.forward_batch(prompt[:-1], 0)
    a = s.generate_sampled(prompt[-1], len(prompt) - 1, n, 0.8, seed=5)
    s.end_sequence()
    s.forward_batch(prompt[:-1], 0)
    b = s.generate_sampled(prompt[-1], len(prompt) - 1, n, 0.8, seed=5)
    close(m, s)
    assert a == b and all(0 <= t < cfg["vocab"] for t in a)


def test_command_line_on_a_checkpoint_directory(tmp_path):
    exe = os.path.join(ROOT, "build", "main")
    if not os.path.exists(exe):
        subprocess.check_call(["make", "-s", "-C", ROOT, "cli"])
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=15)
    prompt = tokens_for(cfg, 17)
    text = " ".join(map(str, prompt))
    r = subprocess.run([exe, folder, "-m", "completion", "-i", text, "-n", "6", "-t", "0", "-p", "fp32"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    ids = [l for l in r.stdout.splitlines() if re.fullmatch(r"(\d+ )+", l)]
    assert ids and [int(x) for x in ids[-1].split()] == O.greedy(cfg, W, prompt, 6)


def test_trace_runner(tmp_path):
    cfg = five_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=14)
    a, b = tokens_for(cfg, 25, 4), tokens_for(cfg, 9, 5)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [19, 3, 19]}], "end": []},   # rows come in the order asked
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[22:], "want": [2]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [8]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    env = dict(os.environ, YALM_B200_LIB=api.LIB_PATH)
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", 5e-2)):
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "25"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == ["done 0", "done 1", "done 2", "done 3"]
        wa, wb = O.forward(cfg, W, a)[0], O.forward(cfg, W, b)[0]
        V = cfg["vocab"]
        close_enough(np.fromfile(out / "0.f32", "<f4").reshape(-1, V), wa[[19, 3, 19]], tol)
        assert not (out / "1.f32").exists()
        close_enough(np.fromfile(out / "2.f32", "<f4").reshape(-1, V), wa[[24]], tol)
        close_enough(np.fromfile(out / "3.f32", "<f4").reshape(-1, V), wb[[8]], tol)
        for f in out.iterdir():
            f.unlink()
