"""-m gpu: the Desalorn design on the layered executor against the plain float64 statement in desalorn_oracle.py.

The new row ops alone (device arrays through the C ABI): norms in groups, with and without the residual add before them; the router
over groups ranked by their two best choice scores (negative scores, groups that only the sum or only the best would keep);
biases + whole-projection norm + cache append; attention with mixed head scores on its three routes (every distance bucket's edges, a
key hundreds of positions back, a window's edges, scores taken from another head only); retention as a scan over portions and as
fused decode rows, with a key that stands out far back.  Then small models with random weights whose sizes differ from layer to
layer: every mechanism through the residual after its layer; whole prompts against token-by-token decoding and portions down to two
tokens; caches given back and used again; long decoding past the window many times over; tensor-core prompt routes and serving
precision; greedy generation through the library's entry points, the command line and the trace runner.
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

import desalorn_oracle as O
from yalm_b200 import api

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 3e-4
vp, i32, f32, sz = C.c_void_p, C.c_int, C.c_float, C.c_size_t
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
    lib.yalm_attn_mixed_workspace.restype = C.c_size_t
    return lib


# ---- norms in groups ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W,groups", [(48, 1), (48, 3), (50, 5), (40, 40), (2048, 2), (1040, 13), (3000, 1), (96, 48)])
@pytest.mark.parametrize("n", [1, 5])
def test_group_norm_and_residual_add(W, groups, n):
    rng = np.random.default_rng(W + groups)
    eps, mult, top = 1e-2, 0.7, 3                                  # an eps that matters, in small parts above all
    x = rng.standard_normal((n, W)) * np.repeat(10.0 ** rng.uniform(-2, 1, groups), W // groups)      # parts of very different size
    w, a, ab, b, y = 1 + 0.3 * rng.standard_normal(W), *(rng.standard_normal(s) for s in ((n, W), (W,), (n, W), (n, top, W)))
    wd, ad, abd, bd, yd = dev(w), dev(a), dev(ab), dev(b), dev(y)
    xd, out, o16 = dev(x), zeros(n, W), zeros(n, W, dtype=torch.bfloat16)
    ok(L().yalm_group_norm_rows(ptr(out), ptr(o16), 1, ptr(xd), None, ptr(wd), groups, f32(eps), n, W, None), "group_norm_rows")
    want = O.group_norm(np.float32(x).astype(np.float64), w, groups, eps)
    close_enough(out.cpu().numpy(), want)
    close_enough(o16.float().cpu().numpy(), want, 1e-2)
    if groups > 1 and W // groups > 1:
        assert np.abs(O.group_norm(x, w, 1, eps) - want).max() > 0.1
    if n > 1:
        rows, two = dev([3, 1], torch.int32), zeros(2, W)
        ok(L().yalm_group_norm_rows(ptr(two), None, 0, ptr(xd), ptr(rows), ptr(wd), groups, f32(eps), 2, W, None), "group_norm_rows gathered")
        close_enough(two.cpu().numpy(), want[[3, 1]])
    for parts in ((1, 1, 1, 1), (1, 0, 0, 0), (1, 1, 1, 0), (0, 0, 0, 1)):
        xd = dev(x)
        s = parts[0] * a + parts[1] * ab + parts[2] * b + parts[3] * y.sum(1)
        ok(L().yalm_residual_group_norm_rows(ptr(xd), f32(mult), ptr(ad) if parts[0] else None, ptr(abd) if parts[1] else None, ptr(bd) if parts[2] else None,
                                             ptr(yd) if parts[3] else None, W, top if parts[3] else 0, ptr(out), None, 0, ptr(wd), groups, f32(eps), n, W, None), "residual + norm")
        close_enough(xd.cpu().numpy(), x + mult * s, 1e-5)
        close_enough(out.cpu().numpy(), O.group_norm(x + mult * s, w, groups, eps))
        xd = dev(x)
        ok(L().yalm_residual_group_norm_rows(ptr(xd), f32(mult), ptr(ad), None, None, None, 0, 0, None, None, 0, None, groups, f32(eps), n, W, None), "residual alone")
        close_enough(xd.cpu().numpy(), x + mult * a, 1e-5)


# ---- router -------------------------------------------------------------------------------------------------------------------
def router_call(x, wr, bias, top, count, keep, group_top=2, dt=api.F32, tt=torch.float32):
    n, W = x.shape
    E = wr.shape[0]
    xd, wd, bd, ids, wts = dev(x), dev(wr, tt), dev(bias), zeros(n, top, dtype=torch.int32), zeros(n, top)
    ok(L().yalm_router_group_topk_rows(ptr(ids), ptr(wts), ptr(xd), W, ptr(wd), dt, n, E, top, W, 1, 0, f32(0), count, keep, group_top, ptr(bd), f32(1.0), None), "router")
    return ids.cpu().numpy(), wts.cpu().numpy()


@pytest.mark.parametrize("E,top,count,keep", [(6, 2, 3, 2), (12, 4, 2, 1), (8, 3, 8, 4), (5, 5, 1, 1), (64, 8, 8, 3), (300, 6, 6, 2), (9, 1, 3, 1)])
@pytest.mark.parametrize("dt,tt", DTYPES)
def test_router_over_groups(E, top, count, keep, dt, tt):
    rng = np.random.default_rng(E)
    n, W = 40, 48
    x, wr = rng.standard_normal((n, W)), O.bf16_round(2.0 * rng.standard_normal((E, W)) / math.sqrt(W))
    for mean in (0.0, -3.0):                                       # -3: every choice score is negative, a closed group must not win with zeros
        bias = mean + 0.3 * rng.standard_normal(E)
        ids, wts = router_call(x, wr, bias, top, count, keep, dt=dt, tt=tt)
        s = 1.0 / (1.0 + np.exp(-(np.float32(x).astype(np.float64) @ wr.T)))
        want = np.stack([O.choose(s[t] + bias, top, count, keep) for t in range(n)])
        np.testing.assert_array_equal(ids, want)
        close_enough(wts, np.take_along_axis(s, want, 1), 1e-5)


def test_router_ranks_groups_by_their_two_best():
    """Group 0 has the best expert, group 1 the best pair, group 2 the best three: two experts rank a group."""
    W = 8
    x, wr = np.zeros((1, W)), np.zeros((9, W))                      # every score is one half: the corrections decide
    bias = np.array([1.0, -2.0, -2.0, 0.6, 0.6, -2.0, 0.55, 0.55, 0.55])
    assert router_call(x, wr, bias, 2, 3, 1)[0].tolist() == [[3, 4]]
    assert router_call(x, wr, bias, 2, 3, 1, group_top=1)[0].tolist() == [[0, 1]]
    assert router_call(x, wr, bias, 2, 3, 1, group_top=3)[0].tolist() == [[6, 7]]
    assert router_call(x, wr, bias, 3, 3, 3)[0].tolist() == [[0, 3, 4]]           # every group kept: the best of all, ties to the lower index
    assert np.allclose(router_call(x, wr, bias, 2, 3, 1)[1], 0.5)                 # the weights leave the correction out


# ---- biases, norm over the whole projection, cache append ---------------------------------------------------------------------
@pytest.mark.parametrize("cache_f32", [1, 0])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 16, 24), (3, 1, 10, 7), (6, 6, 48, 8)])
def test_biases_whole_norm_append(H, G, dk, dv, cache_f32):
    rng = np.random.default_rng(dk)
    T, ring, eps, nq, nk, nv = 23, 16, 1e-2, H * dk, G * dk, G * dv
    ld = nq + nk + nv + 3
    P, b = rng.standard_normal((T, ld)), rng.standard_normal(nq + nk + nv)
    qn, kn = 1 + 0.3 * rng.standard_normal(nq), 1 + 0.3 * rng.standard_normal(nk)
    z = P[:, :ld - 3] + b
    q, k, v = O.rms(z[:, :nq], eps) * qn, O.rms(z[:, nq:nq + nk], eps) * kn, z[:, nq + nk:]
    ct = torch.float32 if cache_f32 else torch.bfloat16
    Pd, bd, qd, kd, kr, vr = dev(P), dev(b), dev(qn), dev(kn), zeros(G, ring, dk, dtype=ct), zeros(G, ring, dv, dtype=ct)
    for at, n in portions(T, [1, 2, 7, 5]):
        ok(L().yalm_qkv_bias_post_rows(ptr(Pd[at:]), ld, ptr(bd), ptr(kr), ptr(vr), None, 0, ptr(qd), ptr(kd), None, 0, n, H, G, dk, dv, ring, f32(eps), cache_f32, at, None, None),
           "qkv_bias_post_rows")
    close_enough(Pd.cpu().numpy()[:, :nq], q)
    tol = F32_TOL if cache_f32 else 1e-2
    for t in range(T - ring, T):                                    # the ring holds the last positions
        close_enough(kr[:, t % ring].float().cpu().numpy(), k[t].reshape(G, dk), tol)
        close_enough(vr[:, t % ring].float().cpu().numpy(), v[t].reshape(G, dv), tol)


# ---- attention with mixed head scores ------------------------------------------------------------------------------------------
def plain_mixed(q, k, v, rel, far, talk, scale, cap, window=0, gate=None):
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        lo = max(0, t - window + 1) if window else 0
        dist = [O.bucket(t - j, rel.shape[0], far) for j in range(lo, t + 1)]
        z = np.stack([k[lo:t + 1, h // (H // G)] @ q[t, h] for h in range(H)]) * scale
        s = talk @ (cap * np.tanh(z / cap) + rel[dist].T)
        for h in range(H):
            out[t, h] = O.softmax(s[h]) @ v[lo:t + 1, h // (H // G)]
    return out if gate is None else out / (1.0 + np.exp(-gate))[:, :, None]


def table(rel, far):
    return np.stack([rel[O.bucket(n, rel.shape[0], far)] for n in range(far + 1)], 1)


ROUTES = ["rows32", "rows16", "decode", "mma"]


def run_mixed(route, q, k, v, rel, far, talk, scale, cap, sizes, window=0, gate=None, ring=None, split=True):
    """The rows in portions; with a ring shorter than the sequence, keys are put there portion by portion as the executor does."""
    T, H, dk = q.shape
    G, dv = k.shape[1], v.shape[2]
    ring = ring or T
    ct = torch.float32 if route == "rows32" else torch.bfloat16
    kr, vr = dev(np.full((G, ring, dk), 9.0), ct), dev(np.full((G, ring, dv), 9.0), ct)      # what other sequences left
    kd, vd = dev(k.transpose(1, 0, 2), ct), dev(v.transpose(1, 0, 2), ct)
    qd, bd, td, out = dev(q.reshape(T, -1)), dev(table(rel, far)), dev(talk), zeros(T, H * dv)
    gd = dev(gate) if gate is not None else None
    nws = int(L().yalm_attn_mixed_workspace(64, H, dv)) if split else 0
    ws = zeros(max(1, nws))
    for at, n in portions(T, sizes):
        slots = torch.arange(at, at + n, device="cuda") % ring
        kr[:, slots], vr[:, slots] = kd[:, at:at + n], vd[:, at:at + n]
        args = [ptr(out[at:]), H * dv, ptr(qd[at:]), H * dk, ptr(kr), ptr(vr), ptr(bd), far + 1, ptr(td), ptr(gd[at:]) if gate is not None else None, H,
                ptr(ws) if split else None, sz(nws), n, H, G, dk, dv, ring, window, f32(scale), f32(cap)]
        if route.startswith("rows"):
            ok(L().yalm_attn_mixed_rows(*args, int(route == "rows32"), T, at, None, None), "attn_mixed_rows")
        else:
            fn = L().yalm_attn_mixed_decode if route == "decode" else L().yalm_attn_mixed_mma
            ok(fn(*args, T, at, None, None), "attn_mixed_" + route)
    return out.cpu().numpy().reshape(T, H, dv)


def mixed_case(T, H, G, dk, dv, rows=10, seed=0):
    rng = np.random.default_rng(seed)
    q, k = O.bf16_round(rng.standard_normal((T, H, dk))), O.bf16_round(rng.standard_normal((T, G, dk)))
    v = O.bf16_round(rng.standard_normal((T, G, dv)))
    return q, k, v, rng.standard_normal((rows, H)), np.eye(H) + 0.4 * rng.standard_normal((H, H)) / math.sqrt(H), 2.0 * rng.standard_normal((T, H))


MIXED = [(4, 2, 16, 32, 10), (8, 2, 64, 96, 18), (3, 1, 32, 16, 7), (6, 6, 48, 80, 4), (16, 4, 128, 128, 32), (20, 4, 32, 48, 12), (1, 1, 16, 16, 2), (2, 1, 64, 128, 9)]


@pytest.mark.parametrize("route,sizes", [("rows32", [1]), ("rows32", [2, 50, 3]), ("rows16", [40, 1, 17]), ("decode", [1]), ("decode", [2, 5]), ("mma", [150]), ("mma", [16, 33, 20, 17])])
@pytest.mark.parametrize("H,G,dk,dv,rows", MIXED)
def test_mixed_attention(H, G, dk, dv, rows, route, sizes):
    T, far, cap = 100, 37, 3.0
    q, k, v, rel, talk, gate = mixed_case(T, H, G, dk, dv, rows, seed=dk + H)
    scale = dk ** -0.5
    want = plain_mixed(q, k, v, rel, far, talk, scale, cap, gate=gate)
    close_enough(run_mixed(route, q, k, v, rel, far, talk, scale, cap, sizes, gate=gate), want, F32_TOL if route.startswith("rows") else 1e-2)
    one = run_mixed(route, q, k, v, rel, far, talk, scale, cap, sizes, gate=gate, split=False)      # one CTA per row, no partials
    close_enough(one, want, F32_TOL if route.startswith("rows") else 1e-2)
    assert np.abs(plain_mixed(q, k, v, rel, far, np.eye(H), scale, cap, gate=gate) - want).max() > 0.03
    assert np.abs(plain_mixed(q, k, v, rel, far, talk, scale, 30.0, gate=gate) - want).max() > 0.03


@pytest.mark.parametrize("route", ["rows32", "decode", "mma"])
def test_every_distance_bucket(route):
    """One bucket at a time gets a bias that outweighs every score: a row then averages the values at exactly that bucket's distances."""
    T, H, G, d, far, rows = 70, 2, 1, 16, 50, 11
    rng = np.random.default_rng(5)
    q, k, v = np.zeros((T, H, d)), np.zeros((T, G, d)), O.bf16_round(rng.standard_normal((T, G, d)))
    for b in range(rows):
        rel = np.zeros((rows, H))
        rel[b] = 40.0
        want = plain_mixed(q, k, v, rel, far, np.eye(H), 1.0, 5.0)
        dist = [n for n in range(T) if O.bucket(n, rows, far) == b]
        np.testing.assert_allclose(want[T - 1, 0], v[[T - 1 - n for n in dist], 0].mean(0), atol=1e-6)
        got = run_mixed(route, q, k, v, rel, far, np.eye(H), 1.0, 5.0, [1] if route == "decode" else [23])
        close_enough(got, want, F32_TOL if route == "rows32" else 1e-2)


@pytest.mark.parametrize("route,sizes", [("rows32", [1]), ("decode", [1]), ("decode", [400]), ("mma", [400]), ("mma", [70, 16, 33])])
def test_a_far_key_through_another_heads_scores(route, sizes):
    """Every row asks, through the query of ONE head, for one key up to hundreds of positions back; the other heads' queries are zero and
    take that head's scores over through the mixing."""
    T, H, G, d = 400, 4, 2, 32
    rng = np.random.default_rng(8)
    k, v = O.bf16_round(O.rms(rng.standard_normal((T, G, d)), 1e-6)), O.bf16_round(rng.standard_normal((T, G, d)))
    q, asked = np.zeros((T, H, d)), np.array([[0, min(1, t), t, t // 3][t % 4] for t in range(T)])
    q[:, 2] = k[asked, 1]
    talk = np.zeros((H, H))
    talk[:, 2] = [1.0, 1.0, 1.0, -1.0]                             # head 3: the key asked for is what it avoids
    rel = np.zeros((4, H))
    want = plain_mixed(q, k, v, rel, 30, talk, 1.0, 60.0)
    np.testing.assert_allclose(want[-2, 0], v[asked[-2], 0], atol=0.05)
    close_enough(run_mixed(route, q, k, v, rel, 30, talk, 1.0, 60.0, sizes), want, F32_TOL if route == "rows32" else 2e-2)


@pytest.mark.parametrize("route,sizes", [("rows32", [1]), ("rows32", [24]), ("rows16", [3]), ("decode", [1]), ("decode", [2]), ("mma", [24]), ("mma", [16])])
@pytest.mark.parametrize("window", [1, 16, 17, 40])
def test_window_edges_over_a_reused_ring(window, route, sizes):
    """Keys just inside and just outside the window stand out, in a ring whose slots are taken over many times."""
    T, H, G, d = 130, 2, 1, 16
    rng = np.random.default_rng(window)
    k, v = O.bf16_round(O.rms(rng.standard_normal((T, G, d)), 1e-6)), O.bf16_round(rng.standard_normal((T, G, d)))
    q = np.zeros((T, H, d))
    for t in range(T):
        q[t, 0], q[t, 1] = 2 * k[max(0, t - window + 1), 0], 2 * k[max(0, t - window), 0]
    rel, talk = np.zeros((4, H)), np.eye(H)
    want = plain_mixed(q, k, v, rel, 9, talk, 1.0, 60.0, window=window)
    if window < 40:
        assert np.abs(plain_mixed(q, k, v, rel, 9, talk, 1.0, 60.0, window=window + 1)[-1, 1] - want[-1, 1]).max() > 0.5
    close_enough(run_mixed(route, q, k, v, rel, 9, talk, 1.0, 60.0, sizes, window=window, ring=64), want, F32_TOL if route == "rows32" else 2e-2)


# ---- retention ----------------------------------------------------------------------------------------------------------------
def retention_case(T, H, D, P, rot, seed=0):
    rng = np.random.default_rng(seed)
    hd, hp = H * D, H * P
    z = rng.standard_normal((T, 2 * hd + 2 * hp + 4))
    decay = 1.0 - 2.0 ** -(1.0 + np.arange(H) * 3.0)
    f = O.rotary_freqs({"dims": rot, "base": 300.0}) if rot else np.zeros(0)
    turn = lambda x: np.stack([O.rotate(x[t], t, f, False) for t in range(T)])
    q, k = turn(z[:, :hd].reshape(T, H, D)), turn(z[:, hd:2 * hd].reshape(T, H, D)) * D ** -0.5
    o = O.retention_scan(q, k, z[:, 2 * hd:2 * hd + hp].reshape(T, H, P), decay)
    out = O.rms(o, 1e-2).reshape(T, hp) * O.silu(z[:, 2 * hd + hp:2 * hd + 2 * hp])
    return z, decay, f, o.reshape(T, hp), out


RET = [(3, 24, 40, 16), (2, 64, 64, 64), (1, 10, 7, 6), (4, 16, 16, 0), (2, 128, 200, 64), (1, 200, 24, 200), (5, 8, 8, 2)]


@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 7], [64], [90]])
@pytest.mark.parametrize("H,D,P,rot", RET)
def test_retention_rows_and_fused_decode_rows(H, D, P, rot, sizes):
    T, hd, hp = 90, H * D, H * P
    z, decay, f, o, out = retention_case(T, H, D, P, rot, seed=D)
    ld, ks = z.shape[1], D ** -0.5
    zd, dd, sd, fd = dev(z), dev(decay), dev(np.full(H, ks)), dev(f) if rot else None
    state, scan, got = dev(np.full((H, P, D), 3.0)), zeros(T, hp), zeros(T, hp)      # the state another sequence left is not read
    keep = zd.clone()
    for at, n in portions(T, sizes):
        if n == 1:
            ok(L().yalm_retention_step(ptr(got[at:]), ptr(state), ptr(keep[at:]), 0, hd, 2 * hd, 2 * hd + hp, ptr(dd), ptr(fd), f32(1.0), rot, 0, f32(ks), H, D, P, f32(1e-2), at,
                                       None, None), "retention_step")
            continue
        ok(L().yalm_rotate_heads_rows(ptr(zd[at:]), ld, 2 * H, D, 0, ptr(fd), f32(1.0), rot, 0, n, at, None, None), "rotate_heads_rows")
        za = zd[at:]
        ok(L().yalm_state_scan_rows(ptr(scan[at:]), hp, ptr(za, hd), ld, ptr(za), ld, ptr(za, 2 * hd), ld, ptr(dd), 0, 0, ptr(sd), 0, None, 0, None, ptr(state), n, H, 1, D, P, at,
                                    None, None), "state_scan_rows")
        ok(L().yalm_head_norm_act_rows(ptr(got[at:]), hp, ptr(scan[at:]), hp, ptr(za, 2 * hd + hp), ld, None, n, H, P, f32(1e-2), 1, None), "head_norm_act_rows")
        close_enough(scan[at:at + n].cpu().numpy(), o[at:at + n])
    close_enough(got.cpu().numpy(), out)


@pytest.mark.parametrize("sizes", [[1], [37, 2], [600]])
def test_retention_recalls_a_far_key(sizes):
    """Six hundred positions without decay: nothing later writes along row 5's key, which the last row's query is."""
    T, D, P = 600, 32, 16
    rng = np.random.default_rng(9)
    k, q, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, P))
    k[5] /= np.linalg.norm(k[5])
    k[:5] -= np.outer(k[:5] @ k[5], k[5])
    k[6:] -= np.outer(k[6:] @ k[5], k[5])
    q[-1] = k[5]
    z = np.concatenate([q, k * D ** 0.5, v, np.full((T, P), 50.0)], 1)          # an open gate
    want = O.rms(O.retention_scan(q[:, None], k[:, None], v[:, None], np.ones(1)), 1e-6)[:, 0] * 50.0
    np.testing.assert_allclose(want[-1] / 50.0, O.rms(v[5], 1e-6), atol=1e-5)
    zd, dd, sd, state, scan, got = dev(z), dev([1.0]), dev([D ** -0.5]), zeros(1, P, D), zeros(T, P), zeros(T, P)
    ld = z.shape[1]
    for at, n in portions(T, sizes):
        za = zd[at:]
        if n == 1:
            ok(L().yalm_retention_step(ptr(got[at:]), ptr(state), ptr(za), 0, D, 2 * D, 2 * D + P, ptr(dd), None, f32(1.0), 0, 0, f32(D ** -0.5), 1, D, P, f32(1e-6), at, None, None),
               "retention_step")
            continue
        ok(L().yalm_state_scan_rows(ptr(scan[at:]), P, ptr(za, D), ld, ptr(za), ld, ptr(za, 2 * D), ld, ptr(dd), 0, 0, ptr(sd), 0, None, 0, None, ptr(state), n, 1, 1, D, P, at, None,
                                    None), "state_scan_rows")
        ok(L().yalm_head_norm_act_rows(ptr(got[at:]), P, ptr(scan[at:]), P, ptr(za, 2 * D + P), ld, None, n, 1, P, f32(1e-6), 1, None), "head_norm_act_rows")
    close_enough(got.cpu().numpy()[-1], want[-1], 1e-3)


# ---- small models -------------------------------------------------------------------------------------------------------------
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


def settled_checkpoint(tmp_path, cfg, seed):
    """Corrections so far apart (powers of two) that rounding never decides between experts or groups: for bf16 against float64."""
    W = O.make_weights(cfg, seed)
    for i, name in enumerate(W):
        if name.endswith("correction"):
            W[name] = np.float32(2.0) ** np.random.default_rng(i).permutation(len(W[name])).astype(np.float32)
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


def six_layers(**kw):
    return O.make_config([
        ("attention", O.attention_mixer(), O.moe_mlp()),
        ("retention", O.retention_mixer(), O.moe_mlp(experts=8, top=3, count=4, keep=2, shared=16)),
        ("latent_attention", O.latent_mixer(), O.moe_mlp(experts=4, top=1, count=1, keep=1, shared=0)),
        ("attention", O.attention_mixer(heads=3, kv_heads=1, dim=24, vdim=8, bias_max=25, softcap=2.0), None),
        ("latent_attention", O.latent_mixer(heads=5, dim=8, rot_dim=8, vdim=16, kv_rank=24, q_rank=16, window=7), O.moe_mlp(experts=6, top=4, count=2, keep=2)),
        ("retention", O.retention_mixer(heads=1, dim=16, vdim=24, rot_dims=16, decay=[0.99]), None),
    ], **kw)


ONE_LAYER = {
    "attention": ("attention", O.attention_mixer(), None),
    "attention, one key head": ("attention", O.attention_mixer(heads=6, kv_heads=1, dim=8, vdim=40, softcap=1.5), None),
    "attention, every head its own keys, sharp scores": ("attention", O.attention_mixer(heads=3, kv_heads=3, scale=1.1, softcap=20.0, bias_max=300), None),
    "attention, one head": ("attention", O.attention_mixer(heads=1, kv_heads=1, dim=40, vdim=16), None),
    "retention": ("retention", O.retention_mixer(), None),
    "retention, one head, all of it rotated": ("retention", O.retention_mixer(heads=1, dim=16, vdim=16, rot_dims=16), None),
    "retention, many heads, values smaller than keys": ("retention", O.retention_mixer(heads=6, dim=40, vdim=8, rot_dims=8), None),
    "latent attention": ("latent_attention", O.latent_mixer(), None),
    "latent attention, window of one": ("latent_attention", O.latent_mixer(window=1), None),
    "latent attention, one head, window beyond the prompt": ("latent_attention", O.latent_mixer(heads=1, dim=8, rot_dim=24, window=500, kv_rank=16), None),
    "experts beside attention": ("attention", O.attention_mixer(heads=2, kv_heads=1), O.moe_mlp()),
    "experts, one group, no shared expert": ("retention", O.retention_mixer(heads=2), O.moe_mlp(experts=5, top=5, count=1, keep=1, shared=0)),
    "experts, groups of one": ("latent_attention", O.latent_mixer(), O.moe_mlp(experts=4, top=2, count=4, keep=3, shared=24)),
}


@pytest.mark.parametrize("name", list(ONE_LAYER))
@pytest.mark.parametrize("groups,mult", [(1, 1.0), (6, 0.45)])
def test_one_layer_models(tmp_path, name, groups, mult):
    cfg = O.make_config([ONE_LAYER[name]], groups=groups, residual_mult=mult)
    folder, W = checkpoint(tmp_path, cfg, seed=3)
    T = 40
    toks = tokens_for(cfg, T)
    want, after = O.forward(cfg, W, toks)
    m, s = open_model(folder, context=64)
    buf = np.zeros((1, T, cfg["width"]), np.float32)
    m.stack_tap(buf)
    got = s.forward_rows(toks, 0, range(T))
    m.stack_tap(None)
    s.end_sequence()
    dec = np.concatenate([s.forward_rows(toks[t:t + 1], t, [0]) for t in range(T)])
    close(m, s)
    close_enough(buf, after)
    close_enough(got, want)
    close_enough(dec, want)


def test_every_layer_of_a_mixed_model(tmp_path):
    cfg = six_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=5)
    T = 50
    toks = tokens_for(cfg, T)
    want, after = oracle_forward(cfg, W, toks)
    m, s = open_model(folder, context=64)
    buf = np.zeros((len(after), T, cfg["width"]), np.float32)
    m.stack_tap(buf)
    got = s.forward_rows(toks, 0, range(T))
    s.end_sequence()
    for t in range(T):
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
        ("attention", O.attention_mixer(heads=3, kv_heads=1, dim=10, vdim=6), None),
        ("retention", O.retention_mixer(heads=3, dim=10, vdim=14, rot_dims=6), O.moe_mlp(ff=13, experts=3, top=3, count=1, keep=1, shared=11)),
        ("latent_attention", O.latent_mixer(heads=3, dim=7, rot_dim=6, vdim=9, kv_rank=19, q_rank=11, window=10), None),
        ("attention", O.attention_mixer(heads=5, kv_heads=5, dim=6, vdim=11), O.moe_mlp(ff=21, experts=2, top=2, count=1, keep=1, shared=0)),
    ], width=54, vocab=51)
    folder, W = checkpoint(tmp_path, cfg, seed=12, rel_rows=9)
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
    cfg = six_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=6)
    T = 60
    toks = tokens_for(cfg, T)
    m, s = open_model(folder, context=64)
    got = s.forward_rows(toks, 0, range(T))
    close(m, s)
    close_enough(got, O.forward(cfg, W, toks)[0])

    def differs(c, w, least=0.02):
        assert np.abs(O.forward(c, w, toks)[0] - got).max() > least
    for name in ("mix.q.b", "mix.k.b", "mix.v.b", "mix.o.b", "mix.g", "mix.rel"):
        differs(cfg, dict(W, **{"l0." + name: W["l0." + name] * 0}))
    differs(cfg, dict(W, **{"l0.mix.talk": np.eye(4)}))
    differs(cfg, dict(W, **{"l0.mix.q.norm": np.ones(64)}))
    differs(cfg, dict(W, **{"l0.mix.rel": np.roll(W["l0.mix.rel"], 1, 0)}))
    differs(cfg, dict(W, **{"l1.mlp.correction": W["l1.mlp.correction"] * 0}))
    differs(cfg, dict(W, **{"l1.mlp.shared.down": W["l1.mlp.shared.down"] * 0}))
    differs(edited(cfg, layers___0__mixer__softcap=100.0), W)
    differs(edited(cfg, layers___0__mixer__bias_max=200), W)
    differs(edited(cfg, layers___1__mixer__decay=[0.5, 0.5, 0.5]), W)
    differs(edited(cfg, layers___1__mixer__rot__base=310.0), W)
    differs(edited(cfg, layers___1__mlp__router__groups={"count": 1, "keep": 1}), W)
    differs(edited(cfg, layers___2__mixer__mask__size=11), W)
    differs(edited(cfg, layers___2__mixer__mask__size=13), W)
    differs(edited(cfg, norm__groups=1), W)
    differs(edited(cfg, norm__eps=1e-1), W)
    differs(edited(cfg, residual_mult=0.65), W)


@pytest.mark.parametrize("sizes", [[1], [2], [3, 2, 11, 2, 5], [17, 64]])
def test_whole_prompt_equals_decoding_equals_portions(tmp_path, sizes):
    cfg = six_layers()
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
    cfg = six_layers()
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
    """The windows' rings are taken over several times; the unbounded layers' rings end exactly at the last position."""
    cfg = six_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=9)
    T = 230
    toks = tokens_for(cfg, T)
    want, _ = oracle_forward(cfg, W, toks)
    m, s = open_model(folder, chunk=chunk, context=T)
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
    """Head sizes and portions that take the tensor-core products, attention kernels and grouped experts; bf16 against the float64 run,
    and whole = portions = decoded in bf16."""
    cfg = O.make_config([
        ("attention", O.attention_mixer(heads=8, kv_heads=2, dim=32, vdim=64, softcap=4.0), O.moe_mlp(ff=64, experts=8, top=2, count=2, keep=1, shared=96)),
        ("latent_attention", O.latent_mixer(heads=4, dim=48, rot_dim=16, vdim=64, kv_rank=64, q_rank=72, window=33), O.moe_mlp(ff=40, experts=6, top=3, count=3, keep=2, shared=48)),
        ("retention", O.retention_mixer(heads=3, dim=64, vdim=48, rot_dims=32), None),
        ("attention", O.attention_mixer(heads=4, kv_heads=4, dim=64, vdim=32, bias_max=90, softcap=9.0), None),
    ], width=136, vocab=160, groups=2)
    folder, W = settled_checkpoint(tmp_path, cfg, seed=10)
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


@pytest.mark.parametrize("switch", ["YALM_STACK_BRANCHES", "YALM_STACK_TC", "YALM_STACK_ATTN_MMA", "YALM_STACK_MOE_TC"])
def test_routes_that_can_be_switched_off(tmp_path, switch):
    """The same rows with one of the faster routes off, in a process of its own."""
    cfg = six_layers(width=96)
    folder, W = settled_checkpoint(tmp_path, cfg, seed=13)
    toks = tokens_for(cfg, 60)
    want, _ = oracle_forward(cfg, W, toks)
    code = ("import sys, numpy as np; sys.path.insert(0, %r); from yalm_b200 import api; m = api.Model(%r, 64, api.BF16).cuda(0); s = api.InferenceState(m); toks = %r; "
            "a = s.forward_rows(toks[:50], 0, range(50)); np.save(%r, np.concatenate([a] + [s.forward_rows(toks[t:t + 1], t, [0]) for t in range(50, 60)]))"
            ) % (ROOT, folder, toks, str(tmp_path / "o.npy"))
    r = subprocess.run([sys.executable, "-c", code], env=dict(os.environ, YALM_B200_LIB=api.LIB_PATH, **{switch: "0"}), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    e = np.abs(np.load(tmp_path / "o.npy") - want).max(1) / max(1.0, np.abs(want).max())
    assert np.median(e) < 2e-2 and e.max() < 6e-2, (float(np.median(e)), float(e.max()))


def test_generation_through_the_entry_points(tmp_path):
    cfg = six_layers()
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


def test_serving_precision_generation_over_the_captured_step(tmp_path):
    """The captured bf16 step (tensor-core attention decode, side streams as graph branches) against one row at a time."""
    cfg = O.make_config([
        ("attention", O.attention_mixer(heads=4, kv_heads=2, dim=32, vdim=32), O.moe_mlp(ff=32, experts=6, top=2, shared=32)),
        ("latent_attention", O.latent_mixer(heads=2, dim=32, rot_dim=32, vdim=32, kv_rank=64, q_rank=32, window=20), None),
        ("retention", O.retention_mixer(heads=3, dim=32, vdim=40), O.moe_mlp(ff=32, experts=4, top=2, count=1, keep=1)),
    ], width=96, vocab=120)
    folder, W = checkpoint(tmp_path, cfg, seed=16)
    prompt, n = tokens_for(cfg, 40), 60
    m, s = open_model(folder, api.BF16, context=160)
    s.forward_batch(prompt[:-1], 0)
    toks = s.generate_greedy(prompt[-1], len(prompt) - 1, n)
    s.end_sequence()
    seq, got = prompt + toks, []
    s.forward_batch(prompt[:-1], 0)
    for t in range(len(prompt) - 1, len(seq) - 1):
        got.append(int(np.argmax(s.forward_rows(seq[t:t + 1], t, [0])[0])))
    close(m, s)
    assert got == toks


def test_command_line_on_a_checkpoint_directory(tmp_path):
    exe = os.path.join(ROOT, "build", "main")
    if not os.path.exists(exe):
        subprocess.check_call(["make", "-s", "-C", ROOT, "cli"])
    cfg = six_layers()
    folder, W = checkpoint(tmp_path, cfg, seed=15)
    prompt = tokens_for(cfg, 17)
    text = " ".join(map(str, prompt))
    r = subprocess.run([exe, folder, "-m", "completion", "-i", text, "-n", "6", "-t", "0", "-p", "fp32"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    ids = [l for l in r.stdout.splitlines() if re.fullmatch(r"(\d+ )+", l)]
    assert ids and [int(x) for x in ids[-1].split()] == O.greedy(cfg, W, prompt, 6)


def test_trace_runner(tmp_path):
    cfg = six_layers()
    folder, W = settled_checkpoint(tmp_path, cfg, seed=14)
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
