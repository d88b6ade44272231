"""Rorosun on the GPU against the plain implementation: each kernel alone, then whole models in portions,
token by token, and through the generation loop, the command line and the trace replay."""

import ctypes
import json
import math
import os
import subprocess
import sys

import pytest
import torch

from conftest import ROOT
from leankv_b200 import _native, registry
from leankv_b200.mixer_engine import MixerDecodeEngine, MixerModelConfig
from leankv_b200.sequence_state import pad16
from oracle import rorosun as plain
from rorosun_util import config, layer, rel, tokens, weights, write_model

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
F32, BF16 = torch.float32, torch.bfloat16
CODE = {BF16: _native.DT_BF16, F32: _native.DT_F32}


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


def rnd(*shape, seed=0, std=1.0, mean=0.0, dtype=F32):
    return (torch.randn(shape, generator=gen(seed)) * std + mean).to(dtype)


def stream():
    return torch.cuda.current_stream().cuda_stream


def ok(rc):
    _native.check(rc, "kernel", _native.mixers())
    torch.cuda.synchronize()


# ── dense GEMV ───────────────────────────────────────────────────────────────────────────────

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,cols", [(1, 8), (7, 20), (48, 48), (33, 250), (650, 264), (1030, 4104), (96, 14336), (5, 9000)])
def test_gemv_plain_bias_residual(dtype, rows, cols):
    w, x = rnd(rows, cols, seed=1, std=cols ** -0.5).to(dtype), rnd(cols, seed=2)
    b, s, r = rnd(rows, seed=3), rnd(rows, seed=4), rnd(rows, seed=5)
    d = [t.to(DEV) for t in (w, x, b, s, r)]
    y = torch.full((rows,), 7.0, device=DEV)
    acc = w.double() @ x.double()
    a = _native.DenseGemv(w=d[0].data_ptr(), x=d[1].data_ptr(), y=y.data_ptr(), dtype=CODE[dtype], rows=rows, cols=cols)
    ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))
    assert rel(y, acc) < 1e-5
    a.bias, a.bias_rows = d[2].data_ptr(), rows // 2
    ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))
    part = b.double().clone()
    part[rows // 2:] = 0
    assert rel(y, acc + part) < 1e-5
    a.bias, a.bias_rows, a.scale, a.residual, a.y = None, 0, d[3].data_ptr(), d[4].data_ptr(), d[4].data_ptr()
    ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))
    assert rel(d[4], r.double() + s.double() * acc) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,cols", [(3, 24), (41, 52), (300, 512), (200, 7176)])
def test_gemv_norm_and_gate(dtype, rows, cols):
    w, x, g = rnd(2 * rows, cols, seed=1, std=cols ** -0.5).to(dtype), rnd(cols, seed=2, std=3.0), torch.tensor(1.7)
    d = [t.to(DEV) for t in (w, x, g)]
    y = torch.empty(rows, device=DEV)
    a = _native.DenseGemv(w=d[0].data_ptr(), x=d[1].data_ptr(), y=y.data_ptr(), dtype=CODE[dtype], rows=rows, cols=cols,
                          gated=1, gain=d[2].data_ptr(), eps=0.01)
    ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))
    v = w.double() @ plain.scalar_norm(x.double(), g.double(), 0.01)
    gate = v[:rows]
    assert rel(y, gate * torch.sigmoid(gate) * v[rows:]) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("ends,cols", [([3, 10, 11, 40], 24), ([130, 131, 700, 1000], 260), ([2048, 4096, 4100, 6000], 1024)])
def test_gemv_token_shift_segments_and_previous_token(dtype, ends, cols):
    rows = ends[-1]
    w, xs = rnd(rows, cols, seed=1, std=cols ** -0.5).to(dtype), rnd(3, cols, seed=2)
    mu, g = rnd(len(ends), cols, seed=3, std=0.4, mean=0.5), torch.tensor(0.6)
    wd, mud, gd = w.to(DEV), mu.to(DEV), g.to(DEV)
    prev, state = torch.zeros(2, cols, device=DEV), torch.zeros(8, dtype=torch.int32, device=DEV)
    y, h_prev = torch.empty(rows, device=DEV), torch.zeros(cols).double()
    for t in range(3):
        x = xs[t].to(DEV)
        a = _native.DenseGemv(w=wd.data_ptr(), x=x.data_ptr(), y=y.data_ptr(), dtype=CODE[dtype], rows=rows, cols=cols,
                              gain=gd.data_ptr(), eps=1e-5, n_mix=len(ends), prev=prev.data_ptr(), state=state.data_ptr())
        for i, e in enumerate(ends):
            a.mix_end[i], a.mu[i] = e, None if i == 1 else mud[i].data_ptr()
        ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))
        state[_native.STATE_PARITY] ^= 1
        h = plain.scalar_norm(xs[t].double(), g.double(), 1e-5)
        lo, want = 0, []
        for i, e in enumerate(ends):
            v = h if i == 1 else h + (h_prev - h) * mu[i].double()
            want.append(w[lo:e].double() @ v)
            lo = e
        assert rel(y, torch.cat(want)) < 1e-5
        h_prev = h


# ── row kernels of a portion ─────────────────────────────────────────────────────────────────

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,W", [(1, 20), (2, 48), (9, 300), (5, 2056)])
def test_stream_norm_residual_shift(dtype, T, W):
    x, dlt, s, mu = rnd(T, W, seed=1), rnd(T, W, seed=2), rnd(W, seed=3), rnd(5, W, seed=4, std=0.4, mean=0.5)
    g, first = torch.tensor(1.4), rnd(W, seed=5)
    d = [t.to(DEV) for t in (x, dlt, s, mu, g, first)]
    xo, h = torch.empty(T, W, device=DEV), torch.empty(T, W, dtype=dtype, device=DEV)
    mixed, last = torch.empty(5, T, W, dtype=dtype, device=DEV), torch.empty(W, device=DEV)
    a = _native.StreamNorm(x_in=d[0].data_ptr(), x_out=xo.data_ptr(), delta=d[1].data_ptr(), scale=d[2].data_ptr(),
                           gain=d[4].data_ptr(), h=h.data_ptr(), mixed=mixed.data_ptr(), prev_in=d[5].data_ptr(),
                           prev_out=last.data_ptr(), dtype=CODE[dtype], delta_dtype=_native.DT_F32, rows=T, width=W,
                           n_mix=5, eps=1e-3)
    for i in range(5):
        a.mu[i] = d[3][i].data_ptr()
    ok(_native.mixers().leankv_stream_norm(ctypes.byref(a), stream()))
    want = x.double() + s.double() * dlt.double()
    hw = plain.scalar_norm(want, g.double(), 1e-3)
    above = torch.cat([first.double()[None], hw[:-1]])
    tol = 1e-5 if dtype == F32 else 4e-3
    assert rel(xo, want) < 1e-6 and rel(h.float(), hw) < tol and rel(last, hw[-1]) < 1e-6
    for i in range(5):
        assert rel(mixed[i].float(), hw + (above - hw) * mu[i].double()) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,n", [(3, 8), (2, 5), (17, 64)])
def test_silu_mul_and_tanh_split(dtype, T, n):
    gu = rnd(T, 2 * n, seed=1, std=2.0).to(dtype)
    x, out = gu.to(DEV), torch.empty(T, n, dtype=dtype, device=DEV)
    ok(_native.mixers().leankv_silu_mul(x.data_ptr(), out.data_ptr(), CODE[dtype], T, n, stream()))
    g, u = gu.double()[:, :n], gu.double()[:, n:]
    assert rel(out.float(), g * torch.sigmoid(g) * u) < (1e-6 if dtype == F32 else 4e-3)
    z = rnd(T, n, seed=2, std=1.5)
    zd, t = z.to(DEV), torch.empty(T, n if dtype == F32 else 2 * n, dtype=dtype, device=DEV)
    ok(_native.mixers().leankv_tanh_split(zd.data_ptr(), t.data_ptr(), CODE[dtype], T, n, stream()))
    t = t.double().cpu()
    assert rel(t if dtype == F32 else t[:, :n] + t[:, n:], torch.tanh(z.double())) < 2e-5


# ── window + pooled-block attention ──────────────────────────────────────────────────────────

class Window:
    """The attention kernels driven alone: portions of projections in, attention rows out."""

    def __init__(self, dtype, H, G, d, dv, size, pool, chunk, limit, scale=0.4, normed=True, talk=True, seed=0):
        self.H, self.G, self.d, self.dv, self.size, self.pool, self.scale, self.dtype = H, G, d, dv, size, pool, scale, dtype
        ring = max(size, pool) + chunk - 1
        z = lambda n, w: torch.full((n, G, pad16(w)), float("nan"), dtype=dtype, device=DEV)
        self.buf = [z(ring, d), z(ring, dv), z(limit // pool + 1, d), z(limit // pool + 1, dv)]
        self.qn, self.kn = rnd(H * d, seed=seed + 1, std=0.3, mean=1.4), rnd(G * d, seed=seed + 2, std=0.3, mean=1.2)
        self.talk = rnd(H, H, seed=seed + 3, std=0.7)
        self.dev = [t.to(DEV) for t in (self.qn, self.kn, self.talk)]
        self.normed, self.talks = normed, talk
        p = lambda t, on: t.data_ptr() if on else None
        self.c = _native.WindowPool(dtype=CODE[dtype], heads=H, kv_heads=G, dim=d, vdim=dv, dim_pad=pad16(d),
                                    vdim_pad=pad16(dv), size=size, pool=pool, ring=ring, max_blocks=limit // pool + 1,
                                    scale=scale, k_ring=self.buf[0].data_ptr(), v_ring=self.buf[1].data_ptr(),
                                    k_pool=self.buf[2].data_ptr(), v_pool=self.buf[3].data_ptr(),
                                    q_norm=p(self.dev[0], normed), k_norm=p(self.dev[1], normed), eps=1e-4,
                                    talk=p(self.dev[2], talk))
        self.limit = limit

    def rows(self, qkv, start):
        lib, T = _native.mixers(), qkv.shape[0]
        x, ref = qkv.to(DEV).float().contiguous(), ctypes.byref(self.c)
        q = torch.empty(T, self.H, pad16(self.d), dtype=self.dtype, device=DEV)
        out = torch.full((T, self.H * self.dv + 3), 9.0, dtype=self.dtype, device=DEV)
        ok(lib.leankv_window_pool_append(ref, x.data_ptr(), x.shape[1], None, q.data_ptr(), T, start, stream()))
        ws = torch.empty(max(16, lib.leankv_window_pool_workspace_bytes(ref, T, start + T)), dtype=torch.uint8, device=DEV)
        ok(lib.leankv_window_pool_attend(ref, q.data_ptr(), out.data_ptr(), out.stride(0), 0.5, T, start, ws.data_ptr(),
                                         ws.numel(), stream()))
        assert bool((out[:, self.H * self.dv:] == 9.0).all())       # columns of the neighbour are left alone
        return out[:, :self.H * self.dv].float().cpu()

    def step(self, y, pos):
        lib, ref = _native.mixers(), ctypes.byref(self.c)
        y = y.to(DEV).float().contiguous()
        out = torch.empty(self.H * self.dv, device=DEV)
        state = torch.zeros(8, dtype=torch.int32, device=DEV)
        state[0] = pos
        ws = torch.empty(max(16, lib.leankv_mixer_step_workspace_bytes(ref, self.limit)), dtype=torch.uint8, device=DEV)
        s = _native.MixerStep(y=y.data_ptr(), out=out.data_ptr(), left_scale=0.5, state=state.data_ptr(),
                              max_pos=self.limit, ws=ws.data_ptr(), ws_bytes=ws.numel())
        ok(lib.leankv_mixer_step(ref, None, ctypes.byref(s), stream()))
        return out.cpu()

    def expected(self, qkv):
        T, n = qkv.shape[0], self.H * self.d
        m = n + self.G * self.d
        x = qkv.double()
        q, k, v = x[:, :n], x[:, n:m], x[:, m:]
        if self.normed:
            q, k = plain.rms(q, 1e-4) * self.qn.double(), plain.rms(k, 1e-4) * self.kn.double()
        w = plain.window_pool_weights(q.reshape(T, self.H, -1), k.reshape(T, self.G, -1), self.scale, self.size, self.pool)
        if self.talks:
            w = plain.talk(w, self.talk.double())
        return 0.5 * plain.apply_values(w, v.reshape(T, self.G, -1), self.pool).reshape(T, -1)

    def qkv(self, T, seed=7, std=1.0):
        return rnd(T, self.H * self.d + self.G * (self.d + self.dv), seed=seed, std=std)


SHAPES = [(4, 2, 16, 24, 10, 3), (6, 3, 10, 6, 5, 8), (8, 8, 64, 64, 33, 4), (12, 2, 32, 48, 1, 1), (16, 2, 128, 128, 40, 16),
          (3, 1, 80, 16, 64, 64), (32, 8, 128, 128, 70, 6), (9, 3, 48, 96, 100, 7)]


def feed(win, qkv, cuts):
    out, at = [], 0
    for n in cuts:
        n = min(n, qkv.shape[0] - at)
        if n == 0:
            break
        out.append(win.rows(qkv[at:at + n], at) if n > 1 else win.step(qkv[at], at)[None])
        at += n
    assert at == qkv.shape[0]
    return torch.cat(out)


def tol(dtype):
    return 2e-5 if dtype == F32 else 3e-2


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES)
def test_window_pool_prompt_portions_and_steps_agree_with_plain(dtype, shape):
    T = 150
    win = Window(dtype, *shape, chunk=T, limit=T)
    qkv = win.qkv(T)
    want = win.expected(qkv)
    assert rel(feed(win, qkv, [T]), want) < tol(dtype)
    small = Window(dtype, *shape, chunk=16, limit=T)       # the ring wraps many times
    assert rel(feed(small, qkv, [2, 3, 16, 5, 1, 1, 16, 11, 1, 2, 13, 7, 16, 16, 16, 16, 16, 16]), want) < tol(dtype)
    steps = Window(dtype, *shape, chunk=1, limit=T)
    assert rel(feed(steps, qkv, [1] * T), want) < tol(dtype)


@pytest.mark.parametrize("normed,talk", [(False, True), (True, False), (False, False)])
def test_window_pool_without_norm_or_mixing(normed, talk):
    win = Window(F32, 4, 2, 16, 24, 10, 3, chunk=60, limit=60, normed=normed, talk=talk)
    qkv = win.qkv(60)
    want = win.expected(qkv)
    assert rel(feed(win, qkv, [40, 20]), want) < 2e-5
    win = Window(F32, 4, 2, 16, 24, 10, 3, chunk=8, limit=60, normed=normed, talk=talk)
    assert rel(feed(win, qkv, [8] + [1] * 52), want) < 2e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("size,pool", [(96, 8), (128, 16), (100, 12), (64, 128)])
@pytest.mark.parametrize("far", ["inside", "outside", "block_in", "block_out", "first"])
def test_one_key_stands_out_at_every_edge(dtype, size, pool, far):
    """One key far larger than the others, at the window's edge or in the newest / next pooled block: seeing it
    or not decides the row."""
    T, H, G, d, dv = 402, 4, 2, 32, 32
    i = T - 2 if far in ("inside", "outside") else T - 2 - ((T - 2 - size + 1) % pool)     # a block just became visible
    key = {"inside": i - size + 1, "outside": i - size, "block_in": i - size - pool // 2,
           "block_out": i - size + 1, "first": 0}[far]
    win = Window(dtype, H, G, d, dv, size, pool, chunk=T, limit=T, normed=False, scale=1.0)
    qkv = win.qkv(T, std=0.3)
    u = torch.randn(d, generator=gen(11))
    u = u / u.norm()
    for h in range(H):
        qkv[:, h * d:(h + 1) * d] = qkv[:, h * d:(h + 1) * d] * 0.1 + 4.0 * u
    gain = 2.5 if far in ("inside", "outside") else 2.5 * pool if far != "first" else 4.0 * pool
    for g in range(G):
        qkv[key, (H + g) * d:(H + g + 1) * d] = gain * u
        qkv[key, (H + G) * d + g * dv:(H + G) * d + (g + 1) * dv] += 5.0
    want = win.expected(qkv)
    near = want[max(0, i - 3):i + 4]
    whole = feed(win, qkv, [T])
    assert rel(whole[max(0, i - 3):i + 4], near) < tol(dtype)
    step = Window(dtype, H, G, d, dv, size, pool, chunk=T, limit=T, normed=False, scale=1.0)
    got = feed(step, qkv, [i - 3] + [1] * (T - i + 3))
    assert rel(got[i - 3:i + 4], near) < tol(dtype)
    # the two sides of the edge differ by far more than the tolerance
    if far in ("inside", "outside"):
        assert rel(want[key + size - 1][None], want[key + size][None]) > 0.3


def test_very_long_context_keeps_weights_outside_shared_memory():
    T, H, G, d = 40000, 32, 2, 16
    win = Window(F32, H, G, d, d, size=6, pool=2, chunk=4096, limit=T)
    assert _native.mixers().leankv_mixer_step_workspace_bytes(ctypes.byref(win.c), T) > 0
    for b, seed in zip(win.buf, range(4)):
        b.copy_(rnd(*b.shape, seed=seed, std=0.3).to(DEV))
    qkv = win.qkv(2, seed=3)
    i = T - 2
    rows = win.rows(qkv, i)
    again = torch.stack([win.step(qkv[0], i), win.step(qkv[1], i + 1)])
    assert rel(rows, again) < 2e-5
    # plain attention over what the buffers hold
    n, m = H * d, (H + G) * d
    q = (plain.rms(qkv[:, :n].double(), 1e-4) * win.qn.double()).reshape(2, H, d)
    for t in range(2):
        pos, nb = i + t, (i + t - 6 + 1) // 2
        slots = [p % win.c.ring for p in range(pos - 5, pos + 1)]
        keys = torch.cat([win.buf[2][:nb], win.buf[0][slots]]).double().cpu().repeat_interleave(H // G, 1)
        vals = torch.cat([win.buf[3][:nb], win.buf[1][slots]]).double().cpu().repeat_interleave(H // G, 1)
        w = torch.softmax(torch.einsum("hd,jhd->hj", q[t], keys) * win.scale, -1)
        want = 0.5 * torch.einsum("hj,jhd->hd", win.talk.double() @ w, vals)
        assert rel(rows[t][None], want.reshape(1, -1)) < 5e-5


# ── time mixing ──────────────────────────────────────────────────────────────────────────────

class Mix:
    def __init__(self, dtype, H, d, seed=0, fast=False):
        self.dtype, self.H, self.d = dtype, H, d
        self.S = torch.zeros(H, d, d, device=DEV)
        self.u, self.norm = rnd(H * d, seed=seed + 1, std=0.8), rnd(H * d, seed=seed + 2, std=0.3, mean=1.0)
        self.w0 = rnd(H * d, seed=seed + 3, std=1.5, mean=1.0 if fast else -3.0)
        self.dev = [t.to(DEV) for t in (self.u, self.w0, self.norm)]
        self.c = _native.TimeMix(dtype=CODE[dtype], heads=H, dim=d, S=self.S.data_ptr(), u=self.dev[0].data_ptr(),
                                 w0=self.dev[1].data_ptr(), norm=self.dev[2].data_ptr(), eps=1e-4)

    def inputs(self, T, seed=5):
        N = self.H * self.d
        return rnd(4, T, N, seed=seed).to(self.dtype), rnd(T, N, seed=seed + 1)

    def rows(self, rkvg, z):
        T, N = z.shape
        x, zd = rkvg.contiguous().to(DEV), z.contiguous().to(DEV)
        out = torch.full((T, N + 5), 9.0, dtype=self.dtype, device=DEV)
        lib = _native.mixers()
        ws = torch.empty(lib.leankv_time_mix_workspace_bytes(ctypes.byref(self.c), T), dtype=torch.uint8, device=DEV)
        ok(lib.leankv_time_mix_rows(ctypes.byref(self.c), *(x[i].data_ptr() for i in range(4)), zd.data_ptr(),
                                    out.data_ptr(), N + 5, 0.7, T, ws.data_ptr(), ws.numel(), stream()))
        assert bool((out[:, N:] == 9.0).all())
        return out[:, :N].float().cpu()

    def expected(self, rkvg, z):
        T, N = z.shape
        r, k, v = (rkvg[i].double().reshape(T, self.H, self.d) for i in range(3))
        g = rkvg[3].double()
        w = torch.exp(-torch.exp(z.double() + self.w0.double())).reshape(T, self.H, self.d)
        o, S = plain.wkv(r, k, v, w, self.u.double().reshape(self.H, self.d))
        return 0.7 * plain.rms(o, 1e-4).reshape(T, N) * self.norm.double() * g * torch.sigmoid(g), S


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,d", [(1, 4), (3, 20), (2, 48), (4, 64), (2, 80), (1, 128), (2, 200), (1, 256)])
@pytest.mark.parametrize("fast", [False, True])
def test_time_mix_rows(dtype, H, d, fast):
    T = 230                                    # long enough to be cut into pieces that run in parallel
    m = Mix(dtype, H, d, fast=fast)
    x, z = m.inputs(T)
    want, S = m.expected(x, z)
    bound = 5e-5 if dtype == F32 else 6e-3
    assert rel(m.rows(x, z), want) < bound
    assert rel(m.S.reshape(1, -1), S.reshape(1, -1)) < 1e-5
    m = Mix(dtype, H, d, fast=fast)
    got, at = [], 0
    for n in (1, 2, 3, 198, 17, 5, 4):
        got.append(m.rows(x[:, at:at + n], z[at:at + n]))
        at += n
    assert at == T and rel(torch.cat(got), want) < bound
    assert rel(m.S.reshape(1, -1), S.reshape(1, -1)) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,d,rank", [(1, 4, 3), (3, 20, 5), (9, 64, 16), (2, 80, 70), (2, 200, 33)])
def test_time_mix_steps(dtype, H, d, rank):
    T, N = 12, H * d
    m = Mix(dtype, H, d)
    y = rnd(T, 4 * N + rank, seed=8)
    w2 = rnd(N, rank, seed=9, std=rank ** -0.5).to(dtype)
    z = torch.tanh(y[:, 4 * N:].double()) @ w2.double().T
    x = y[:, :4 * N].reshape(T, 4, N).transpose(0, 1)
    want, S = m.expected(x, z)
    w2d, out, state = w2.to(DEV), torch.empty(N, device=DEV), torch.zeros(8, dtype=torch.int32, device=DEV)
    got = []
    for t in range(T):
        yd = y[t].to(DEV)
        s = _native.MixerStep(y=yd.data_ptr(), rkvg_off=0, w1_off=4 * N, rank=rank, w2=w2d.data_ptr(), out=out.data_ptr(),
                              right_off=0, right_scale=0.7, state=state.data_ptr(), max_pos=T)
        ok(_native.mixers().leankv_mixer_step(None, ctypes.byref(m.c), ctypes.byref(s), stream()))
        got.append(out.cpu().clone())
    assert rel(torch.stack(got), want) < 5e-5
    assert rel(m.S.reshape(1, -1), S.reshape(1, -1)) < 1e-5


# ── whole models ─────────────────────────────────────────────────────────────────────────────

WIDE = config([layer(heads=8, kv_heads=2, dim=64, vdim=64, size=48, pool=8, r_heads=4, r_dim=64, ff=320, scale=0.125),
               layer(heads=5, kv_heads=5, dim=48, vdim=80, size=33, pool=5, r_heads=2, r_dim=96, ff=None),
               layer(heads=16, kv_heads=4, dim=32, vdim=16, size=20, pool=40, r_heads=8, r_dim=16, ff=512)],
              vocab=203, width=136)
ODD = config([layer(heads=1, kv_heads=1, dim=1, vdim=1, size=1, pool=1, r_heads=1, r_dim=1, ff=1),
              layer(heads=3, kv_heads=1, dim=7, vdim=13, size=6, pool=2, r_heads=5, r_dim=9, ff=11)], vocab=19, width=21,
             eps=1e-2)
MODELS = {"small": config(), "wide": WIDE, "odd": ODD}
MODEL_TOL = {F32: 2e-4, BF16: 0.12}


def engine(name, dtype, limit=256, chunk=256, seed=0, rank=5):
    cfg = MODELS[name]
    w = weights(cfg, seed, rank)
    return cfg, w, MixerDecodeEngine(MixerModelConfig.from_dict(cfg), w, DEV, max_seq_len=limit, dtype=dtype,
                                     max_chunk=chunk)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_portions_and_single_tokens(name, dtype):
    cfg, w, eng = engine(name, dtype)
    ids = tokens(cfg, 140)
    want = plain.forward(cfg, w, ids)
    everything = list(range(140))
    assert rel(eng.extend(ids, everything), want) < MODEL_TOL[dtype]
    for cuts in ([2] * 70, [7, 1, 1, 31, 2, 64, 3, 31], [139, 1], [1] * 140):
        eng.reset()
        got, at = [], 0
        for n in cuts:
            got.append(eng.extend(ids[at:at + n], list(range(n))))
            at += n
        assert at == 140 and rel(torch.cat(got), want) < MODEL_TOL[dtype], cuts[:3]


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_first_tokens_and_short_sequences(dtype):
    cfg, w, eng = engine("small", dtype)
    for n in (1, 2, 3, 4, 5):
        ids = tokens(cfg, n, seed=n)
        want = plain.forward(cfg, w, ids)
        eng.reset()
        assert rel(eng.extend(ids, list(range(n))), want) < MODEL_TOL[dtype]
        eng.reset()
        assert rel(torch.cat([eng.extend([t], [0]) for t in ids]), want) < MODEL_TOL[dtype]


def test_small_portions_wrap_every_ring_and_wanted_rows_keep_their_order():
    cfg, w, eng = engine("small", F32, chunk=6)
    ids = tokens(cfg, 200)
    want = plain.forward(cfg, w, ids)
    places = [150, 3, 199, 0, 77, 78]
    assert rel(eng.extend(ids, places), want[places]) < MODEL_TOL[F32]


def test_a_sequence_leaves_nothing_behind():
    cfg, w, eng = engine("wide", F32)
    a, b = tokens(cfg, 120, seed=1), tokens(cfg, 90, seed=2)
    first = eng.extend(b[:40], [39])
    rest = [eng.extend([t], [0]) for t in b[40:50]]
    eng.reset()
    eng.extend(a, [])
    for t in a[:7]:
        eng.extend([t], [])
    eng.reset()
    assert torch.equal(eng.extend(b[:40], [39]), first)
    for t, r in zip(b[40:50], rest):
        assert torch.equal(eng.extend([t], [0]), r)


def test_long_decoding_past_windows_and_blocks():
    cfg, w, eng = engine("small", F32, limit=420)
    ids = tokens(cfg, 400, seed=4)
    want = plain.forward(cfg, w, ids)
    eng.extend(ids[:5], [])
    got = torch.cat([eng.extend([t], [0]) for t in ids[5:]])
    assert rel(got, want[5:]) < MODEL_TOL[F32]


def test_far_token_shows_through_a_pooled_block():
    """Changing a token that lies far outside the window changes the logits, through pooled blocks and the
    recurrence alone, exactly as the plain implementation says."""
    cfg, w, eng = engine("wide", F32)
    ids = tokens(cfg, 150, seed=6)
    other = list(ids)
    other[3] = (other[3] + 1) % cfg["vocab"]
    a, b = plain.forward(cfg, w, ids)[-1:], plain.forward(cfg, w, other)[-1:]
    ga = eng.extend(ids, [149])
    eng.reset()
    gb = eng.extend(other, [149])
    assert float((a - b).norm() / a.norm()) > 1e-4
    assert rel((ga - gb).double().cpu(), a - b) < 0.05


@pytest.mark.parametrize("eps,left,right", [(1e-2, 1.0, 1.0), (1e-6, 0.0, 1.3), (1e-5, -2.0, 0.0)])
def test_constants_come_from_the_configuration(eps, left, right):
    cfg = config([layer(left_scale=left, right_scale=right, scale=1.0, size=4, pool=1), layer(pool=20, ff=None)], eps=eps)
    w, ids = weights(cfg, 3), tokens(cfg, 60)
    eng = MixerDecodeEngine(MixerModelConfig.from_dict(cfg), w, DEV, max_seq_len=64, dtype=F32)
    assert rel(eng.extend(ids[:40], list(range(40))), plain.forward(cfg, w, ids)[:40]) < MODEL_TOL[F32]
    got = torch.cat([eng.extend([t], [0]) for t in ids[40:]])
    assert rel(got, plain.forward(cfg, w, ids)[40:]) < MODEL_TOL[F32]


def test_window_and_block_longer_than_the_sequence():
    cfg = config([layer(size=1000, pool=3), layer(size=5, pool=700), layer(size=4000, pool=2000, ff=None)])
    w, ids = weights(cfg, 5), tokens(cfg, 64)
    eng = MixerDecodeEngine(MixerModelConfig.from_dict(cfg), w, DEV, max_seq_len=64, dtype=F32)
    want = plain.forward(cfg, w, ids)
    assert rel(eng.extend(ids[:50], list(range(50))), want[:50]) < MODEL_TOL[F32]
    assert rel(torch.cat([eng.extend([t], [0]) for t in ids[50:]]), want[50:]) < MODEL_TOL[F32]


def test_engine_refuses_what_does_not_fit():
    cfg, w, eng = engine("small", F32, limit=10)
    with pytest.raises(ValueError):
        eng.extend(tokens(cfg, 11), [])
    with pytest.raises(ValueError):
        eng.extend([cfg["vocab"]], [])
    with pytest.raises(ValueError):
        eng.extend([1, 2], [2])
    eng.extend(tokens(cfg, 10), [])
    with pytest.raises(RuntimeError, match="full"):
        eng.step()


def greedy(cfg, w, prompt, n):
    """Greedy continuation by the plain implementation, and the smallest margin between the best two logits."""
    ids, margin = list(prompt), math.inf
    for _ in range(n):
        top = plain.forward(cfg, w, ids)[-1].topk(2)
        margin = min(margin, float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margin


@pytest.mark.parametrize("host", [True, False])
def test_greedy_generation(host):
    cfg, w, eng = engine("small", F32)
    for seed, n in ((3, 37), (5, 1), (6, 12)):
        prompt = tokens(cfg, n, seed=seed)
        want, margin = greedy(cfg, w, prompt, 24)
        assert margin > 1e-4
        assert eng.generate(prompt, 24, stream_to_host=host) == want
    assert eng.prefill(prompt, chunk=3) == want[0]


def test_command_line_and_trace_replay(tmp_path):
    cfg, w = MODELS["small"], weights(MODELS["small"])
    folder = write_model(tmp_path / "model", cfg, w)
    prompt = tokens(cfg, 20)
    want, _ = greedy(cfg, w, prompt, 8)
    out = subprocess.run([sys.executable, "-m", "leankv_b200", "generate", "--model", folder, "--dtype", "float32",
                          "--prompt", ",".join(map(str, prompt)), "--max-new-tokens", "8"], cwd=ROOT,
                         capture_output=True, text=True)
    assert out.returncode == 0, out.stderr
    assert json.loads(out.stdout.splitlines()[-1])["tokens"] == want
    a, b = tokens(cfg, 30, seed=8), tokens(cfg, 5, seed=9)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:28], "want": [27, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[28:29], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[29:], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [0, 1, 2, 3, 4]}], "end": ["b"]}]
    res = tmp_path / "out"
    res.mkdir()
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(res),
                          "--max-tokens", "32"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                         text=True)
    assert run.returncode == 0, run.stderr
    assert [l for l in run.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda i: torch.frombuffer(bytearray((res / f"{i}.f32").read_bytes()), dtype=F32).reshape(-1, cfg["vocab"])
    la, lb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert rel(read(0), la[[27, 4]]) < MODEL_TOL[F32] and rel(read(2), la[29:]) < MODEL_TOL[F32]
    assert rel(read(3), lb) < MODEL_TOL[F32] and not (res / "1.f32").exists()


def test_llama_checkpoints_load_through_the_registry(tmp_path):
    from leankv_b200.engine import PROJ_NAMES, DecodeEngine, DecoderConfig

    cfg = DecoderConfig(vocab_size=256, hidden_size=512, intermediate_size=512, num_layers=2, num_q_heads=4, num_kv_heads=1)
    g, t = gen(1), {}
    draw = lambda n, *s: t.__setitem__(n, (torch.randn(s, generator=g) * 0.02).half())
    draw("model.embed_tokens.weight", 256, 512)
    draw("lm_head.weight", 256, 512)
    t["model.norm.weight"] = torch.ones(512).half()
    shape = {"q_proj": (512, 512), "k_proj": (128, 512), "v_proj": (128, 512), "o_proj": (512, 512),
             "gate_proj": (512, 512), "up_proj": (512, 512), "down_proj": (512, 512)}
    for i in range(2):
        p = f"model.layers.{i}."
        t[p + "input_layernorm.weight"] = t[p + "post_attention_layernorm.weight"] = torch.ones(512).half()
        for n in PROJ_NAMES:
            draw(f"{p}{'self_attn' if n in ('q_proj', 'k_proj', 'v_proj', 'o_proj') else 'mlp'}.{n}.weight", *shape[n])
    c = {"architectures": ["LlamaForCausalLM"], "vocab_size": 256, "hidden_size": 512, "intermediate_size": 512,
         "num_hidden_layers": 2, "num_attention_heads": 4, "num_key_value_heads": 1, "head_dim": 128, "rope_theta": 1e6,
         "rms_norm_eps": 1e-5}
    eng = registry.load_engine(write_model(tmp_path / "m", c, t), max_seq_len=64)
    full = {"embed": t["model.embed_tokens.weight"], "final_norm": t["model.norm.weight"], "lm_head": t["lm_head.weight"],
            "layers": [{"ln1": t[f"model.layers.{i}.input_layernorm.weight"],
                        "ln2": t[f"model.layers.{i}.post_attention_layernorm.weight"],
                        **{n: t[f"model.layers.{i}.{'self_attn' if n in PROJ_NAMES[:4] else 'mlp'}.{n}.weight"]
                           for n in PROJ_NAMES}} for i in range(2)]}
    move = lambda v: v.to(DEV) if torch.is_tensor(v) else [{k: x.to(DEV) for k, x in l.items()} for l in v]
    ref = DecodeEngine(cfg, DecodeEngine.shard_weights({k: move(v) for k, v in full.items()}, cfg, 0, 1), DEV, max_seq_len=64)
    prompt = list(range(3, 20))
    assert eng.generate(prompt, 6) == ref.generate(prompt, 6)
