"""Pefitar on the GPU against the plain implementation: each mechanism alone, then whole models in portions,
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
from leankv_b200 import _native
from leankv_b200.mixer_engine import MixerDecodeEngine, MixerModelConfig
from leankv_b200.mixers import Rotation
from leankv_b200.sequence_state import pad16
from oracle import pefitar as plain
from pefitar_util import attention, config, latent, weights
from rorosun_util import config as parallel_config
from rorosun_util import rel, tokens, write_model
from rorosun_util import weights as parallel_weights

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda", 0)
F32, BF16 = torch.float32, torch.bfloat16
CODE = {BF16: _native.DT_BF16, F32: _native.DT_F32}


def rnd(*shape, seed=0, std=1.0, mean=0.0, dtype=F32):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * std + mean).to(dtype)


def stream():
    return torch.cuda.current_stream().cuda_stream


def ok(rc):
    _native.check(rc, "kernel", _native.mixers())
    torch.cuda.synchronize()


def gemv(**kw):
    a = _native.DenseGemv(**{k: v.data_ptr() if torch.is_tensor(v) else v for k, v in kw.items()})
    ok(_native.mixers().leankv_dense_gemv(ctypes.byref(a), stream()))


# ── steps fused into the projections ─────────────────────────────────────────────────────────

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,cols", [(3, 24), (41, 53), (300, 512), (1030, 4104), (64, 9000)])
@pytest.mark.parametrize("joined", [False, True])
def test_gemv_gain_per_column_and_joined_branch(dtype, rows, cols, joined):
    w = rnd(rows, cols, seed=1, std=cols ** -0.5).to(dtype)
    x, g, d, pg = (rnd(cols, seed=s, std=0.7, mean=0.5) for s in (2, 3, 4, 5))
    dev = [t.to(DEV) for t in (w, x, g, d, pg)]
    y, out = torch.empty(rows, device=DEV), torch.full((cols,), 7.0, device=DEV)
    more = dict(delta=dev[3], post_gain=dev[4], post_mult=0.6, x_out=out) if joined else {}
    gemv(w=dev[0], x=dev[1], y=y, dtype=CODE[dtype], rows=rows, cols=cols, gain=dev[2], gain_per_col=1, eps=1e-2, **more)
    stream_ = x.double() + 0.6 * plain.rms_norm(d.double(), pg.double(), 1e-2) if joined else x.double()
    assert rel(y, w.double() @ plain.rms_norm(stream_, g.double(), 1e-2)) < 1e-5
    if joined:
        assert rel(out, stream_) < 1e-6 and torch.equal(dev[1].cpu(), x)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_gemv_gated_after_joined_branch(dtype):
    rows, cols = 77, 260
    w = rnd(2 * rows, cols, seed=1, std=cols ** -0.5).to(dtype)
    x, g, d, pg = (rnd(cols, seed=s, mean=0.5) for s in (2, 3, 4, 5))
    dev = [t.to(DEV) for t in (w, x, g, d, pg)]
    y, out = torch.empty(rows, device=DEV), torch.empty(cols, device=DEV)
    gemv(w=dev[0], x=dev[1], y=y, dtype=CODE[dtype], rows=rows, cols=cols, gated=1, gain=dev[2], gain_per_col=1, eps=1e-5,
         delta=dev[3], post_gain=dev[4], post_mult=-1.5, x_out=out)
    h = plain.rms_norm(x.double() - 1.5 * plain.rms_norm(d.double(), pg.double(), 1e-5), g.double(), 1e-5)
    v = w.double() @ h
    assert rel(y, v[:rows] * torch.sigmoid(v[:rows]) * v[rows:]) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("groups,n,cols,stride", [(1, 5, 8, 8), (3, 28, 10, 16), (7, 33, 20, 27), (16, 512, 128, 192),
                                                  (32, 128, 512, 512), (5, 1, 300, 304)])
def test_gemv_row_groups_with_an_input_each(dtype, groups, n, cols, stride):
    w = rnd(groups * n, cols, seed=1, std=cols ** -0.5).to(dtype)
    x = rnd(groups * stride, seed=2)
    wd, xd, y = w.to(DEV), x.to(DEV), torch.empty(groups * n, device=DEV)
    gemv(w=wd, x=xd, y=y, dtype=CODE[dtype], rows=groups * n, cols=cols, group_rows=n, group_stride=stride)
    want = torch.cat([w[i * n:(i + 1) * n].double() @ x[i * stride:i * stride + cols].double() for i in range(groups)])
    assert rel(y, want) < 1e-5


def test_softcap_in_the_head_and_on_rows():
    w, x = rnd(50, 24, seed=1, std=3.0), rnd(24, seed=2)
    wd, xd, y = w.to(DEV), x.to(DEV), torch.empty(50, device=DEV)
    gemv(w=wd, x=xd, y=y, dtype=CODE[F32], rows=50, cols=24, softcap=4.0)
    want = plain.softcap(w.double() @ x.double(), 4.0)
    assert rel(y, want) < 1e-5
    z = (w.double() @ x.double()).float().to(DEV)
    ok(_native.mixers().leankv_softcap(z.data_ptr(), 50, 4.0, stream()))
    assert rel(z, want) < 1e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,W", [(1, 20), (2, 47), (9, 300), (5, 2056), (3, 9000)])
def test_normed_branch_joins_the_rows(dtype, T, W):
    x, d, g, pg = rnd(T, W, seed=1), rnd(T, W, seed=2, std=3.0), rnd(W, seed=3, mean=1.0), rnd(W, seed=4, mean=1.0)
    xd, dd, gd, pgd = (t.to(DEV) for t in (x, d, g, pg))
    xo, h = torch.empty(T, W, device=DEV), torch.empty(T, W, dtype=dtype, device=DEV)
    a = _native.StreamNorm(x_in=xd.data_ptr(), x_out=xo.data_ptr(), delta=dd.data_ptr(), gain=gd.data_ptr(), gain_per_col=1,
                           h=h.data_ptr(), dtype=CODE[dtype], delta_dtype=_native.DT_F32, rows=T, width=W, eps=1e-3,
                           post_gain=pgd.data_ptr(), post_mult=0.4)
    ok(_native.mixers().leankv_stream_norm(ctypes.byref(a), stream()))
    want = x.double() + 0.4 * plain.rms_norm(d.double(), pg.double(), 1e-3)
    assert rel(xo, want) < 1e-6
    assert rel(h.float(), plain.rms_norm(want, g.double(), 1e-3)) < (1e-5 if dtype == F32 else 4e-3)
    xo.fill_(0.0)
    a.gain, a.gain_per_col, a.h = None, 0, None             # the last branch only joins
    ok(_native.mixers().leankv_stream_norm(ctypes.byref(a), stream()))
    assert rel(xo, want) < 1e-6


# ── rotation, norm and placement of rows ─────────────────────────────────────────────────────

@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,n,rot,base", [(3, 16, 16, 100.0), (1, 7, 4, 10000.0), (5, 64, 2, 3.0), (2, 9, 0, 1.0)])
def test_place_rows_rotates_at_the_position_and_wraps(dtype, heads, n, rot, base):
    T, start, ring, pad = 11, 1234, 16, pad16(n)
    x = rnd(T, heads * n + 3, seed=1)
    rate = Rotation(base, rot).rate(DEV)
    xd = x.to(DEV)
    dst = torch.full((ring, heads, pad), 5.0, dtype=dtype, device=DEV)
    a = _native.PlaceRows(dtype=CODE[dtype], rows=T, start=start, n_seg=1, rate=rate.data_ptr(), eps=1e-5)
    a.seg[0] = _native.RowSegment(src=xd.data_ptr() + 12, ld=x.shape[1], heads=heads, head_stride=n, n=n, dst=dst.data_ptr(),
                                  dst_ld=heads * pad, dst_head_stride=pad, n_pad=pad, ring=ring, rot=rot)
    ok(_native.mixers().leankv_place_rows(ctypes.byref(a), stream()))
    seq = torch.zeros(start + T, heads, n, dtype=torch.float64)
    seq[start:] = x[:, 3:].double().reshape(T, heads, n)
    want = plain.rotate(seq, base, rot)[start:]
    got = dst.float().cpu()
    for t in range(T):
        row = got[(start + t) % ring]
        assert rel(row[:, :n], want[t]) < (2e-4 if dtype == F32 else 6e-3)
        assert bool((row[:, n:] == 0).all())
    left = [s for s in range(ring) if s not in {(start + t) % ring for t in range(T)}]
    assert bool((got[left] == 5.0).all())


@pytest.mark.parametrize("n", [20, 33, 512])
def test_place_rows_norms_a_latent(n):
    T = 6
    x, g = rnd(T, n + 5, seed=1, std=2.0), rnd(n, seed=2, mean=1.0)
    xd, gd = x.to(DEV), g.to(DEV)
    dst = torch.empty(T, pad16(n), device=DEV)
    a = _native.PlaceRows(dtype=CODE[F32], rows=T, start=9, n_seg=1, eps=1e-2)
    a.seg[0] = _native.RowSegment(src=xd.data_ptr(), ld=n + 5, heads=1, n=n, dst=dst.data_ptr(), dst_ld=pad16(n), n_pad=pad16(n),
                                  gain=gd.data_ptr())
    ok(_native.mixers().leankv_place_rows(ctypes.byref(a), stream()))
    assert rel(dst[:, :n], plain.rms_norm(x[:, :n].double(), g.double(), 1e-2)) < 1e-5


# ── causal attention ─────────────────────────────────────────────────────────────────────────

class Causal:
    """The attention kernels driven alone. Keys: ``dim`` numbers per kv head, then ``shared`` common ones; dv 0: the
    values are the keys' own part."""

    def __init__(self, dtype, H, G, dim, shared, dv, size, chunk, limit, scale=0.3, rot=0, base=200.0, gated=True):
        self.dtype, self.H, self.G, self.dim, self.shared, self.dv, self.size = dtype, H, G, dim, shared, dv, size
        self.scale, self.rot, self.base, self.limit, self.gated = scale, rot, base, limit, gated
        ring = (min(size + chunk - 1, limit) + 127) // 128 * 128
        # stale numbers of another sequence must not show
        mk = lambda *s: torch.full(s, 3.0, dtype=dtype, device=DEV)
        self.buf = [mk(ring, G, pad16(dim)), mk(ring, G, pad16(dv)) if dv else None, mk(ring, pad16(shared)) if shared else None]
        self.out_dim = dv or dim
        p = lambda t: None if t is None else t.data_ptr()
        self.c = _native.CausalAttn(dtype=CODE[dtype], heads=H, kv_heads=G, dim=dim, shared_dim=shared, vdim=self.out_dim,
                                    dim_pad=pad16(dim), shared_pad=pad16(shared), vdim_pad=pad16(self.out_dim), size=size,
                                    scale=scale, k=p(self.buf[0]), v=p(self.buf[1]), k_ring=ring, k_rows=ring,
                                    shared=p(self.buf[2]), s_ring=ring if shared else 0)
        self.rate = Rotation(base, rot).rate(DEV)
        self.status = torch.zeros(1, dtype=torch.int32, device=DEV)
        need = _native.mixers().leankv_causal_step_workspace_bytes(ctypes.byref(self.c), limit)
        assert need > 0
        self.ws = torch.zeros(need, dtype=torch.uint8, device=DEV)

    def inputs(self, T, seed=7, std=1.0):
        """q [T, H, dim + shared], k [T, G, dim], shared [T, shared], v [T, G, dv], gate [T, H * out_dim]"""
        return [rnd(T, self.H, self.dim + self.shared, seed=seed, std=std), rnd(T, self.G, self.dim, seed=seed + 1, std=std),
                rnd(T, self.shared, seed=seed + 2, std=std), rnd(T, self.G, self.dv, seed=seed + 3),
                rnd(T, self.H * self.out_dim, seed=seed + 4)]

    def rows(self, x, start):
        lib = _native.mixers()
        q, k, sh, v, g = (t.to(DEV).contiguous() for t in x)
        T, d, s, H, G = q.shape[0], self.dim, self.shared, self.H, self.G
        dp, sp, vp = pad16(d), pad16(s), pad16(self.dv)
        qb = torch.empty(T, H, dp + sp, dtype=self.dtype, device=DEV)
        a = _native.PlaceRows(dtype=CODE[self.dtype], rows=T, start=start, rate=self.rate.data_ptr(), eps=1e-5)
        es = qb.element_size()
        own, com = (0, self.rot) if s else (self.rot, 0)
        segs = [dict(src=q.data_ptr(), ld=H * (d + s), heads=H, head_stride=d + s, n=d, dst=qb.data_ptr(), dst_ld=H * (dp + sp),
                     dst_head_stride=dp + sp, n_pad=dp, rot=own),
                dict(src=k.data_ptr(), ld=G * d, heads=G, head_stride=d, n=d, dst=self.c.k, dst_ld=G * dp, dst_head_stride=dp,
                     n_pad=dp, ring=self.c.k_ring, rot=own)]
        if s:
            segs += [dict(src=q.data_ptr() + 4 * d, ld=H * (d + s), heads=H, head_stride=d + s, n=s, dst=qb.data_ptr() + es * dp,
                          dst_ld=H * (dp + sp), dst_head_stride=dp + sp, n_pad=sp, rot=com),
                     dict(src=sh.data_ptr(), ld=s, heads=1, n=s, dst=self.c.shared, dst_ld=sp, n_pad=sp, ring=self.c.s_ring,
                          rot=com)]
        if self.dv:
            segs.append(dict(src=v.data_ptr(), ld=G * self.dv, heads=G, head_stride=self.dv, n=self.dv, dst=self.c.v,
                             dst_ld=G * vp, dst_head_stride=vp, n_pad=vp, ring=self.c.k_ring))
        for i in range(0, len(segs), _native.MAX_ROW_SEGMENTS):
            part = segs[i:i + _native.MAX_ROW_SEGMENTS]
            a.n_seg = len(part)
            for j, e in enumerate(part):
                a.seg[j] = _native.RowSegment(**e)
            ok(lib.leankv_place_rows(ctypes.byref(a), stream()))
        n = H * self.out_dim
        out = torch.full((T, n + 8), 9.0, dtype=self.dtype, device=DEV)
        ok(lib.leankv_causal_attend(ctypes.byref(self.c), qb.data_ptr(), g.data_ptr() if self.gated else None, n, out.data_ptr(),
                                    n + 8, T, start, self.status.data_ptr(), stream()))
        assert int(self.status) == 0 and bool((out[:, n:] == 9.0).all())
        return out[:, :n].float().cpu()

    def step(self, x, pos):
        lib = _native.mixers()
        q, k, sh, v, g = (t.to(DEV).contiguous() for t in x)
        out = torch.full((self.H * self.out_dim,), 9.0, device=DEV)
        state = torch.zeros(8, dtype=torch.int32, device=DEV)
        state[0] = pos
        own, com = (0, self.rot) if self.shared else (self.rot, 0)
        s = _native.CausalStep(q=q.data_ptr(), q_shared=q.data_ptr() + 4 * self.dim, k_new=k.data_ptr(), shared_new=sh.data_ptr(),
                               v_new=v.data_ptr() if self.dv else None, q_stride=self.dim + self.shared,
                               qs_stride=self.dim + self.shared, rate=self.rate.data_ptr(), rot_own=own, rot_shared=com,
                               gate=g.data_ptr() if self.gated else None, out=out.data_ptr(), state=state.data_ptr(),
                               max_pos=self.limit, ws=self.ws.data_ptr(), ws_bytes=self.ws.numel())
        ok(lib.leankv_causal_step(ctypes.byref(self.c), ctypes.byref(s), stream()))
        return out.cpu()

    def expected(self, x):
        q, k, sh, v, g = (t.double() for t in x)
        T, d = q.shape[0], self.dim
        if self.shared:
            q = torch.cat([q[..., :d], plain.rotate(q[..., d:], self.base, self.rot)], -1)
            turned = plain.rotate(sh[:, None], self.base, self.rot).expand(T, self.G, self.shared)
            keys = torch.cat([k, turned], -1)
        else:
            q, keys = plain.rotate(q, self.base, self.rot), plain.rotate(k, self.base, self.rot)
        o = plain.attend(q, keys, v if self.dv else k, self.scale, self.size).reshape(T, -1)
        return o * torch.sigmoid(g) if self.gated else o

    def feed(self, x, cuts):
        out, at, T = [], 0, x[0].shape[0]
        for n in cuts:
            n = min(n, T - at)
            if n == 0:
                break
            out.append(self.rows([t[at:at + n] for t in x], at) if n > 1 else self.step([t[at] for t in x], at)[None])
            at += n
        assert at == T
        return torch.cat(out)


def tol(dtype):
    return 3e-5 if dtype == F32 else 3e-2


# heads, kv heads, own key part, shared part, value columns (0: the key's own part), window
SHAPES = [(4, 2, 16, 0, 24, 1000), (3, 1, 10, 0, 6, 37), (8, 8, 64, 0, 64, 1), (12, 4, 48, 0, 32, 128), (32, 8, 128, 0, 128, 129),
          (5, 1, 112, 0, 144, 64), (40, 1, 32, 0, 16, 500), (6, 6, 20, 12, 28, 50), (4, 4, 128, 64, 128, 200),
          (20, 1, 96, 16, 0, 70), (33, 1, 64, 32, 0, 1000), (2, 2, 200, 8, 256, 90), (7, 7, 300, 0, 40, 60),
          (16, 1, 512, 64, 0, 130)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_causal_attention_portions_and_steps_agree_with_plain(dtype, shape):
    T = 300
    H, G, d, s, dv, size = shape
    kw = dict(rot=s if s else d // 4 * 2, scale=(d + s) ** -0.5, gated=H != 12)
    c = Causal(dtype, H, G, d, s, dv, size, T, T, **kw)
    x = c.inputs(T)
    want = c.expected(x)
    assert rel(c.feed(x, [T]), want) < tol(dtype)
    c = Causal(dtype, H, G, d, s, dv, size, 40, T, **kw)
    assert rel(c.feed(x, [2, 3, 40, 1, 1, 33, 40, 40, 7, 1, 2, 40, 40, 40, 40]), want) < tol(dtype)
    c = Causal(dtype, H, G, d, s, dv, size, 1, T, **kw)
    assert rel(c.feed(x, [1] * T), want) < tol(dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(4, 2, 32, 0, 48), (6, 1, 48, 16, 0), (3, 3, 24, 8, 40)], ids=str)
@pytest.mark.parametrize("size", [64, 127, 128, 129, 200, 256])
def test_one_key_stands_out_at_the_windows_edges(dtype, shape, size):
    """One key far larger than all others: seeing it or not decides the row, for the last position inside and the
    first one outside the window, at tile borders, in prompts and in decoding."""
    H, G, d, s, dv = shape
    T = 400
    for key in (0, 1, 127, 128, 130):
        c = Causal(dtype, H, G, d, s, dv, size, T, T, scale=1.0, gated=False)
        x = c.inputs(T, std=0.05)
        u = rnd(d, seed=3)
        u = u / u.norm()
        x[0][..., :d] += 3.0 * u
        x[1][key] += 6.0 * u
        if dv:
            x[3][key] += 4.0
        want = c.expected(x)
        edge = key + size
        rows = [r for r in (key, key + 1, edge - 2, edge - 1, edge, edge + 1, T - 1) if r < T]
        assert rel(c.feed(x, [T])[rows], want[rows]) < tol(dtype)
        if edge < T:
            assert rel(want[edge - 1][None], want[edge][None]) > 0.3
        c = Causal(dtype, H, G, d, s, dv, size, T, T, scale=1.0, gated=False)
        at = max(2, min(edge, T) - 3)
        got = c.feed(x, [at] + [1] * 6 + [T])
        assert rel(got[rows], want[rows]) < tol(dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("shape", [(4, 1, 64, 0, 64), (8, 2, 128, 0, 128), (10, 1, 64, 16, 0)], ids=str)
def test_far_key_among_thousands(dtype, shape):
    """A single early key that one late query looks for, over a long sequence, in a prompt and in decoding."""
    H, G, d, s, dv = shape
    T, far = 3001, 5
    c = Causal(dtype, H, G, d, s, dv, T, T, T, scale=1.0, gated=False)
    x = c.inputs(T, std=0.02)
    u = rnd(d, seed=3)
    u = u / u.norm()
    x[0][-2:, :, :d] += 4.0 * u
    x[1][far] += 4.0 * u
    if dv:
        x[3][far] += 3.0
    q = c.expected([t if i else torch.zeros_like(t) for i, t in enumerate(x)])[-1:]
    want = c.expected(x)[-2:]
    assert rel(want[-1:], q) > 0.5                         # the key decides
    assert rel(c.feed(x, [T])[-2:], want) < tol(dtype)
    c = Causal(dtype, H, G, d, s, dv, T, T, T, scale=1.0, gated=False)
    assert rel(c.feed(x, [T - 2, 1, 1])[-2:], want) < tol(dtype)


def test_scores_of_very_different_size_stay_exact():
    """The running maximum grows late and by far: outputs that were summed before are rescaled."""
    for dtype in (F32, BF16):
        c = Causal(dtype, 4, 1, 32, 0, 32, 600, 600, 600, scale=1.0, gated=False)
        x = c.inputs(600, std=0.5)
        x[1] *= torch.linspace(0.1, 8.0, 600).reshape(-1, 1, 1)
        want = c.expected([t.to(dtype).float() for t in x])
        x = [t.to(dtype).float() for t in x]
        assert rel(c.feed(x, [600]), want) < tol(dtype)
        c = Causal(dtype, 4, 1, 32, 0, 32, 600, 600, 600, scale=1.0, gated=False)
        assert rel(c.feed(x, [590] + [1] * 10)[-10:], want[-10:]) < tol(dtype)


# ── whole models ─────────────────────────────────────────────────────────────────────────────

WIDE = config([attention(heads=8, kv_heads=2, dim=64, vdim=64, dims=32, base=1e4, scale=0.125, ff=320),
               latent(heads=4, dim=32, rot_dim=16, vdim=48, q_rank=72, kv_rank=64, size=33, ff=None),
               latent(heads=16, dim=16, rot_dim=32, vdim=16, q_rank=40, kv_rank=136, size=140, scale=0.15, ff=512)],
              vocab=203, width=136, loop=(0, 2, 2), mult=0.3, cap=40.0)
ODD = config([attention(heads=1, kv_heads=1, dim=2, vdim=5, dims=2, base=2.0, ff=7),
              latent(heads=1, dim=1, rot_dim=2, vdim=3, q_rank=3, kv_rank=5, size=1, ff=9),
              attention(heads=3, kv_heads=3, dim=7, vdim=13, dims=4, ff=11),
              latent(heads=2, dim=5, rot_dim=4, vdim=3, q_rank=7, kv_rank=11, size=6, ff=None)], vocab=19, width=21, eps=1e-2,
             loop=(2, 4, 1), mult=1.0, cap=3.0)
LAST = config([latent(size=300), attention(kv_heads=4), attention(ff=None)], loop=(1, 3, 4), vocab=64, width=64)
MODELS = {"small": config(), "wide": WIDE, "odd": ODD, "last": LAST}
MODEL_TOL = {F32: 2e-4, BF16: 0.12}


def engine(name, dtype, limit=256, chunk=256, seed=0):
    cfg = MODELS[name] if isinstance(name, str) else name
    w = weights(cfg, seed)
    return cfg, w, MixerDecodeEngine(MixerModelConfig.from_dict(cfg), w, DEV, max_seq_len=limit, dtype=dtype, max_chunk=chunk)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MODELS))
def test_model_whole_portions_and_single_tokens(name, dtype):
    cfg, w, eng = engine(name, dtype)
    ids = tokens(cfg, 170)
    want = plain.forward(cfg, w, ids)
    assert rel(eng.extend(ids, list(range(170))), want) < MODEL_TOL[dtype]
    for cuts in ([2] * 85, [7, 1, 1, 31, 2, 94, 3, 31], [169, 1], [1] * 170):
        eng.reset()
        got, at = [], 0
        for n in cuts:
            got.append(eng.extend(ids[at:at + n], list(range(n))))
            at += n
        assert at == 170 and rel(torch.cat(got), want) < MODEL_TOL[dtype], cuts[:3]


def test_latents_heads_and_feed_forwards_of_one_number():
    """The norm of a branch (or latent) made from one number leaves little but a sign, so only in fp32."""
    cfg = config([latent(heads=1, dim=1, rot_dim=2, vdim=1, q_rank=1, kv_rank=1, size=3, ff=1),
                  attention(heads=1, kv_heads=1, dim=1, vdim=1, dims=0, ff=1)], loop=(0, 1, 2), eps=1e-2)
    _, w, eng = engine(cfg, F32, limit=40)
    ids = tokens(cfg, 40)
    got = torch.cat([eng.extend(ids[:20], list(range(20))), *(eng.extend([t], [0]) for t in ids[20:])])
    assert rel(got, plain.forward(cfg, w, ids)) < 1e-3


def test_stream_after_every_layer_run():
    cfg, w, eng = engine("small", F32)
    ids, seen, want = tokens(cfg, 40), [], []
    plain.forward(cfg, w, ids, layers_out=want)
    eng.stream_probe = lambda x: seen.append(x.clone())
    eng.extend(ids, [])
    assert len(seen) == len(want) == 8
    for a, b in zip(seen, want):
        assert rel(a, b) < 1e-4


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
    cfg, w, eng = engine("small", F32, limit=512, chunk=6)
    ids = tokens(cfg, 500)
    want = plain.forward(cfg, w, ids)
    assert min(l.mixer.state.ring for l in eng.layers) < 500       # rings of the windows wrap
    places = [450, 3, 499, 0, 77, 78]
    assert rel(eng.extend(ids, places), want[places]) < MODEL_TOL[F32]


def test_a_sequence_leaves_nothing_behind():
    for dtype in (F32, BF16):
        cfg, w, eng = engine("wide", dtype)
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


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_past_the_windows(dtype):
    cfg, w, eng = engine("small", dtype, limit=420)
    ids = tokens(cfg, 400, seed=4)
    want = plain.forward(cfg, w, ids)
    eng.extend(ids[:5], [])
    got = torch.cat([eng.extend([t], [0]) for t in ids[5:]])
    assert rel(got, want[5:]) < MODEL_TOL[dtype]


def test_passes_of_a_loop_keep_their_own_state():
    """Decoding after a prompt equals the whole prompt only if no pass reads another one's keys."""
    layers = [attention(), latent(size=12)]
    for times in (1, 2, 5):
        cfg = config(layers, loop=(0, 2, times))
        _, w, eng = engine(cfg, F32, limit=64)
        assert len(eng.layers) == 2 * times and len({l.mixer.c.k for l in eng.layers}) == 2 * times
        ids = tokens(cfg, 48, seed=times)
        want = plain.forward(cfg, w, ids)
        got = torch.cat([eng.extend(ids[:30], list(range(30))), *(eng.extend([t], [0]) for t in ids[30:])])
        assert rel(got, want) < MODEL_TOL[F32]
    no_loop = {k: v for k, v in config(layers).items() if k != "loop"}
    _, w, eng = engine(no_loop, F32, limit=64)
    ids = tokens(no_loop, 20)
    assert rel(eng.extend(ids, list(range(20))), plain.forward(no_loop, w, ids)) < MODEL_TOL[F32]


@pytest.mark.parametrize("eps,mult,cap", [(1e-2, 1.0, 2.0), (1e-6, -0.4, 500.0), (1e-5, 0.05, 25.0)])
def test_constants_come_from_the_configuration(eps, mult, cap):
    cfg = config([attention(scale=1.0, base=7.0, dims=2), latent(size=4, base=3e5, scale=0.9), latent(ff=None)], eps=eps, mult=mult,
                 cap=cap, loop=(0, 1, 2))
    w, ids = weights(cfg, 3), tokens(cfg, 60)
    eng = MixerDecodeEngine(MixerModelConfig.from_dict(cfg), w, DEV, max_seq_len=64, dtype=F32)
    want = plain.forward(cfg, w, ids)
    assert rel(eng.extend(ids[:40], list(range(40))), want[:40]) < MODEL_TOL[F32]
    assert rel(torch.cat([eng.extend([t], [0]) for t in ids[40:]]), want[40:]) < MODEL_TOL[F32]


def test_window_longer_than_the_sequence():
    cfg = config([latent(size=100000), attention()])
    _, w, eng = engine(config([latent(size=100000), attention()], loop=(0, 0, 1)), F32, limit=64)
    cfg["loop"] = {"start": 0, "stop": 0, "times": 1}
    ids = tokens(cfg, 64)
    want = plain.forward(cfg, w, ids)
    assert rel(eng.extend(ids[:50], list(range(50))), want[:50]) < MODEL_TOL[F32]
    assert rel(torch.cat([eng.extend([t], [0]) for t in ids[50:]]), want[50:]) < MODEL_TOL[F32]


def test_a_loop_over_another_designs_mixers():
    """The order of layers is the engine's, whatever the mixers: a parallel model's layer run twice."""
    cfg = parallel_config()
    w, ids = parallel_weights(cfg), tokens(cfg, 30)
    mc = MixerModelConfig.from_dict(cfg)
    twice = MixerModelConfig(**{**mc.__dict__, "loop": (0, 1, 2)})
    unrolled = dict(cfg, layers=[cfg["layers"][0], *cfg["layers"]])
    wu = {n: t for n, t in w.items() if not n.startswith("l")}
    for i, j in enumerate((0, 0, 1, 2)):
        wu.update({f"l{i}." + n.split(".", 1)[1]: t for n, t in w.items() if n.startswith(f"l{j}.")})
    a = MixerDecodeEngine(twice, w, DEV, max_seq_len=32, dtype=F32)
    b = MixerDecodeEngine(MixerModelConfig.from_dict(unrolled), wu, DEV, max_seq_len=32, dtype=F32)
    for part in ([*range(20)], [20], [21], [*range(22, 30)]):
        t = [ids[i] for i in part]
        assert torch.equal(a.extend(t, [len(t) - 1]), b.extend(t, [len(t) - 1]))


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
    read = lambda i: torch.frombuffer(bytearray((res / f"{i}.f32").read_bytes()), dtype=F32).reshape(-1, cfg["vocab"])
    la, lb = plain.forward(cfg, w, a), plain.forward(cfg, w, b)
    assert rel(read(0), la[[27, 4]]) < MODEL_TOL[F32] and rel(read(2), la[29:]) < MODEL_TOL[F32]
    assert rel(read(3), lb) < MODEL_TOL[F32]
