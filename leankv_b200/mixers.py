"""Token mixers: host side of the kernels in ``csrc/window_pool*``, ``csrc/time_mix.cu`` and
``csrc/mixer_step.cu``.

A mixer owns its parameters in kernel layout and its part of the sequence state. Every mechanism (window and
pooled blocks, query / key norm, weights mixed across heads, token shift, low-rank decay) is a parameter of
the kernels, so a model combines them as its configuration says.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass, replace

import torch

from . import _native
from .checkpoint import TensorBag
from .sequence_state import SequenceState, pad16

SHIFTED = ("r", "k", "v", "g", "w")        # the inputs of the time mixing, each with a shift of its own


def dtype_code(dtype: torch.dtype) -> int:
    return {torch.bfloat16: _native.DT_BF16, torch.float32: _native.DT_F32}[dtype]


def matmul(a: torch.Tensor, w: torch.Tensor, exact_out: bool = True) -> torch.Tensor:
    """a [.., K] times w [N, K] transposed; fp32 result if ``exact_out``, else of a's type."""
    if exact_out and a.dtype != torch.float32:
        return torch.mm(a, w.t(), out_dtype=torch.float32)
    return torch.mm(a, w.t())


@dataclass(frozen=True)
class WindowPoolSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    size: int
    pool: int
    scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "WindowPoolSpec":
        d, mask = dict(d), dict(d["mask"])
        del d["mask"]
        spec = cls(size=mask.pop("size"), pool=mask.pop("pool"), **d)
        if mask:
            raise ValueError(f"unknown mask settings: {sorted(mask)}")
        if min(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.size, spec.pool) < 1 or spec.heads % spec.kv_heads:
            raise ValueError(f"bad attention sizes: {spec}")
        return spec

    def bounded(self, max_seq_len: int) -> "WindowPoolSpec":
        """The same visibility for sequences of at most ``max_seq_len`` tokens, with no larger ring than they
        need: a longer window shows every token, a longer block is never complete."""
        return replace(self, size=min(self.size, max_seq_len), pool=min(self.pool, max_seq_len + 1))

    @property
    def q_width(self) -> int:
        return self.heads * self.dim

    @property
    def qkv_width(self) -> int:
        return self.q_width + self.kv_heads * (self.dim + self.vdim)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class TimeMixSpec:
    heads: int
    dim: int

    @classmethod
    def from_dict(cls, d: dict) -> "TimeMixSpec":
        spec = cls(**d)
        if min(spec.heads, spec.dim) < 1:
            raise ValueError(f"bad time-mixing sizes: {spec}")
        return spec

    @property
    def out_width(self) -> int:
        return self.heads * self.dim


class Parameters:
    """Checkpoint tensors under one prefix, converted for the kernels."""

    def __init__(self, bag: TensorBag, prefix: str, device, dtype: torch.dtype):
        self.bag, self.prefix, self.dev, self.dtype = bag, prefix, device, dtype

    def under(self, name: str) -> "Parameters":
        return Parameters(self.bag, f"{self.prefix}{name}.", self.dev, self.dtype)

    def matrix(self, name: str, *shape: int) -> torch.Tensor:
        return self.bag.take(self.prefix + name, *shape).to(self.dev, self.dtype)

    def vector(self, name: str, *shape: int) -> torch.Tensor:
        return self.bag.take(self.prefix + name, *shape).to(self.dev, torch.float32).contiguous()


class WindowPoolAttention:
    """Window + pooled-block attention over normed queries and keys, weights mixed across heads."""

    def __init__(self, spec: WindowPoolSpec, p: Parameters, seq: SequenceState, eps: float):
        self.spec = spec = spec.bounded(seq.max_seq_len)
        self.seq = seq
        self.lib = _native.mixers()
        self.q_norm = p.vector("q.norm", spec.q_width)
        self.k_norm = p.vector("k.norm", spec.kv_heads * spec.dim)
        self.talk = p.vector("talk", spec.heads, spec.heads)
        self.state = s = seq.window(spec.kv_heads, spec.dim, spec.vdim, spec.size, spec.pool)
        self.c = _native.WindowPool(
            dtype=dtype_code(seq.dtype), heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim, vdim=spec.vdim,
            dim_pad=pad16(spec.dim), vdim_pad=pad16(spec.vdim), size=spec.size, pool=spec.pool, ring=s.ring,
            max_blocks=s.max_blocks, scale=spec.scale, k_ring=s.k_ring.data_ptr(), v_ring=s.v_ring.data_ptr(),
            k_pool=s.k_pool.data_ptr(), v_pool=s.v_pool.data_ptr(), q_norm=self.q_norm.data_ptr(),
            k_norm=self.k_norm.data_ptr(), eps=eps, talk=self.talk.data_ptr())

    def portion(self, qkv: torch.Tensor, bias: torch.Tensor, out: torch.Tensor, out_scale: float, start: int,
                scratch) -> None:
        """qkv fp32 [T][.. q | k | v columns first]; writes out[:, :heads * vdim] (a view of wider rows)."""
        T, st = qkv.shape[0], torch.cuda.current_stream().cuda_stream
        q = torch.empty(T, self.spec.heads, self.c.dim_pad, dtype=self.seq.dtype, device=qkv.device)
        ref = ctypes.byref(self.c)
        _native.check(self.lib.leankv_window_pool_append(ref, qkv.data_ptr(), qkv.stride(0), bias.data_ptr(),
                                                         q.data_ptr(), T, start, st), "window_pool_append", self.lib)
        ws = scratch(self.lib.leankv_window_pool_workspace_bytes(ref, T, start + T))
        _native.check(self.lib.leankv_window_pool_attend(ref, q.data_ptr(), out.data_ptr(), out.stride(0), out_scale,
                                                         T, start, ws.data_ptr(), ws.numel(), st),
                      "window_pool_attend", self.lib)


class TimeMix:
    """Matrix-state recurrence with a data-dependent decay per key channel and a bonus for the current token."""

    def __init__(self, spec: TimeMixSpec, p: Parameters, seq: SequenceState, eps: float):
        self.spec, self.seq = spec, seq
        self.lib = _native.mixers()
        N = spec.out_width
        self.rank = p.bag.shape(p.prefix + "w1")[0]
        self.u = p.vector("u", spec.heads, spec.dim)
        self.w0 = p.vector("w0", N)
        self.norm = p.vector("norm", N)
        self.w2 = p.matrix("w2", N, self.rank).contiguous()
        # bf16: tanh(..) enters the second product as two bf16 numbers, so that the decay keeps 16 bits of it
        self.w2_rows = torch.cat([self.w2, self.w2], dim=1) if seq.dtype == torch.bfloat16 else self.w2
        self.S = seq.carried(spec.heads, spec.dim, spec.dim)
        self.c = _native.TimeMix(dtype=dtype_code(seq.dtype), heads=spec.heads, dim=spec.dim, S=self.S.data_ptr(),
                                 u=self.u.data_ptr(), w0=self.w0.data_ptr(), norm=self.norm.data_ptr(), eps=eps)

    def portion(self, rkvg: torch.Tensor, low: torch.Tensor, out: torch.Tensor, out_scale: float, scratch) -> None:
        """rkvg [4][T][heads * dim]; low fp32 [T][rank]; writes out[:, :heads * dim] (a view of wider rows)."""
        T, st = low.shape[0], torch.cuda.current_stream().cuda_stream
        t = torch.empty(T, self.w2_rows.shape[1], dtype=self.seq.dtype, device=low.device)
        _native.check(self.lib.leankv_tanh_split(low.data_ptr(), t.data_ptr(), self.c.dtype, T, self.rank, st),
                      "tanh_split", self.lib)
        z = matmul(t, self.w2_rows)
        ref = ctypes.byref(self.c)
        ws = scratch(self.lib.leankv_time_mix_workspace_bytes(ref, T))
        _native.check(self.lib.leankv_time_mix_rows(ref, *(rkvg[i].data_ptr() for i in range(4)), z.data_ptr(),
                                                    out.data_ptr(), out.stride(0), out_scale, T, ws.data_ptr(),
                                                    ws.numel(), st), "time_mix_rows", self.lib)


class ParallelMixer:
    """Attention (left) and time mixing (right) side by side on the same input, their outputs scaled and
    summed by one projection over the concatenation."""

    def __init__(self, spec: dict, p: Parameters, seq: SequenceState, width: int, eps: float):
        spec = dict(spec)
        left = WindowPoolSpec.from_dict(spec.pop("left"))
        right = TimeMixSpec.from_dict(spec.pop("right"))
        self.left_scale, self.right_scale = float(spec.pop("left_scale")), float(spec.pop("right_scale"))
        if spec:
            raise ValueError(f"unknown mixer settings: {sorted(spec)}")
        self.lib, self.seq, self.width = _native.mixers(), seq, width
        pl, pr = p.under("left"), p.under("right")
        self.left = WindowPoolAttention(left, pl, seq, eps)
        self.right = TimeMix(right, pr, seq, eps)
        N, kd, vd = right.out_width, left.kv_heads * left.dim, left.kv_heads * left.vdim
        # all input projections as one matrix: q | k | v | r | k | v | g | w1 rows
        self.w_in = torch.cat([pl.matrix("q", left.q_width, width), pl.matrix("k", kd, width),
                               pl.matrix("v", vd, width), *(pr.matrix(s, N, width) for s in "rkvg"),
                               pr.matrix("w1", self.right.rank, width)]).contiguous()
        self.bias = torch.cat([pl.vector("q.b", left.q_width), pl.vector("k.b", kd), pl.vector("v.b", vd)])
        self.mu = torch.stack([pr.vector("mu." + s, width) for s in SHIFTED]).contiguous()
        self.w_out = torch.cat([pl.matrix("o", width, left.out_width), pr.matrix("o", width, N)], dim=1).contiguous()
        self.prev = seq.carried(2, width)
        n0 = left.qkv_width
        self.in_width, self.out_width = n0 + 4 * N + self.right.rank, left.out_width + N
        self.w_qkv, self.w_rkvg = self.w_in[:n0], self.w_in[n0:n0 + 4 * N].view(4, N, width)
        self.w_low = self.w_in[n0 + 4 * N:]
        self.mix_end = [n0, n0 + N, n0 + 2 * N, n0 + 3 * N, n0 + 4 * N, self.in_width]

    # ── portion of a prompt ──────────────────────────────────────────────

    def portion(self, h: torch.Tensor, mixed: torch.Tensor, start: int, scratch) -> torch.Tensor:
        """h [T][width] and its five shifted mixes [5][T][width] -> fp32 [T][width]."""
        T, left, right = h.shape[0], self.left, self.right
        cat = torch.empty(T, self.out_width, dtype=h.dtype, device=h.device)
        left.portion(matmul(h, self.w_qkv), self.bias, cat, self.left_scale, start, scratch)
        rkvg = torch.bmm(mixed[:4], self.w_rkvg.transpose(1, 2))
        right.portion(rkvg, matmul(mixed[4], self.w_low), cat[:, left.spec.out_width:], self.right_scale, scratch)
        return matmul(cat, self.w_out)

    # ── decode step ──────────────────────────────────────────────────────

    def prepare_step(self, gain: torch.Tensor, eps: float, x: torch.Tensor, scale: torch.Tensor, y: torch.Tensor,
                     out: torch.Tensor, state: torch.Tensor, max_pos: int) -> None:
        """Argument blocks of the step's three launches on fixed buffers: x (stream) -> y (projections) -> out
        (both mixers) -> x += scale * W out."""
        code, n0, N = dtype_code(self.seq.dtype), self.left.spec.qkv_width, self.right.spec.out_width
        a = _native.DenseGemv(w=self.w_in.data_ptr(), x=x.data_ptr(), y=y.data_ptr(), dtype=code, rows=self.in_width,
                              cols=self.width, gain=gain.data_ptr(), eps=eps, n_mix=len(self.mix_end),
                              prev=self.prev.data_ptr(), state=state.data_ptr(), bias=self.bias.data_ptr(),
                              bias_rows=n0)
        for i, e in enumerate(self.mix_end):
            a.mix_end[i] = e
            a.mu[i] = self.mu[i - 1].data_ptr() if i > 0 else None
        need = self.lib.leankv_mixer_step_workspace_bytes(ctypes.byref(self.left.c), max_pos)
        self._step_ws = torch.empty(max(need, 16), dtype=torch.uint8, device=x.device)
        s = _native.MixerStep(y=y.data_ptr(), qkv_off=0, rkvg_off=n0, w1_off=n0 + 4 * N, rank=self.right.rank,
                              w2=self.right.w2.data_ptr(), out=out.data_ptr(), right_off=self.left.spec.out_width,
                              left_scale=self.left_scale, right_scale=self.right_scale, state=state.data_ptr(),
                              max_pos=max_pos, ws=self._step_ws.data_ptr(), ws_bytes=self._step_ws.numel())
        o = _native.DenseGemv(w=self.w_out.data_ptr(), x=out.data_ptr(), y=x.data_ptr(), dtype=code, rows=self.width,
                              cols=self.out_width, scale=scale.data_ptr(), residual=x.data_ptr())
        self._step_args = (a, s, o)

    def step(self, st: int) -> int:
        """Launch the step; returns the number of kernels."""
        a, s, o = self._step_args
        _native.check(self.lib.leankv_dense_gemv(ctypes.byref(a), st), "input projections", self.lib)
        _native.check(self.lib.leankv_mixer_step(ctypes.byref(self.left.c), ctypes.byref(self.right.c),
                                                 ctypes.byref(s), st), "mixer_step", self.lib)
        _native.check(self.lib.leankv_dense_gemv(ctypes.byref(o), st), "output projection", self.lib)
        return 3


class GatedMLP:
    """W_down (silu(W_gate h) * (W_up h))."""

    def __init__(self, spec: dict, p: Parameters, width: int):
        spec = dict(spec)
        kind, self.inter = spec.pop("kind"), spec.pop("ff")
        if kind != "dense" or spec:
            raise ValueError(f"unknown feed-forward: {kind}, settings {sorted(spec)}")
        self.lib, self.width, self.dtype = _native.mixers(), width, p.dtype
        self.w_gu = torch.cat([p.matrix("gate", self.inter, width), p.matrix("up", self.inter, width)]).contiguous()
        self.w_down = p.matrix("down", width, self.inter).contiguous()

    def portion(self, h: torch.Tensor) -> torch.Tensor:
        T, st = h.shape[0], torch.cuda.current_stream().cuda_stream
        gu = matmul(h, self.w_gu, exact_out=False)
        act = torch.empty(T, self.inter, dtype=h.dtype, device=h.device)
        _native.check(self.lib.leankv_silu_mul(gu.data_ptr(), act.data_ptr(), dtype_code(h.dtype), T, self.inter, st),
                      "silu_mul", self.lib)
        return matmul(act, self.w_down)

    def prepare_step(self, gain: torch.Tensor, eps: float, x: torch.Tensor, scale: torch.Tensor,
                     act: torch.Tensor) -> None:
        code = dtype_code(self.dtype)
        self._step_args = (
            _native.DenseGemv(w=self.w_gu.data_ptr(), x=x.data_ptr(), y=act.data_ptr(), dtype=code, rows=self.inter,
                              cols=self.width, gated=1, gain=gain.data_ptr(), eps=eps),
            _native.DenseGemv(w=self.w_down.data_ptr(), x=act.data_ptr(), y=x.data_ptr(), dtype=code, rows=self.width,
                              cols=self.inter, scale=scale.data_ptr(), residual=x.data_ptr()))

    def step(self, st: int) -> int:
        for a, what in zip(self._step_args, ("gate / up projection", "down projection")):
            _native.check(self.lib.leankv_dense_gemv(ctypes.byref(a), st), what, self.lib)
        return 2


MIXERS = {"parallel": ParallelMixer}
