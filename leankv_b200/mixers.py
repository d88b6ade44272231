"""Token mixers: host side of the kernels in ``csrc/window_pool*``, ``csrc/time_mix.cu``, ``csrc/mixer_step.cu``
and ``csrc/causal_*``.

A mixer holds its parameters in kernel layout; ``bind`` gives a copy of it, on the same weights, its own part of
the sequence state, so that layers that run several times keep one state per pass. Every mechanism (window and
pooled blocks, query / key norm, weights mixed across heads, token shift, low-rank decay, rotation, latent keys,
gated outputs) is a parameter of the kernels, so a model combines them as its configuration says.

In a decode step a branch begins with a GEMV whose input fields the engine gives (``entry``: the stream and its
norm) and ends with one whose output fields it gives (``exit``: where the branch goes).
"""

from __future__ import annotations

import copy
import ctypes
from dataclasses import dataclass, replace
from typing import Optional

import torch

from . import _native
from .checkpoint import TensorBag
from .sequence_state import RING_STEP, SequenceState, pad16

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

    def __init__(self, spec: WindowPoolSpec, p: Parameters, eps: float):
        self.spec, self.eps, self.lib = spec, eps, _native.mixers()
        self.q_norm = p.vector("q.norm", spec.q_width)
        self.k_norm = p.vector("k.norm", spec.kv_heads * spec.dim)
        self.talk = p.vector("talk", spec.heads, spec.heads)

    def bind(self, seq: SequenceState) -> "WindowPoolAttention":
        bound = copy.copy(self)
        bound._attach(seq)
        return bound

    def _attach(self, seq: SequenceState) -> None:
        self.spec = spec = self.spec.bounded(seq.max_seq_len)
        self.seq = seq
        self.state = s = seq.window(spec.kv_heads, spec.dim, spec.vdim, spec.size, spec.pool)
        self.c = _native.WindowPool(
            dtype=dtype_code(seq.dtype), heads=spec.heads, kv_heads=spec.kv_heads, dim=spec.dim, vdim=spec.vdim,
            dim_pad=pad16(spec.dim), vdim_pad=pad16(spec.vdim), size=spec.size, pool=spec.pool, ring=s.ring,
            max_blocks=s.max_blocks, scale=spec.scale, k_ring=s.k_ring.data_ptr(), v_ring=s.v_ring.data_ptr(),
            k_pool=s.k_pool.data_ptr(), v_pool=s.v_pool.data_ptr(), q_norm=self.q_norm.data_ptr(),
            k_norm=self.k_norm.data_ptr(), eps=self.eps, talk=self.talk.data_ptr())

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

    def __init__(self, spec: TimeMixSpec, p: Parameters, eps: float):
        self.spec, self.eps, self.lib = spec, eps, _native.mixers()
        N = spec.out_width
        self.rank = p.bag.shape(p.prefix + "w1")[0]
        self.u = p.vector("u", spec.heads, spec.dim)
        self.w0 = p.vector("w0", N)
        self.norm = p.vector("norm", N)
        self.w2 = p.matrix("w2", N, self.rank).contiguous()
        # bf16: tanh(..) enters the second product as two bf16 numbers, so that the decay keeps 16 bits of it
        self.w2_rows = torch.cat([self.w2, self.w2], dim=1) if p.dtype == torch.bfloat16 else self.w2

    def bind(self, seq: SequenceState) -> "TimeMix":
        bound = copy.copy(self)
        bound._attach(seq)
        return bound

    def _attach(self, seq: SequenceState) -> None:
        spec, self.seq = self.spec, seq
        self.S = seq.carried(spec.heads, spec.dim, spec.dim)
        self.c = _native.TimeMix(dtype=dtype_code(seq.dtype), heads=spec.heads, dim=spec.dim, S=self.S.data_ptr(),
                                 u=self.u.data_ptr(), w0=self.w0.data_ptr(), norm=self.norm.data_ptr(), eps=self.eps)

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

    def __init__(self, spec: dict, p: Parameters, width: int, eps: float):
        spec = dict(spec)
        left = WindowPoolSpec.from_dict(spec.pop("left"))
        right = TimeMixSpec.from_dict(spec.pop("right"))
        self.left_scale, self.right_scale = float(spec.pop("left_scale")), float(spec.pop("right_scale"))
        if spec:
            raise ValueError(f"unknown mixer settings: {sorted(spec)}")
        self.lib, self.width = _native.mixers(), width
        pl, pr = p.under("left"), p.under("right")
        self.left = WindowPoolAttention(left, pl, eps)
        self.right = TimeMix(right, pr, eps)
        N, kd, vd = right.out_width, left.kv_heads * left.dim, left.kv_heads * left.vdim
        # all input projections as one matrix: q | k | v | r | k | v | g | w1 rows
        self.w_in = torch.cat([pl.matrix("q", left.q_width, width), pl.matrix("k", kd, width),
                               pl.matrix("v", vd, width), *(pr.matrix(s, N, width) for s in "rkvg"),
                               pr.matrix("w1", self.right.rank, width)]).contiguous()
        self.bias = torch.cat([pl.vector("q.b", left.q_width), pl.vector("k.b", kd), pl.vector("v.b", vd)])
        self.mu = torch.stack([pr.vector("mu." + s, width) for s in SHIFTED]).contiguous()
        self.w_out = torch.cat([pl.matrix("o", width, left.out_width), pr.matrix("o", width, N)], dim=1).contiguous()
        n0 = left.qkv_width
        self.in_width, self.out_width = n0 + 4 * N + self.right.rank, left.out_width + N
        self.w_qkv, self.w_rkvg = self.w_in[:n0], self.w_in[n0:n0 + 4 * N].view(4, N, width)
        self.w_low = self.w_in[n0 + 4 * N:]
        self.mix_end = [n0, n0 + N, n0 + 2 * N, n0 + 3 * N, n0 + 4 * N, self.in_width]
        self.step_floats = {"y": self.in_width, "out": self.out_width}

    def bind(self, seq: SequenceState) -> "ParallelMixer":
        bound = copy.copy(self)
        bound.seq, bound.left, bound.right = seq, self.left.bind(seq), self.right.bind(seq)
        bound.prev = seq.carried(2, self.width)
        return bound

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

    def prepare_step(self, entry: dict, exit: dict, bufs: dict, state: torch.Tensor, max_pos: int) -> None:
        """Argument blocks of the step's three launches on fixed buffers: stream -> y (projections) -> out
        (both mixers) -> branch output."""
        y, out = bufs["y"], bufs["out"]
        code, n0, N = dtype_code(self.seq.dtype), self.left.spec.qkv_width, self.right.spec.out_width
        a = _native.DenseGemv(w=self.w_in.data_ptr(), y=y.data_ptr(), dtype=code, rows=self.in_width,
                              cols=self.width, n_mix=len(self.mix_end),
                              prev=self.prev.data_ptr(), state=state.data_ptr(), bias=self.bias.data_ptr(),
                              bias_rows=n0, **entry)
        for i, e in enumerate(self.mix_end):
            a.mix_end[i] = e
            a.mu[i] = self.mu[i - 1].data_ptr() if i > 0 else None
        need = self.lib.leankv_mixer_step_workspace_bytes(ctypes.byref(self.left.c), max_pos)
        self._step_ws = torch.empty(max(need, 16), dtype=torch.uint8, device=y.device)
        s = _native.MixerStep(y=y.data_ptr(), qkv_off=0, rkvg_off=n0, w1_off=n0 + 4 * N, rank=self.right.rank,
                              w2=self.right.w2.data_ptr(), out=out.data_ptr(), right_off=self.left.spec.out_width,
                              left_scale=self.left_scale, right_scale=self.right_scale, state=state.data_ptr(),
                              max_pos=max_pos, ws=self._step_ws.data_ptr(), ws_bytes=self._step_ws.numel())
        o = _native.DenseGemv(w=self.w_out.data_ptr(), x=out.data_ptr(), dtype=code, rows=self.width,
                              cols=self.out_width, **exit)
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
        self.step_floats = {"act": self.inter}

    def portion(self, h: torch.Tensor) -> torch.Tensor:
        T, st = h.shape[0], torch.cuda.current_stream().cuda_stream
        gu = matmul(h, self.w_gu, exact_out=False)
        act = torch.empty(T, self.inter, dtype=h.dtype, device=h.device)
        _native.check(self.lib.leankv_silu_mul(gu.data_ptr(), act.data_ptr(), dtype_code(h.dtype), T, self.inter, st),
                      "silu_mul", self.lib)
        return matmul(act, self.w_down)

    def prepare_step(self, entry: dict, exit: dict, bufs: dict) -> None:
        code, act = dtype_code(self.dtype), bufs["act"]
        self._step_args = (
            _native.DenseGemv(w=self.w_gu.data_ptr(), y=act.data_ptr(), dtype=code, rows=self.inter, cols=self.width,
                              gated=1, **entry),
            _native.DenseGemv(w=self.w_down.data_ptr(), x=act.data_ptr(), dtype=code, rows=self.width, cols=self.inter,
                              **exit))

    def bind(self, seq: SequenceState) -> "GatedMLP":
        return copy.copy(self)

    def step(self, st: int) -> int:
        for a, what in zip(self._step_args, ("gate / up projection", "down projection")):
            _native.check(self.lib.leankv_dense_gemv(ctypes.byref(a), st), what, self.lib)
        return 2


# ── causal attention: whole sequence or a window, rotated keys, keys and values per head or from a latent ────

@dataclass(frozen=True)
class Rotation:
    """Coordinates 2i, 2i + 1 < dims of a head turn by position * base^(-2i / dims)."""

    base: float
    dims: int

    @classmethod
    def from_dict(cls, d: Optional[dict], limit: int) -> "Rotation":
        r = cls(1.0, 0) if d is None else cls(base=float(d["base"]), dims=int(d["dims"]))
        if d is not None and set(d) != {"base", "dims"}:
            raise ValueError(f"unknown rotation settings: {sorted(d)}")
        if r.dims < 0 or r.dims % 2 or r.dims > limit or r.base <= 0:
            raise ValueError(f"bad rotation: {d} of {limit} dimensions")
        return r

    def rate(self, device) -> torch.Tensor:
        i = torch.arange(max(self.dims // 2, 1), dtype=torch.float64)
        return (self.base ** (-2.0 * i / max(self.dims, 1))).float().to(device)


def _window(mask: Optional[dict]) -> Optional[int]:
    """Visible positions of a ``mask`` entry; None sees the whole sequence."""
    if mask is None:
        return None
    if set(mask) != {"size"} or int(mask["size"]) < 1:
        raise ValueError(f"bad mask settings: {mask}")
    return int(mask["size"])


def _checked(spec, *sizes: int):
    if min(sizes) < 1:
        raise ValueError(f"bad attention sizes: {spec}")
    return spec


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    size: Optional[int]

    @classmethod
    def from_dict(cls, d: dict) -> "AttentionSpec":
        d = dict(d)
        rot, size = Rotation.from_dict(d.pop("rot", None), d["dim"]), _window(d.pop("mask", None))
        s = _checked(cls(rot=rot, size=size, **d), d["heads"], d["kv_heads"], d["dim"], d["vdim"])
        if s.heads % s.kv_heads:
            raise ValueError(f"bad attention sizes: {s}")
        return s


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotation
    size: Optional[int]

    @classmethod
    def from_dict(cls, d: dict) -> "LatentSpec":
        d = dict(d)
        rot, size = Rotation.from_dict(d.pop("rot", None), d["rot_dim"]), _window(d.pop("mask", None))
        return _checked(cls(rot=rot, size=size, **d), d["heads"], d["dim"], d["vdim"], d["q_rank"], d["kv_rank"],
                        d["rot_dim"] + 1)


class _CausalMixer:
    """What the two attention mixers share: rows into rings and operand buffers, the decode step's workspace."""

    def bind(self, seq: SequenceState):
        bound = copy.copy(self)
        bound.seq = seq
        bound.size = seq.max_seq_len if self.spec.size is None else min(self.spec.size, seq.max_seq_len)
        bound.rate = self.spec.rot.rate(seq.dev)
        bound._attach(seq)
        return bound

    def _place(self, start: int, rows: int, segments: list) -> None:
        a = _native.PlaceRows(dtype=dtype_code(self.seq.dtype), rows=rows, start=start, n_seg=len(segments),
                              rate=self.rate.data_ptr(), eps=self.eps)
        for i, s in enumerate(segments):
            a.seg[i] = _native.RowSegment(**s)
        _native.check(self.lib.leankv_place_rows(ctypes.byref(a), torch.cuda.current_stream().cuda_stream), "place_rows",
                      self.lib)

    def _attend(self, c: _native.CausalAttn, q: torch.Tensor, gate: Optional[torch.Tensor], start: int) -> torch.Tensor:
        T = q.shape[0]
        out = torch.empty(T, c.heads * c.vdim, dtype=q.dtype, device=q.device)
        _native.check(self.lib.leankv_causal_attend(
            ctypes.byref(c), q.data_ptr(), _native.ptr(gate), gate.stride(0) if gate is not None else 0, out.data_ptr(),
            out.stride(0), T, start, self.seq.status.data_ptr(), torch.cuda.current_stream().cuda_stream),
            "causal_attend", self.lib)
        return out

    def _step_block(self, state: torch.Tensor, max_pos: int, **kw) -> _native.CausalStep:
        need = self.lib.leankv_causal_step_workspace_bytes(ctypes.byref(self.c), max_pos)
        if need == 0:
            raise ValueError(f"the decode step does not take these sizes: {self.spec}")
        self._step_ws = torch.zeros(need, dtype=torch.uint8, device=state.device)
        return _native.CausalStep(eps=self.eps, rate=self.rate.data_ptr(), state=state.data_ptr(), max_pos=max_pos,
                                  ws=self._step_ws.data_ptr(), ws_bytes=need, **kw)

    def step(self, st: int) -> int:
        """Launch the step; returns the number of kernels."""
        for a in self._step_args:
            if isinstance(a, _native.CausalStep):
                _native.check(self.lib.leankv_causal_step(ctypes.byref(self.c), ctypes.byref(a), st), "causal_step", self.lib)
            else:
                _native.check(self.lib.leankv_dense_gemv(ctypes.byref(a), st), "projection", self.lib)
        return len(self._step_args)


class RotaryAttention(_CausalMixer):
    """Grouped-query attention over rotated queries and keys, the heads gated by a projection of the input."""

    def __init__(self, spec: dict, p: Parameters, width: int, eps: float):
        self.spec = s = AttentionSpec.from_dict(spec)
        self.lib, self.width, self.eps = _native.mixers(), width, eps
        nq, nk, nv, no = s.heads * s.dim, s.kv_heads * s.dim, s.kv_heads * s.vdim, s.heads * s.vdim
        self.w_in = torch.cat([p.matrix("q", nq, width), p.matrix("k", nk, width), p.matrix("v", nv, width),
                               p.matrix("g", no, width)]).contiguous()
        self.w_out = p.matrix("o", width, no).contiguous()
        self.at_k, self.at_v, self.at_g, self.in_width = nq, nq + nk, nq + nk + nv, nq + nk + nv + no
        self.out_width = no
        self.step_floats = {"y": self.in_width, "out": no}

    def _attach(self, seq: SequenceState) -> None:
        s = self.spec
        self.state = st = seq.causal(s.kv_heads, s.dim, s.vdim, 0, self.size)
        self.c = _native.CausalAttn(dtype=dtype_code(seq.dtype), heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim,
                                    dim_pad=pad16(s.dim), vdim_pad=pad16(s.vdim), size=self.size, scale=s.scale,
                                    k=st.k.data_ptr(), v=st.v.data_ptr(), k_ring=st.ring, k_rows=st.ring)

    def place(self, y: torch.Tensor, start: int) -> torch.Tensor:
        """Projections [T][q | k | v | ..]: keys and values into the rings; returns the queries."""
        s, c, T = self.spec, self.c, y.shape[0]
        q = torch.empty(T, s.heads, c.dim_pad, dtype=self.seq.dtype, device=y.device)
        src, n = y.data_ptr(), y.stride(0)
        self._place(start, T, [
            dict(src=src, ld=n, heads=s.heads, head_stride=s.dim, n=s.dim, dst=q.data_ptr(), dst_ld=s.heads * c.dim_pad,
                 dst_head_stride=c.dim_pad, n_pad=c.dim_pad, rot=s.rot.dims),
            dict(src=src + 4 * self.at_k, ld=n, heads=s.kv_heads, head_stride=s.dim, n=s.dim, dst=c.k,
                 dst_ld=s.kv_heads * c.dim_pad, dst_head_stride=c.dim_pad, n_pad=c.dim_pad, ring=c.k_ring, rot=s.rot.dims),
            dict(src=src + 4 * self.at_v, ld=n, heads=s.kv_heads, head_stride=s.vdim, n=s.vdim, dst=c.v,
                 dst_ld=s.kv_heads * c.vdim_pad, dst_head_stride=c.vdim_pad, n_pad=c.vdim_pad, ring=c.k_ring)])
        return q

    def portion(self, h: torch.Tensor, mixed, start: int, scratch) -> torch.Tensor:
        y = matmul(h, self.w_in)
        return matmul(self._attend(self.c, self.place(y, start), y[:, self.at_g:], start), self.w_out)

    def prepare_step(self, entry: dict, exit: dict, bufs: dict, state: torch.Tensor, max_pos: int) -> None:
        """Stream -> y (q | k | v | gate) -> out (gated heads) -> branch output."""
        s, code, y, out = self.spec, self.c.dtype, bufs["y"].data_ptr(), bufs["out"].data_ptr()
        self._step_args = (
            _native.DenseGemv(w=self.w_in.data_ptr(), y=y, dtype=code, rows=self.in_width, cols=self.width, **entry),
            self._step_block(state, max_pos, q=y, q_stride=s.dim, k_new=y + 4 * self.at_k, v_new=y + 4 * self.at_v,
                             rot_own=s.rot.dims, gate=y + 4 * self.at_g, out=out),
            _native.DenseGemv(w=self.w_out.data_ptr(), x=out, dtype=code, rows=self.width, cols=self.out_width, **exit))


def _per_head_padded(w: torch.Tensor, heads: int, n: int) -> torch.Tensor:
    """[heads * n, k] with zero rows behind every head, so that products come out [.., heads, pad16(n)]."""
    if n % 16 == 0:
        return w.contiguous()
    out = torch.zeros(heads, pad16(n), w.shape[1], dtype=w.dtype, device=w.device)
    out[:, :n] = w.reshape(heads, n, -1)
    return out.reshape(heads * pad16(n), -1)


class LatentAttention(_CausalMixer):
    """Attention whose cache is one normed latent and one rotated key part per position, shared by all heads.

    Prompts expand the latents they see into per-head keys and values. A decode step folds the key expansion
    into the query and the value expansion into the output, and attends over the latents themselves."""

    def __init__(self, spec: dict, p: Parameters, width: int, eps: float):
        self.spec = s = LatentSpec.from_dict(spec)
        self.lib, self.width, self.eps = _native.mixers(), width, eps
        H, d, r, n = s.heads, s.dim, s.rot_dim, s.kv_rank
        self.w_down = torch.cat([p.matrix("dq", s.q_rank, width), p.matrix("dkv", n + r, width)]).contiguous()
        self.q_norm, self.kv_norm = p.vector("dq.norm", s.q_rank), p.vector("dkv.norm", n)
        self.w_q = p.matrix("uq", H * (d + r), s.q_rank).contiguous()
        w_k, w_v = p.matrix("uk", H * d, n), p.matrix("uv", H * s.vdim, n)
        self.w_k, self.w_v = _per_head_padded(w_k, H, d), _per_head_padded(w_v, H, s.vdim)      # prompts
        self.w_fold = w_k.reshape(H, d, n).transpose(1, 2).contiguous()                         # decode: [H][rank][dim]
        self.w_unfold = self.w_v if s.vdim % 16 == 0 else w_v.contiguous()
        self.w_out = p.matrix("o", width, H * s.vdim).contiguous()
        self.in_width, self.out_width = s.q_rank + n + r, H * s.vdim
        self.step_floats = {"y": self.in_width, "q": H * (d + r), "folded": H * n, "latent": H * n, "out": self.out_width}

    def _attach(self, seq: SequenceState) -> None:
        s = self.spec
        self.state = st = seq.causal(1, s.kv_rank, 0, s.rot_dim, self.size)
        self.c = _native.CausalAttn(dtype=dtype_code(seq.dtype), heads=s.heads, kv_heads=1, dim=s.kv_rank, shared_dim=s.rot_dim,
                                    vdim=s.kv_rank, dim_pad=pad16(s.kv_rank), shared_pad=pad16(s.rot_dim),
                                    vdim_pad=pad16(s.kv_rank), size=self.size, scale=s.scale, k=st.k.data_ptr(), k_ring=st.ring,
                                    k_rows=st.ring, shared=_native.ptr(st.shared), s_ring=st.ring)

    def place_latents(self, y: torch.Tensor, start: int) -> torch.Tensor:
        """Projections [T][query latent | latent | key part]: the last two into the rings; returns the normed query latents."""
        s, c, T = self.spec, self.c, y.shape[0]
        cq = torch.empty(T, s.q_rank, dtype=self.seq.dtype, device=y.device)
        src, ld, n, r = y.data_ptr(), y.stride(0), s.kv_rank, s.rot_dim
        segments = [dict(src=src, ld=ld, heads=1, n=s.q_rank, dst=cq.data_ptr(), dst_ld=s.q_rank, n_pad=s.q_rank,
                         gain=self.q_norm.data_ptr()),
                    dict(src=src + 4 * s.q_rank, ld=ld, heads=1, n=n, dst=c.k, dst_ld=c.dim_pad, n_pad=c.dim_pad,
                         ring=c.k_ring, gain=self.kv_norm.data_ptr())]
        if r:
            segments.append(dict(src=src + 4 * (s.q_rank + n), ld=ld, heads=1, n=r, dst=c.shared, dst_ld=c.shared_pad,
                                 n_pad=c.shared_pad, ring=c.s_ring, rot=s.rot.dims))
        self._place(start, T, segments)
        return cq

    def place_q(self, z: torch.Tensor, start: int) -> torch.Tensor:
        """Queries [T][heads][own | rotated part] as operands, both parts padded."""
        s, T = self.spec, z.shape[0]
        H, d, r, dp, rp = s.heads, s.dim, s.rot_dim, pad16(s.dim), pad16(s.rot_dim)
        q = torch.empty(T, H, dp + rp, dtype=self.seq.dtype, device=z.device)
        part = lambda off, at, m, pad, rot: dict(src=z.data_ptr() + 4 * off, ld=z.stride(0), heads=H, head_stride=d + r, n=m,
                                                 dst=q.data_ptr() + q.element_size() * at, dst_ld=H * (dp + rp),
                                                 dst_head_stride=dp + rp, n_pad=pad, rot=rot)
        self._place(start, T, [part(0, 0, d, dp, 0)] + ([part(d, dp, r, rp, s.rot.dims)] if r else []))
        return q

    def _expanded(self, start: int, T: int) -> tuple:
        """Per-head keys and values of the positions that a portion sees, from a multiple of the ring step on: the
        attention over them, and the buffers it reads."""
        s, c, ring = self.spec, self.c, self.state.ring
        base = max(0, start - self.size + 1) // RING_STEP * RING_STEP
        n = start + T - base
        k = torch.empty(n, s.heads * pad16(s.dim), dtype=self.seq.dtype, device=self.seq.dev)
        v = torch.empty(n, s.heads * pad16(s.vdim), dtype=self.seq.dtype, device=self.seq.dev)
        at = 0
        while at < n:
            slot = (base + at) % ring
            m = min(n - at, ring - slot)
            latents = self.state.k[slot:slot + m, 0, :s.kv_rank]
            torch.mm(latents, self.w_k.t(), out=k[at:at + m])
            torch.mm(latents, self.w_v.t(), out=v[at:at + m])
            at += m
        e = _native.CausalAttn(dtype=c.dtype, heads=s.heads, kv_heads=s.heads, dim=s.dim, shared_dim=s.rot_dim, vdim=s.vdim,
                               dim_pad=pad16(s.dim), shared_pad=c.shared_pad, vdim_pad=pad16(s.vdim), size=self.size,
                               scale=s.scale, k=k.data_ptr(), v=v.data_ptr(), k_base=base,
                               k_ring=(n + RING_STEP - 1) // RING_STEP * RING_STEP, k_rows=n, shared=c.shared, s_ring=c.s_ring)
        return e, (k, v)

    def portion(self, h: torch.Tensor, mixed, start: int, scratch) -> torch.Tensor:
        cq = self.place_latents(matmul(h, self.w_down), start)
        q = self.place_q(matmul(cq, self.w_q), start)
        e, buffers = self._expanded(start, h.shape[0])
        return matmul(self._attend(e, q, None, start), self.w_out)

    def prepare_step(self, entry: dict, exit: dict, bufs: dict, state: torch.Tensor, max_pos: int) -> None:
        """Stream -> y (query latent | latent | key part) -> q -> folded (queries against latents) -> latent (mean
        latents) -> out (heads) -> branch output."""
        s, code = self.spec, self.c.dtype
        H, d, r, n = s.heads, s.dim, s.rot_dim, s.kv_rank
        y, q, folded, latent, out = (bufs[b].data_ptr() for b in ("y", "q", "folded", "latent", "out"))
        gemv = lambda w, **kw: _native.DenseGemv(w=w.data_ptr(), dtype=code, **kw)
        self._step_args = (
            gemv(self.w_down, y=y, rows=self.in_width, cols=self.width, **entry),
            gemv(self.w_q, x=y, y=q, rows=H * (d + r), cols=s.q_rank, gain=self.q_norm.data_ptr(), gain_per_col=1, eps=self.eps),
            gemv(self.w_fold, x=q, y=folded, rows=H * n, cols=d, group_rows=n, group_stride=d + r),
            self._step_block(state, max_pos, q=folded, q_stride=n, q_shared=q + 4 * d if r else None, qs_stride=d + r,
                             k_new=y + 4 * s.q_rank, shared_new=y + 4 * (s.q_rank + n) if r else None,
                             k_gain=self.kv_norm.data_ptr(), rot_shared=s.rot.dims, out=latent),
            gemv(self.w_unfold, x=latent, y=out, rows=H * s.vdim, cols=n, group_rows=s.vdim, group_stride=n),
            gemv(self.w_out, x=out, rows=self.width, cols=self.out_width, **exit))


MIXERS = {"parallel": ParallelMixer, "attention": RotaryAttention, "latent_attention": LatentAttention}
