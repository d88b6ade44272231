"""Decode engine of models whose layers are pre-norm token mixers with bounded state (``mixers.py``): one
residual stream in fp32, a norm with a single gain, a per-channel scale on every branch.

Prompts run in portions of any size (library GEMMs between the row kernels); a single token runs as one
replay of the captured step graph, five kernels per layer: {norm, token shift, every input projection},
{both mixers}, {output projection, residual}, {norm, gate / up, silu}, {down, residual}.
"""

from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Optional, Sequence

import torch

from . import _native
from .checkpoint import TensorBag
from .decode_loop import DecodeLoop
from .mixers import MIXERS, GatedMLP, Parameters, dtype_code, matmul
from .sequence_state import SequenceState


@dataclass(frozen=True)
class MixerModelConfig:
    """Sizes and constants of a mixer model, as its ``config.json`` gives them."""

    architecture: str
    vocab_size: int
    hidden_size: int
    eps: float
    layers: tuple           # per layer: {"type", "mixer": {...}, "mlp": {...} or None}

    @classmethod
    def from_dict(cls, c: dict) -> "MixerModelConfig":
        known = {"architecture", "vocab", "width", "norm", "layers"}
        if set(c) - known:
            raise ValueError(f"unknown settings: {sorted(set(c) - known)}")
        if set(c["norm"]) != {"eps"}:
            raise ValueError(f"unknown norm settings: {sorted(c['norm'])}")
        for l in c["layers"]:
            if set(l) != {"type", "mixer", "mlp"}:
                raise ValueError(f"bad layer settings: {sorted(l)}")
            if l["type"] not in MIXERS:
                raise ValueError(f"unknown mixer {l['type']}")
        return cls(c["architecture"], int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), tuple(c["layers"]))


class _Layer:
    """norm1 -> mixer -> ls1, norm2 -> feed-forward -> ls2 (the latter pair only if there is one)."""

    def __init__(self, spec: dict, p: Parameters, seq: SequenceState, cfg: MixerModelConfig):
        W = cfg.hidden_size
        self.norm1, self.ls1 = p.vector("norm1"), p.vector("ls1", W)
        self.mixer = MIXERS[spec["type"]](spec["mixer"], p.under("mix"), seq, W, cfg.eps)
        self.mlp: Optional[GatedMLP] = None
        if spec["mlp"] is not None:
            self.norm2, self.ls2 = p.vector("norm2"), p.vector("ls2", W)
            self.mlp = GatedMLP(spec["mlp"], p.under("mlp"), W)


class MixerDecodeEngine(DecodeLoop):
    """Weights, sequence state and step graph of a mixer model on one GPU. ``dtype`` bfloat16 or float32 is the
    storage type of weights, caches and GEMM operands; float32 runs everything in true 32-bit."""

    dtypes = (torch.bfloat16, torch.float32)

    def __init__(self, cfg: MixerModelConfig, tensors: dict, device, max_seq_len: int = 4096,
                 dtype: torch.dtype = torch.bfloat16, max_chunk: int = 4096):
        if dtype not in self.dtypes:
            raise ValueError(f"dtype must be one of {self.dtypes}")
        self.cfg, self.dev, self.dtype = cfg, torch.device(device), dtype
        self.lib = _native.mixers()
        self._init_loop(max_seq_len)
        self.max_chunk = max(1, min(max_chunk, max_seq_len))
        self.seq = SequenceState(self.dev, dtype, max_seq_len, self.max_chunk)
        bag = TensorBag(tensors)
        p = Parameters(bag, "", self.dev, dtype)
        W, V = cfg.hidden_size, cfg.vocab_size
        self.embed = p.matrix("embed", V, W).contiguous()
        self.head = p.matrix("head", V, W).contiguous()
        self.final_norm = p.vector("final.norm")
        self.layers = [_Layer(s, p.under(f"l{i}"), self.seq, cfg) for i, s in enumerate(cfg.layers)]
        bag.finish()

        f32 = lambda n: torch.zeros(n, dtype=torch.float32, device=self.dev)
        self.x, self.logits = f32(W), f32(V)
        self._y = f32(max(l.mixer.in_width for l in self.layers))
        self._out = f32(max(l.mixer.out_width for l in self.layers))
        self._act = f32(max([l.mlp.inter for l in self.layers if l.mlp] + [1]))
        for l in self.layers:
            l.mixer.prepare_step(l.norm1, cfg.eps, self.x, l.ls1, self._y, self._out, self.state, max_seq_len)
            if l.mlp:
                l.mlp.prepare_step(l.norm2, cfg.eps, self.x, l.ls2, self._act)
        self._head_args = _native.DenseGemv(w=self.head.data_ptr(), x=self.x.data_ptr(), y=self.logits.data_ptr(),
                                            dtype=dtype_code(dtype), rows=V, cols=W, gain=self.final_norm.data_ptr(),
                                            eps=cfg.eps)
        self._scratch_buf = torch.zeros(0, dtype=torch.uint8, device=self.dev)
        self.pos = self._parity = 0          # host mirror of the state words
        self.stream_probe = None             # tests: called with the fp32 stream after every layer of a portion

    @classmethod
    def random_tensors(cls, cfg: MixerModelConfig, device, seed: int = 0, rank: int = 64) -> dict:
        """Random checkpoint tensors of this configuration (bf16), drawn on ``device``."""
        gen = torch.Generator(device=device).manual_seed(seed)
        W, V, t = cfg.hidden_size, cfg.vocab_size, {}

        def draw(name, *shape, std=0.02, mean=0.0):
            t[name] = (torch.randn(shape, generator=gen, device=device) * std + mean).bfloat16()

        draw("embed", V, W, std=1.0)
        draw("head", V, W)
        draw("final.norm", std=0.0, mean=1.0)
        for i, spec in enumerate(cfg.layers):
            p, left, right = f"l{i}.", spec["mixer"]["left"], spec["mixer"]["right"]
            q, k, v = left["heads"] * left["dim"], left["kv_heads"] * left["dim"], left["kv_heads"] * left["vdim"]
            N = right["heads"] * right["dim"]
            draw(p + "norm1", std=0.0, mean=1.0)
            for n, rows in (("q", q), ("k", k), ("v", v)):
                draw(f"{p}mix.left.{n}", rows, W)
                draw(f"{p}mix.left.{n}.b", rows)
            draw(p + "mix.left.q.norm", q, std=0.1, mean=1.0)
            draw(p + "mix.left.k.norm", k, std=0.1, mean=1.0)
            draw(p + "mix.left.talk", left["heads"], left["heads"], std=left["heads"] ** -0.5)
            draw(p + "mix.left.o", W, left["heads"] * left["vdim"])
            for s in "rkvgw":
                draw(f"{p}mix.right.mu.{s}", W, std=0.2, mean=0.5)
            for s in "rkvg":
                draw(f"{p}mix.right.{s}", N, W)
            draw(p + "mix.right.w1", rank, W)
            draw(p + "mix.right.w2", N, rank, std=rank ** -0.5)
            draw(p + "mix.right.w0", N, std=1.0, mean=-3.0)
            draw(p + "mix.right.u", right["heads"], right["dim"], std=0.3)
            draw(p + "mix.right.norm", N, std=0.1, mean=1.0)
            draw(p + "mix.right.o", W, N)
            draw(p + "ls1", W, std=0.1, mean=1.0)
            if spec["mlp"] is not None:
                ff = spec["mlp"]["ff"]
                draw(p + "norm2", std=0.0, mean=1.0)
                draw(p + "mlp.gate", ff, W)
                draw(p + "mlp.up", ff, W)
                draw(p + "mlp.down", W, ff)
                draw(p + "ls2", W, std=0.1, mean=1.0)
        return t

    # ── decode step ──────────────────────────────────────────────────────

    def _step_state(self) -> list:
        return [self.state, self.token, self.history, *self.seq.carried_tensors]

    def _step_launches(self) -> None:
        lib, st, V = self.lib, self._st(), self.cfg.vocab_size
        _native.check(lib.leankv_embed_begin(self.embed.data_ptr(), dtype_code(self.dtype), self.token.data_ptr(),
                                             self.x.data_ptr(), self.cfg.hidden_size, V, self.state.data_ptr(), st),
                      "embed_begin", lib)
        n = 1
        for l in self.layers:
            n += l.mixer.step(st)
            if l.mlp:
                n += l.mlp.step(st)
        _native.check(lib.leankv_dense_gemv(ctypes.byref(self._head_args), st), "output head", lib)
        _native.check(lib.leankv_greedy_end(self.logits.data_ptr(), V, self.token.data_ptr(), self.history.data_ptr(),
                                            self.history_cap, self.state.data_ptr(), st), "greedy_end", lib)
        self.launches_per_step = n + 2

    def step(self, use_graph: bool = True) -> None:
        """One token: ``self.token`` at position ``self.pos`` -> ``self.logits``, the next greedy token."""
        if self.pos >= self.max_seq_len:
            raise RuntimeError("sequence is full")
        super().step(use_graph)
        self.pos += 1
        self._parity ^= 1

    # ── portions of a prompt ─────────────────────────────────────────────

    def _scratch(self, nbytes: int) -> torch.Tensor:
        """Workspace shared by the launches of a portion (they follow one another on one stream)."""
        if self._scratch_buf.numel() < nbytes:
            self._scratch_buf = torch.empty(nbytes, dtype=torch.uint8, device=self.dev)
        return self._scratch_buf

    def _stream_norm(self, x, gain, h=None, delta=None, scale=None, mixer=None, mixed=None):
        """x (+ scale * delta) -> normed h, shifted mixes for ``mixer``; returns the updated stream."""
        T, W = x.shape
        x_out = torch.empty_like(x) if delta is not None else x
        a = _native.StreamNorm(x_in=x.data_ptr(), x_out=x_out.data_ptr() if delta is not None else None,
                               delta=_native.ptr(delta), scale=_native.ptr(scale), gain=gain.data_ptr(),
                               h=_native.ptr(h), mixed=_native.ptr(mixed), dtype=dtype_code(self.dtype),
                               delta_dtype=_native.DT_F32, rows=T, width=W, eps=self.cfg.eps)
        if mixer is not None:
            a.n_mix = mixer.mu.shape[0]
            for i in range(a.n_mix):
                a.mu[i] = mixer.mu[i].data_ptr()
            a.prev_in = mixer.prev[self._parity].data_ptr()
            a.prev_out = mixer.prev[self._parity ^ 1].data_ptr()
        _native.check(self.lib.leankv_stream_norm(ctypes.byref(a), self._st()), "stream_norm", self.lib)
        return x_out

    def _portion(self, ids: torch.Tensor) -> torch.Tensor:
        """Run the tokens ``ids`` at the current position; returns the fp32 stream [T][width] after the last layer."""
        T, W, dev = ids.numel(), self.cfg.hidden_size, self.dev
        x = self.embed[ids].float()
        h = torch.empty(T, W, dtype=self.dtype, device=dev)
        delta = scale = None
        for l in self.layers:
            mixed = torch.empty(l.mixer.mu.shape[0], T, W, dtype=self.dtype, device=dev)
            x = self._stream_norm(x, l.norm1, h, delta, scale, l.mixer, mixed)
            if self.stream_probe is not None and delta is not None:
                self.stream_probe(x)
            delta, scale = l.mixer.portion(h, mixed, self.pos, self._scratch), l.ls1
            if l.mlp:
                x = self._stream_norm(x, l.norm2, h, delta, scale)
                delta, scale = l.mlp.portion(h), l.ls2
        x = torch.addcmul(x, delta, scale)
        if self.stream_probe is not None:
            self.stream_probe(x)
        self.pos += T
        self._parity ^= 1
        self.state[0] = self.pos
        self.state[_native.STATE_PARITY] = self._parity
        return x

    def _logits_of(self, x: torch.Tensor) -> torch.Tensor:
        h = torch.empty(x.shape, dtype=self.dtype, device=self.dev)
        self._stream_norm(x, self.final_norm, h)
        return matmul(h, self.head)

    # ── sequences ────────────────────────────────────────────────────────

    def reset(self) -> None:
        """Give back what the current sequence holds; the next token starts a new one at position 0."""
        self.seq.reset()
        self.state.zero_()
        self.history.zero_()
        self.pos = self._parity = 0

    @torch.no_grad()
    def extend(self, tokens: Sequence[int], want: Sequence[int] = ()) -> torch.Tensor:
        """Feed the sequence's next tokens (any number) and return the fp32 logits [len(want)][vocab] at the
        places ``want`` among them. One token is one decode step; more are a portion of a prompt."""
        n = len(tokens)
        if n < 1 or self.pos + n > self.max_seq_len:
            raise ValueError(f"{n} tokens at position {self.pos} do not fit {self.max_seq_len}")
        if min(tokens) < 0 or max(tokens) >= self.cfg.vocab_size:
            raise ValueError("token outside the vocabulary")
        if any(not 0 <= w < n for w in want):
            raise ValueError("wanted place outside the portion")
        out = torch.empty(len(want), self.cfg.vocab_size, dtype=torch.float32, device=self.dev)
        with torch.cuda.device(self.dev):
            if n == 1:
                self.token.fill_(int(tokens[0]))
                self.step()
                if len(want):
                    out[:] = self.logits
                return out
            ids = torch.as_tensor(list(tokens), dtype=torch.int64, device=self.dev)
            for s0 in range(0, n, self.max_chunk):
                x = self._portion(ids[s0:s0 + self.max_chunk])
                rows = [k for k, w in enumerate(want) if s0 <= w < s0 + x.shape[0]]
                if rows:
                    at = torch.tensor([want[k] - s0 for k in rows], device=self.dev)
                    out[torch.tensor(rows, device=self.dev)] = self._logits_of(x[at])
        return out

    @torch.no_grad()
    def prefill(self, prompt_ids, chunk: Optional[int] = None) -> int:
        """Start a new sequence with this prompt and leave the first generated token ready for ``step``.
        ``chunk``: tokens per pass (default: as many as the engine's portions hold)."""
        ids = [int(t) for t in torch.as_tensor(prompt_ids).reshape(-1).tolist()]
        T = len(ids)
        if T < 1 or T >= self.max_seq_len:
            raise ValueError("prompt length must be in [1, max_seq_len)")
        if chunk is not None and chunk < 1:
            raise ValueError("chunk must be positive")
        self.reset()
        for s0 in range(0, T, chunk or T):
            part = ids[s0:s0 + (chunk or T)]
            logits = self.extend(part, [len(part) - 1] if s0 + len(part) == T else [])
        with torch.cuda.device(self.dev):
            self.prefill_logits = logits[0]
            tok = torch.argmax(logits[0]).reshape(1)
            self.token.copy_(tok)
            self.history.zero_()
            self.history[0] = tok[0]
            self.state[1] = 1
        return int(tok.item())
