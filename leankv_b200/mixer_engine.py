"""Decode engine of models whose layers are pre-norm token mixers and feed-forwards (``mixers.py``) on one
residual stream in fp32. What differs between the designs it serves is in ``DESIGNS``: one norm gain or one per
channel, branches that join the stream scaled per channel or normed again, a head of its own or the embedding
table. A range of layers may run several times; every run of a layer has its own state.

Prompts run in portions of any size (library GEMMs between the row kernels); a single token runs as one
replay of the captured step graph. There the norm, and where branches are normed the end of the branch before
it, is part of a branch's first GEMV: {norm, every input projection}, {mixers}, {output projection, residual},
{norm, gate / up, silu}, {down, residual}.
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
class Design:
    mixers: tuple                   # layer types
    gain_per_channel: bool          # norm gains are vectors, else one number
    normed_branches: bool           # x += residual_mult * norm(branch), else x += per-channel scale * branch
    tied_head: bool                 # logits from the embedding table
    settings: tuple = ()            # top-level settings beyond the common ones


DESIGNS = {
    "Rorosun": Design(("parallel",), gain_per_channel=False, normed_branches=False, tied_head=False),
    "Pefitar": Design(("attention", "latent_attention"), gain_per_channel=True, normed_branches=True, tied_head=True,
                      settings=("loop", "residual_mult", "logit_softcap")),
}


@dataclass(frozen=True)
class MixerModelConfig:
    """Sizes and constants of a mixer model, as its ``config.json`` gives them."""

    architecture: str
    vocab_size: int
    hidden_size: int
    eps: float
    layers: tuple                          # per layer: {"type", "mixer": {...}, "mlp": {...} or None}
    loop: tuple = (0, 0, 1)                # layers start .. stop - 1 run `times` times in a row
    residual_mult: float = 1.0
    logit_softcap: float = 0.0             # 0: none

    @property
    def design(self) -> Design:
        return DESIGNS[self.architecture]

    @property
    def order(self) -> list[int]:
        """Layer numbers in the order they run."""
        start, stop, times = self.loop
        return [*range(start), *list(range(start, stop)) * times, *range(stop, len(self.layers))]

    @classmethod
    def from_dict(cls, c: dict) -> "MixerModelConfig":
        design = DESIGNS[c["architecture"]]
        known = {"architecture", "vocab", "width", "norm", "layers", *design.settings}
        if set(c) - known:
            raise ValueError(f"unknown settings: {sorted(set(c) - known)}")
        if set(c["norm"]) != {"eps"}:
            raise ValueError(f"unknown norm settings: {sorted(c['norm'])}")
        for l in c["layers"]:
            if set(l) != {"type", "mixer", "mlp"}:
                raise ValueError(f"bad layer settings: {sorted(l)}")
            if l["type"] not in design.mixers:
                raise ValueError(f"unknown mixer {l['type']}")
        loop = c.get("loop") or {"start": 0, "stop": 0, "times": 1}
        if set(loop) != {"start", "stop", "times"}:
            raise ValueError(f"bad loop settings: {sorted(loop)}")
        start, stop, times = (int(loop[n]) for n in ("start", "stop", "times"))
        if not 0 <= start <= stop <= len(c["layers"]) or times < 1:
            raise ValueError(f"loop {loop} does not fit {len(c['layers'])} layers")
        mult, cap = c.get("residual_mult"), c.get("logit_softcap")
        return cls(c["architecture"], int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), tuple(c["layers"]),
                   (start, stop, times), 1.0 if mult is None else float(mult), float(cap or 0.0))


class _Sublayer:
    """norm -> mixer or feed-forward -> join with the stream: the weights of one, whatever runs it how often."""

    def __init__(self, body, p: Parameters, number: int, cfg: MixerModelConfig):
        W, d = cfg.hidden_size, cfg.design
        self.body = body
        self.norm = p.vector(f"norm{number}", *((W,) if d.gain_per_channel else ()))
        self.after = p.vector(f"norm{number}b", W) if d.normed_branches else None
        self.scale = None if d.normed_branches else p.vector(f"ls{number}", W)

    def bind(self, seq: SequenceState) -> "_Sublayer":
        bound = object.__new__(_Sublayer)
        bound.__dict__.update(self.__dict__, body=self.body.bind(seq))
        return bound


class _Run:
    """One run of a layer: its sublayers bound to the state of this run."""

    def __init__(self, layer: list, seq: SequenceState):
        bound = [s.bind(seq) for s in layer]
        self.first, self.second = bound[0], bound[1] if len(bound) > 1 else None
        self.mixer, self.mlp = self.first.body, self.second.body if self.second else None


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
        self.head = self.embed if cfg.design.tied_head else p.matrix("head", V, W).contiguous()
        self.final_norm = p.vector("final.norm", *((W,) if cfg.design.gain_per_channel else ()))
        weights = [self._load_layer(s, p.under(f"l{i}")) for i, s in enumerate(cfg.layers)]
        self.layers = [_Run(weights[i], self.seq) for i in cfg.order]
        bag.finish()
        self._prepare_steps()
        self._scratch_buf = torch.zeros(0, dtype=torch.uint8, device=self.dev)
        self.pos = self._parity = 0          # host mirror of the state words
        self.stream_probe = None             # tests: called with the fp32 stream after every layer of a portion

    def _load_layer(self, spec: dict, p: Parameters) -> list[_Sublayer]:
        W = self.cfg.hidden_size
        layer = [_Sublayer(MIXERS[spec["type"]](spec["mixer"], p.under("mix"), W, self.cfg.eps), p, 1, self.cfg)]
        if spec["mlp"] is not None:
            layer.append(_Sublayer(GatedMLP(spec["mlp"], p.under("mlp"), W), p, 2, self.cfg))
        return layer

    def _prepare_steps(self) -> None:
        """Argument blocks of the decode step on fixed buffers. A branch that is normed before it joins the stream goes
        to a buffer of its own, and the next branch's first GEMV adds it: two streams, written in turn."""
        cfg, W, V = self.cfg, self.cfg.hidden_size, self.cfg.vocab_size
        f32 = lambda n: torch.zeros(n, dtype=torch.float32, device=self.dev)
        self.x, self.logits = f32(W), f32(V)
        self._streams, self._branch = (self.x, f32(W)), f32(W)
        streams = self._streams
        sizes: dict[str, int] = {}
        for run in self.layers:
            for body in (run.mixer, run.mlp):
                for name, n in (body.step_floats if body else {}).items():
                    sizes[name] = max(n, sizes.get(name, 0))
        self._bufs = {name: f32(n) for name, n in sizes.items()}
        at, pending = 0, None

        def entry(norm: torch.Tensor) -> dict:
            nonlocal at, pending
            d = dict(x=streams[at].data_ptr(), gain=norm.data_ptr(), gain_per_col=int(norm.dim() > 0), eps=cfg.eps)
            if pending is not None:
                at ^= 1
                d.update(delta=self._branch.data_ptr(), post_gain=pending.data_ptr(), post_mult=cfg.residual_mult,
                         x_out=streams[at].data_ptr())
                pending = None
            return d

        for run in self.layers:
            for sub in (run.first, run.second):
                if sub is None:
                    continue
                into = entry(sub.norm)
                x = streams[at].data_ptr()
                if sub.after is not None:
                    out, pending = dict(y=self._branch.data_ptr()), sub.after
                else:
                    out = dict(y=x, scale=sub.scale.data_ptr(), residual=x)
                if sub is run.first:
                    sub.body.prepare_step(into, out, self._bufs, self.state, self.max_seq_len)
                else:
                    sub.body.prepare_step(into, out, self._bufs)
        self._head_args = _native.DenseGemv(w=self.head.data_ptr(), y=self.logits.data_ptr(), dtype=dtype_code(self.dtype),
                                            rows=V, cols=W, softcap=cfg.logit_softcap, **entry(self.final_norm))

    @classmethod
    def random_tensors(cls, cfg: MixerModelConfig, device, seed: int = 0, rank: int = 64) -> dict:
        """Random checkpoint tensors of this configuration (bf16), drawn on ``device``."""
        gen = torch.Generator(device=device).manual_seed(seed)
        W, V, t = cfg.hidden_size, cfg.vocab_size, {}

        def draw(name, *shape, std=0.02, mean=0.0):
            t[name] = (torch.randn(shape, generator=gen, device=device) * std + mean).bfloat16()

        ones = lambda name, *shape: draw(name, *shape, std=0.0 if not shape else 0.1, mean=1.0)
        per_channel = (W,) if cfg.design.gain_per_channel else ()

        def parallel(p, mixer):
            left, right = mixer["left"], mixer["right"]
            q, k, v = left["heads"] * left["dim"], left["kv_heads"] * left["dim"], left["kv_heads"] * left["vdim"]
            N = right["heads"] * right["dim"]
            for n, rows in (("q", q), ("k", k), ("v", v)):
                draw(f"{p}left.{n}", rows, W)
                draw(f"{p}left.{n}.b", rows)
            ones(p + "left.q.norm", q)
            ones(p + "left.k.norm", k)
            draw(p + "left.talk", left["heads"], left["heads"], std=left["heads"] ** -0.5)
            draw(p + "left.o", W, left["heads"] * left["vdim"])
            for s in "rkvgw":
                draw(f"{p}right.mu.{s}", W, std=0.2, mean=0.5)
            for s in "rkvg":
                draw(f"{p}right.{s}", N, W)
            draw(p + "right.w1", rank, W)
            draw(p + "right.w2", N, rank, std=rank ** -0.5)
            draw(p + "right.w0", N, std=1.0, mean=-3.0)
            draw(p + "right.u", right["heads"], right["dim"], std=0.3)
            ones(p + "right.norm", N)
            draw(p + "right.o", W, N)

        def attention(p, m):
            H, G = m["heads"], m["kv_heads"]
            for n, rows in (("q", H * m["dim"]), ("k", G * m["dim"]), ("v", G * m["vdim"]), ("g", H * m["vdim"])):
                draw(p + n, rows, W)
            draw(p + "o", W, H * m["vdim"])

        def latent_attention(p, m):
            H = m["heads"]
            draw(p + "dq", m["q_rank"], W)
            ones(p + "dq.norm", m["q_rank"])
            draw(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            draw(p + "dkv", m["kv_rank"] + m["rot_dim"], W)
            ones(p + "dkv.norm", m["kv_rank"])
            draw(p + "uk", H * m["dim"], m["kv_rank"])
            draw(p + "uv", H * m["vdim"], m["kv_rank"])
            draw(p + "o", W, H * m["vdim"])

        mixers = {"parallel": parallel, "attention": attention, "latent_attention": latent_attention}
        draw("embed", V, W, std=1.0)
        if not cfg.design.tied_head:
            draw("head", V, W)
        ones("final.norm", *per_channel)
        for i, spec in enumerate(cfg.layers):
            p, ff = f"l{i}.", spec["mlp"]["ff"] if spec["mlp"] is not None else 0
            mixers[spec["type"]](p + "mix.", spec["mixer"])
            for s in (1, 2) if ff else (1,):
                ones(f"{p}norm{s}", *per_channel)
                ones(f"{p}norm{s}b" if cfg.design.normed_branches else f"{p}ls{s}", W)
            if ff:
                draw(p + "mlp.gate", ff, W)
                draw(p + "mlp.up", ff, W)
                draw(p + "mlp.down", W, ff)
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

    def _stream_norm(self, x, gain, h=None, delta=None, join=None, mixer=None, mixed=None):
        """x (+ the branch ``delta`` as the sublayer ``join`` adds it) -> normed h, shifted mixes for ``mixer``;
        returns the updated stream. Without ``gain`` only the sum."""
        T, W = x.shape
        x_out = torch.empty_like(x) if delta is not None else x
        a = _native.StreamNorm(x_in=x.data_ptr(), x_out=x_out.data_ptr() if delta is not None else None,
                               delta=_native.ptr(delta), gain=_native.ptr(gain),
                               gain_per_col=int(gain is not None and gain.dim() > 0),
                               h=_native.ptr(h), mixed=_native.ptr(mixed), dtype=dtype_code(self.dtype),
                               delta_dtype=_native.DT_F32, rows=T, width=W, eps=self.cfg.eps)
        if delta is not None and join.after is not None:
            a.post_gain, a.post_mult = join.after.data_ptr(), self.cfg.residual_mult
        elif delta is not None:
            a.scale = join.scale.data_ptr()
        if mixed is not None:
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
        delta = join = None
        for l in self.layers:
            mu = getattr(l.mixer, "mu", None)          # token shift
            mixed = torch.empty(mu.shape[0], T, W, dtype=self.dtype, device=dev) if mu is not None else None
            x = self._stream_norm(x, l.first.norm, h, delta, join, l.mixer, mixed)
            if self.stream_probe is not None and delta is not None:
                self.stream_probe(x)
            delta, join = l.mixer.portion(h, mixed, self.pos, self._scratch), l.first
            if l.second:
                x = self._stream_norm(x, l.second.norm, h, delta, join)
                delta, join = l.mlp.portion(h), l.second
        x = self._stream_norm(x, None, None, delta, join)
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
        z = matmul(h, self.head)
        if self.cfg.logit_softcap > 0:
            _native.check(self.lib.leankv_softcap(z.data_ptr(), z.numel(), self.cfg.logit_softcap, self._st()), "softcap",
                          self.lib)
        return z

    # ── kernel status ────────────────────────────────────────────────────

    def check_status(self) -> None:
        """Raise if a wait inside an attention kernel ran out (its results are not to be used)."""
        if int(self.seq.status.item()):
            raise RuntimeError("an attention kernel gave up waiting for its copies")

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
            if len(want):
                self.check_status()
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
