"""The greedy decode loop every engine shares: one decode step captured in a CUDA graph and replayed per
token, with tokens (and kernel status words) streamed to pinned host memory.

An engine supplies ``prefill`` (fills its cache / state and leaves the first generated token in
``self.token``), ``_step_launches`` (the kernels of one step, which consume ``self.token`` at the position
its device state words hold and leave the next token there) and ``_step_state`` (what a step changes).
"""

from __future__ import annotations

from typing import Optional

import torch


class DecodeLoop:
    dev: torch.device
    max_seq_len: int
    token: torch.Tensor            # int64 [1]
    history: torch.Tensor          # int64 [history_cap]
    graph: Optional[torch.cuda.CUDAGraph] = None
    launches_per_step: int = 0

    def _init_loop(self, max_seq_len: int) -> None:
        """Token, history and state words of a single-sequence loop, and the pinned words it streams into."""
        self.max_seq_len = max_seq_len
        self.token = torch.zeros(1, dtype=torch.int64, device=self.dev)
        self.history_cap = max_seq_len + 8
        self.history = torch.zeros(self.history_cap, dtype=torch.int64, device=self.dev)
        self.state = torch.zeros(8, dtype=torch.int32, device=self.dev)
        pin = torch.cuda.is_available()
        self._pinned_token = torch.zeros(1, dtype=torch.int64).pin_memory() if pin else None
        self._pinned_status = torch.zeros(2, dtype=torch.int32).pin_memory() if pin else None
        self.graph = None
        self.launches_per_step = 0

    # ── what an engine supplies ──────────────────────────────────────────

    def _step_launches(self) -> None:
        raise NotImplementedError

    def _step_state(self) -> list:
        """Tensors that one step changes (restored after the throw-away step of ``capture``)."""
        raise NotImplementedError

    def prefill(self, prompt_ids, **kw) -> int:
        raise NotImplementedError

    def _queue_status(self) -> None:
        """Queue copies of the kernels' status words into ``_pinned_status`` (none by default)."""

    def check_status(self) -> None:
        """Raise if a kernel of this engine has reported a failure."""

    def _capture_barrier(self) -> None:
        """Called once the graph exists (ranks that exchange inside a step start their replays together)."""

    # ── the loop ─────────────────────────────────────────────────────────

    def _st(self) -> int:
        return torch.cuda.current_stream().cuda_stream

    def capture(self) -> None:
        """Capture one decode step into a CUDA graph (a throw-away eager step warms everything up first)."""
        with torch.cuda.device(self.dev):
            live = self._step_state()
            snap = [t.clone() for t in live]
            side = torch.cuda.Stream()
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):
                self._step_launches()
            torch.cuda.current_stream().wait_stream(side)
            torch.cuda.synchronize()
            for t, s in zip(live, snap):
                t.copy_(s)
            self.graph = torch.cuda.CUDAGraph()
            # thread_local: the NCCL watchdog thread (tensor parallel runs) may touch CUDA while we capture
            with torch.cuda.graph(self.graph, capture_error_mode="thread_local"):
                self._step_launches()
            # capture does not execute; state is unchanged
            self._capture_barrier()

    def step(self, use_graph: bool = True) -> None:
        if use_graph:
            if self.graph is None:
                self.capture()
            self.graph.replay()
        else:
            with torch.cuda.device(self.dev):
                self._step_launches()

    @torch.no_grad()
    def generate(self, prompt_ids, max_new_tokens: int, stream_to_host: bool = True) -> list[int]:
        """Greedy generation. With ``stream_to_host`` every token is copied to pinned host memory and
        waited for before the next step is launched (what an interactive caller sees); without it the
        steps are enqueued back to back and the tokens are read once at the end."""
        first = self.prefill(prompt_ids)
        n_steps = min(max_new_tokens - 1, self.max_seq_len - len(prompt_ids) - 1)
        out = [first]
        with torch.cuda.device(self.dev):
            if self.graph is None:
                self.capture()
            for _ in range(max(n_steps, 0)):
                self.step()
                if stream_to_host:
                    self._pinned_token.copy_(self.token, non_blocking=True)
                    self._queue_status()
                    torch.cuda.current_stream().synchronize()
                    if int(self._pinned_status[0]) or int(self._pinned_status[1]):
                        self.check_status()
                    out.append(int(self._pinned_token[0]))
            if not stream_to_host:
                out = self.history[:1 + max(n_steps, 0)].tolist()
            self.check_status()
        return out
