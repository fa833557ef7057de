"""What every engine offers the sessions and the serving backend: launches with their instrumentation, graph rehearsal, the
prompt driver and the defaults of optional capabilities.

An engine runs passes over "rows" (one token each): `set_rows` describes them (token, position, slot), `forward_rows` runs
them, `chosen` / `logits_rows` hold the result.  Rows of one slot are adjacent and in order.
"""
from __future__ import annotations

import contextlib
from typing import List, Optional

import torch

from ..ops import lib


class RowsEngine:
    partial_prefix = True      # can a prompt continue a snapshot that only shares a leading part with it?

    def _init_instruments(self):
        import os
        from ..utils.trace import ActivationTrace
        self.launches = 0
        self.only = None          # a set of tags restricts a pass to some kernels for profiling
        self.layer_timer = None   # utils.trace.LayerTimer: device time per layer of eager passes
        # DS41_NVTX=1: every launch sits in an NVTX range named after its kernel class (for timeline tools)
        self.nvtx = os.environ.get("DS41_NVTX", "") == "1"
        self.activation_trace = ActivationTrace.from_env()
        self.timeline = None      # set to a list to record (tag, start event, end event) per launch of eager passes

    def _run(self, tag, fn, *args, **kw):
        """Launch one kernel; `self.only` (a set of tags) restricts a pass to some kernels for profiling."""
        if self.only is not None and tag not in self.only:
            return
        self.launches += 1
        if self.nvtx:
            torch.cuda.nvtx.range_push(tag)
            try:
                err = fn(*args, **kw)
            finally:
                torch.cuda.nvtx.range_pop()
            if err is not None:
                lib.check(err, tag)
            return
        if self.timeline is not None:           # eager passes only: a CUDA event pair around every launch
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            err = fn(*args, **kw)
            e1.record()
            self.timeline.append((tag, e0, e1))
        else:
            err = fn(*args, **kw)
        if err is not None:
            lib.check(err, tag)

    # ------------------------------------------------------------------ capabilities with a default
    @property
    def replay_window(self) -> int:
        """Tokens to run again before the cut when a prompt continues a truncated snapshot."""
        return self.cfg.window

    def ced_usable(self, start: int, n_new: int) -> bool:
        return False

    def sp_rows(self, n: int) -> int:
        return n

    # ------------------------------------------------------------------ graphs
    @contextlib.contextmanager
    def rehearsal(self):
        """Around the eager pass and the capture that precede a graph's first replay: the pass inputs come back
        unchanged, and nothing the pass does may count as a step of a request."""
        keep = (self.in_tokens.clone(), self.row_pos.clone(), self.row_slot.clone())
        self._enter_rehearsal()
        try:
            yield
        finally:
            self.in_tokens.copy_(keep[0])
            self.row_pos.copy_(keep[1])
            self.row_slot.copy_(keep[2])

    def _enter_rehearsal(self):
        pass

    def capture(self, enqueue) -> torch.cuda.CUDAGraph:
        """Graph of the launches that `enqueue` makes; one eager pass first sets function attributes and warms every
        code path."""
        with self.rehearsal():
            enqueue()
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g):
                enqueue()
        return g

    # ------------------------------------------------------------------ drivers
    def prefill(self, slot: int, tokens: List[int], start: int = 0, chunk: Optional[int] = None) -> int:
        """Run the prompt through the engine in chunks of up to max_rows rows; returns the greedy next token."""
        chunk = chunk or self.max_rows
        assert self.cache.ensure(slot, start + len(tokens) + 1)
        nxt = -1
        for c0 in range(0, len(tokens), chunk):
            part = tokens[c0:c0 + chunk]
            pos = list(range(start + c0, start + c0 + len(part)))
            self.set_rows(part, pos, [slot] * len(part))
            last = c0 + chunk >= len(tokens)
            # a chunk may run padded up to the row-sharded granularity (the padding rows have no slot)
            self.forward_rows(self.sp_rows(len(part)), head=last, head_row=len(part) - 1)
            if last:
                nxt = int(self.chosen[self.last_head_row].item())
        return nxt

    def check_status(self, what: str = "engine pass"):
        lib.raise_on_status(self.status, what)
