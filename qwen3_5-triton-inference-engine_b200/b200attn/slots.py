"""What every engine of this package shares, whatever the architecture: sequence slots, the paged-cache bookkeeping, the
device-resident position and next-token buffers, and the captured decode step.

A subclass allocates its own caches and states (`self.num_pages` physical pages, `self.batch` slots) and implements
    _prefill(prompts, slots)  packed prefill of prompts into slots (a list, or None for all of them in order): fills the
                              caches, sets `pos` and `tok`, returns the first generated tokens;
    _decode(tok)              one token per slot with no host value that changes from step to step: returns the next
                              ids (possibly `self.tok` itself, written in place) and advances `pos` on the device.
"""
from __future__ import annotations

import torch

from . import ops


class SlotEngine:
    def __init__(self, batch: int, max_context: int, device, page_seed: int = 0, on_demand_pages: bool = False,
                 num_pages: int | None = None):
        """on_demand_pages: KV pages come from a shared pool of `num_pages` (default: enough for every slot at
        `max_context`) as sequences grow (`serving.PageAllocator`), the `batch` sequences are independent SLOTS that
        `prefill_slots` fills one group at a time, and `set_active` masks the idle ones - what `ContinuousBatcher`
        drives.  Without it every slot owns its pages from the start, as the reference reserves them
        (engine/cache.py:154-159)."""
        self.batch, self.device = batch, torch.device(device)
        pages_per_seq = (max_context + ops.PAGE_SIZE - 1) // ops.PAGE_SIZE
        self.pages = None
        self.active = None
        if on_demand_pages:
            from .serving import PageAllocator
            num_pages = batch * pages_per_seq + 1 if num_pages is None else num_pages
            self.pages = PageAllocator(num_pages, batch, pages_per_seq, device=self.device)
            self.block_table = self.pages.block_table
            self.active = torch.ones(batch, dtype=torch.int64, device=self.device)   # 1 = the slot decodes
        else:
            num_pages = batch * pages_per_seq
            perm = torch.randperm(num_pages, generator=torch.Generator().manual_seed(page_seed))
            self.block_table = perm.view(batch, pages_per_seq).to(torch.int32).to(self.device)
        self.num_pages = num_pages
        self.max_context = pages_per_seq * ops.PAGE_SIZE
        self.pos = torch.zeros(batch, dtype=torch.int64, device=self.device)
        self.tok = torch.zeros(batch, dtype=torch.int64, device=self.device)   # input of the next step
        self.argmax_ws = ops.argmax_workspace(self.device)
        self.graph = None
        self._warmed = False     # an eager decode step has run (first-call set-up of the kernels is done)

    # ------------------------------------------------------------------------------------------------------- prefill
    @torch.no_grad()
    def prefill(self, prompts: list[list[int]]) -> torch.Tensor:
        """Packed varlen prefill of `batch` prompts (engine/runner.py:212-405 with a PackedBatch); fills every cache,
        sets pos, returns the first generated token of each sequence (int64 [B]) and leaves it in `self.tok`."""
        assert len(prompts) == self.batch
        if self.pages is not None:
            for slot, prompt in enumerate(prompts):
                self.pages.release(slot)
                self.pages.ensure(slot, len(prompt) + 1)
        return self._prefill(prompts, None)

    @torch.no_grad()
    def prefill_slots(self, slots: list[int], prompts: list[list[int]]) -> torch.Tensor:
        """Packed prefill of `prompts` into the given slots only (their pages must already be there: the caller is the
        batcher, which calls `pages.ensure` first); the other slots keep their state.  Returns the first generated
        token of each prompt (int64 [len(slots)]) and leaves them in `self.tok[slots]`."""
        assert self.pages is not None, "slot-wise prefill needs on_demand_pages=True"
        assert len(slots) == len(prompts) and len(set(slots)) == len(slots)
        assert all(0 <= s < self.batch for s in slots)
        return self._prefill(prompts, list(slots))

    def set_active(self, mask) -> None:
        """Which slots decode (host list of bools).  An idle slot still rides along in the step's launches - the batch
        dimension of a captured graph is fixed - but its page table row points at the spare page and nothing it writes
        is ever read."""
        assert self.active is not None and len(mask) == self.batch
        self.active.copy_(torch.tensor([1 if m else 0 for m in mask], dtype=torch.int64), non_blocking=True)

    # -------------------------------------------------------------------------------------------------------- decode
    def capture(self) -> None:
        """Capture one decode step (read self.tok, write the next ids back into self.tok) into a CUDA graph.
        At least one eager `step()` must have run before: the first call of several kernels does per-device set-up
        (shared-memory limits, symbol addresses, workspaces) that must not happen under stream capture."""
        assert self._warmed, "run one eager step() before capture(): first calls do set-up that cannot be captured"
        side = torch.cuda.Stream(device=self.device)
        side.wait_stream(torch.cuda.current_stream(self.device))
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.stream(side):
            with torch.cuda.graph(graph, stream=side):
                self._advance()
        torch.cuda.current_stream(self.device).wait_stream(side)
        self.graph = graph

    def step(self) -> torch.Tensor:
        """Advance every sequence by one token; returns the device tensor holding the new ids (valid until the next
        step)."""
        if self.graph is not None:
            self.graph.replay()
        else:
            self._advance()
            self._warmed = True
        return self.tok

    def _advance(self) -> None:
        nxt = self._decode(self.tok)
        if nxt.data_ptr() != self.tok.data_ptr():        # a step that did not write the ids in place
            self.tok.copy_(nxt)
