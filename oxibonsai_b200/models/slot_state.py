"""Per-slot device state every step runner keeps: what a captured decode step reads and writes.

The tensors never move, so a decode step captured into a CUDA graph stays valid: the last token and position of every slot,
its block-table row, its sampler settings and vocabulary mask, and the status word in which a kernel records an expired wait.
"""
from __future__ import annotations

import torch

from ..ops import cuda_ops as K


class SlotState:
    def init_slots(self, max_batch: int, max_pages: int, vocab: int, device) -> None:
        B = max_batch
        f32, i32 = dict(dtype=torch.float32, device=device), dict(dtype=torch.int32, device=device)
        # [status word, token of slot 0, token of slot 1, ...]: one device-to-host copy brings the sampled tokens and the
        # word in which a kernel records an expired bounded wait (copy pipeline, tensor-parallel peer)
        self.ctl = torch.zeros(B + 1, **i32)
        self.status = self.ctl[:1]
        self.tokens = self.ctl[1:]
        self.positions = torch.zeros(B, **i32)
        self.block_table = torch.zeros((B, max_pages), **i32)
        self.temps = torch.zeros(B, **f32)
        self.topks = torch.zeros(B, **i32)
        self.topps = torch.ones(B, **f32)
        self.rng = torch.full((B,), 42, dtype=torch.int64, device=device)
        # per-slot vocabulary masks of constrained decoding (bit set = token allowed), read by the sampler of a masked step
        self.mask_words = (vocab + 31) // 32
        self.allow_mask = torch.full((B, self.mask_words), -1, **i32)

    STATUS_TEXT = {1: "a tile pipeline of the tensor-core GEMM stalled", 2: "a tensor-parallel peer did not deliver its partial sums",
                   3: "a tensor-parallel peer did not reach a barrier", 4: "a tensor-parallel peer did not enter an all-reduce",
                   5: "the weight copy pipeline of a GEMV stalled"}

    def check_status(self, value: int | None = None) -> None:
        """Raises when a kernel of an earlier step recorded an expired wait (``value``: the status word as already read by
        the caller, else it is read here)."""
        v = int(self.status.item()) if value is None else int(value)
        if v:
            self.status.zero_()
            raise K.CudaKernelError(f"decode step reported status {v}: {self.STATUS_TEXT.get(v, 'a bounded wait expired')}")

    def sample_rows(self, lo: int, hi: int, masked: bool = False, advance: bool = False) -> None:
        """Samples the next tokens of slots lo .. hi-1 from ``logits`` into ``tokens`` (and advances their positions)."""
        s = slice(lo, hi)
        self.sample_fn(self.logits[s], self.temps[s], self.topks[s], self.topps[s], self.rng[s], positions=self.positions[s] if advance else None,
                       advance=advance, allow_mask=self.allow_mask[s] if masked else None, out=self.tokens[s])

    sample_fn = staticmethod(K.sample)

    # sequences of models with recurrent state also own a state row; the others have nothing to do here
    def bind_state(self, slot: int) -> None:
        pass

    def release_state(self, slot: int) -> None:
        pass

    def move_state(self, src: int, dst: int) -> None:
        pass
