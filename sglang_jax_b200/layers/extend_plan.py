"""Which sequences of a ragged step go through a prefill attention kernel and which token by token."""

from __future__ import annotations

from typing import NamedTuple

import numpy as np
import torch

# a sequence with at least this many new tokens takes the prefill kernel
MIN_TILE_TOKENS = 32
# query rows per CTA of the prefill kernels (`csrc/latent_extend.cu`, `csrc/window_extend.cu`)
TILE_ROWS = 256
# keys per tile of the prefill kernels
KEY_TILE = 64


class Context(NamedTuple):
    """The tokens that the long sequences of a step attend to, laid end to end: first row of each (and the end), how many of a
    sequence's tokens are left out in front (None: of none), rows in all."""
    start: torch.Tensor
    skip: torch.Tensor | None
    total: int


class ExtendPlan:
    """How the sequences of an extend step are split between an attention's two routes, as device tensors: a prefill kernel
    that works on tiles of one sequence's new tokens, and a decode kernel that takes every token as a query of its own.
    `tiles`: whether the prefill kernel can be used at all."""

    def __init__(self, fb, tiles: bool):
        n = np.asarray(fb.extend_seq_lens_cpu, np.int64)
        pre = np.asarray(fb.extend_prefix_lens_cpu, np.int64)
        start = np.concatenate([[0], np.cumsum(n)[:-1]])
        long = np.nonzero(n >= MIN_TILE_TOKENS)[0] if tiles else np.empty(0, np.int64)
        dev = fb.positions.device
        self.long = len(long)
        # every token as a query of its own: its sequence's row, and the tokens up to and including itself
        self.token_rows = torch.repeat_interleave(fb.req_pool_indices, fb.extend_seq_lens.long(), output_size=fb.num_tokens)
        self.token_lens = fb.positions + 1
        self.short_tokens = None
        if self.long:
            self._prefix, self._end, self._contexts = pre[long], (pre + n)[long], {}
            self.num_tiles = int(((n[long] + TILE_ROWS - 1) // TILE_ROWS).sum())
            rows = fb.req_pool_indices[torch.from_numpy(long).to(dev)]
            meta = torch.from_numpy(np.concatenate([start[long], n[long], pre[long]]).astype(np.int32)).to(dev)
            L = self.long
            self.q_start, self.q_len, self.prefix = meta[:L], meta[L:2 * L], meta[2 * L:]
            self.rows = rows
            if L < len(n):
                keep = np.ones(len(n), bool)
                keep[long] = False
                short = np.concatenate([np.arange(start[i], start[i] + n[i]) for i in np.nonzero(keep)[0]])
                if len(short):
                    self.short_tokens = torch.from_numpy(short).to(dev)


    def context(self, window: int = 0) -> Context:
        """What the long sequences see under a window (0: everything), from a multiple of `KEY_TILE` on."""
        if window not in self._contexts:
            skip = np.maximum(self._prefix - window + 1, 0) // KEY_TILE * KEY_TILE if window else np.zeros_like(self._prefix)
            start = np.concatenate([[0], np.cumsum(self._end - skip)])
            meta = torch.from_numpy(np.concatenate([start, skip]).astype(np.int32)).to(self.rows.device)
            self._contexts[window] = Context(meta[:len(start)], meta[len(start):] if skip.any() else None, int(start[-1]))
        return self._contexts[window]


def extend_plan(fb, tiles: bool) -> ExtendPlan:
    """The step's plan, made once per forward."""
    key = ("extend_plan", tiles)
    plan = fb.extras.get(key)
    if plan is None:
        plan = fb.extras[key] = ExtendPlan(fb, tiles)
    return plan
