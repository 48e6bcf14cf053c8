"""Per-request state of the linear-attention layers of hybrid models: the short-convolution
window and the `[H, Dk, Dv]` recurrent matrix (reference
`python/sgl_jax/srt/mem_cache/recurrent_state_pool.py:77`, `copy_slots` :230).

A slot belongs to one request (`HybridReqToTokenPool` keeps the request -> slot ledger).  Slot 0 is
a scratch slot used by padding rows.  `copy_slots` clones states (copy-on-write when a prefix with
a recurrent checkpoint is shared)."""

from __future__ import annotations

import torch


def slot_bytes(num_layers: int = 0, conv_dim: int = 0, conv_kernel: int = 1, num_heads: int = 0, head_k_dim: int = 0,
               head_v_dim: int = 0, conv_dtype=torch.bfloat16, state_dtype=torch.float32,
               layers: list[dict] | None = None) -> int:
    """Bytes one state slot takes over all linear-attention layers (what `RecurrentStatePool` allocates per slot)."""
    if layers is not None:
        return sum(slot_bytes(1, conv_dtype=conv_dtype, state_dtype=state_dtype, **d) for d in layers)
    conv = conv_dim * (conv_kernel - 1) * torch.empty((), dtype=conv_dtype).element_size()
    rec = num_heads * head_k_dim * head_v_dim * torch.empty((), dtype=state_dtype).element_size()
    return num_layers * (conv + rec)


def plan_state_slots(request_slots: int, per_slot_bytes: int, available_bytes: int, max_state_size: int | None,
                     snapshot_slots: int, memory_ratio: float, sharing: bool) -> tuple[int, int]:
    """`(snapshot slots, bytes the pool will take)` (reference `model_runner_kv_cache_mixin.py`
    `handle_recurrent_cache`, `_split_state_kv_budget`).  Priority: an explicit total (`--max-recurrent-state-size`,
    request slots included); without prefix sharing no checkpoint slots at all; an explicit
    `--recurrent-snapshot-slots >= 0`; else (`-1`) the share `ratio / (1 + ratio)` of the available memory, less the
    request slots."""
    if max_state_size is not None:
        snap = max(int(max_state_size) - request_slots, 0)
    elif not sharing:
        snap = 0
    elif snapshot_slots >= 0:
        snap = int(snapshot_slots)
    else:
        if memory_ratio <= 0:
            raise ValueError(f"recurrent_state_memory_ratio={memory_ratio} is invalid for a hybrid recurrent model; "
                             f"set --recurrent-state-memory-ratio > 0")
        total = int(available_bytes * memory_ratio / (1.0 + memory_ratio)) // max(per_slot_bytes, 1)
        snap = max(total - request_slots, 0)
    return snap, (request_slots + 1 + snap) * per_slot_bytes


class RecurrentStatePool:
    """`conv_state[layer]` is `[slots, conv_dim, conv_kernel - 1]` and `recurrent_state[layer]` `[slots, heads, Dk, Dv]`;
    both are one tensor over all layers, or, for a model whose layers differ (`layers`: the sizes of each, under the same
    names), a list of tensors."""

    def __init__(self, size: int, num_layers: int = 0, conv_dim: int = 0, conv_kernel: int = 1, num_heads: int = 0,
                 head_k_dim: int = 0, head_v_dim: int = 0, device: str = "cpu", conv_dtype=torch.bfloat16,
                 state_dtype=torch.float32, snapshot_slots: int = 0, layers: list[dict] | None = None):
        self.size = size
        # slots 1..size belong to request rows; `snapshot_slots` more hold prefix-cache checkpoints
        # (owned by the scheduler's unified radix cache)
        self.snapshot_slots = snapshot_slots
        n = size + 1 + snapshot_slots
        if layers is None:
            self.num_layers = num_layers
            self.conv_state = torch.zeros((num_layers, n, conv_dim, conv_kernel - 1), dtype=conv_dtype, device=device)
            self.recurrent_state = torch.zeros((num_layers, n, num_heads, head_k_dim, head_v_dim), dtype=state_dtype,
                                               device=device)
        else:
            self.num_layers = len(layers)
            self.conv_state = [torch.zeros((n, d["conv_dim"], d["conv_kernel"] - 1), dtype=conv_dtype, device=device)
                               for d in layers]
            self.recurrent_state = [torch.zeros((n, d["num_heads"], d["head_k_dim"], d["head_v_dim"]), dtype=state_dtype,
                                                device=device) for d in layers]
        self.free_slots = list(range(1, size + 1))
        self.device = device

    def _planes(self):
        """Every tensor with its slots as dimension `axis`: `(tensor, axis)`."""
        if isinstance(self.conv_state, torch.Tensor):
            return [(self.conv_state, 1), (self.recurrent_state, 1)]
        return [(t, 0) for t in [*self.conv_state, *self.recurrent_state]]

    def available_size(self) -> int:
        return len(self.free_slots)

    def alloc(self, n: int) -> list[int] | None:
        if n > len(self.free_slots):
            return None
        out, self.free_slots = self.free_slots[:n], self.free_slots[n:]
        self.clear_slots(out)
        return out

    def free(self, slots) -> None:
        self.free_slots.extend(int(s) for s in slots)

    def clear_slots(self, slots) -> None:
        idx = torch.as_tensor(list(slots), dtype=torch.long, device=self.device)
        if idx.numel():
            for t, axis in self._planes():
                t.index_fill_(axis, idx, 0)

    def copy_sequence(self, pairs) -> None:
        """Run `(src, dst)` copies in order (a later copy may read what an earlier one wrote)."""
        for s, d in pairs:
            for t, axis in self._planes():
                t.select(axis, d).copy_(t.select(axis, s))

    def copy_slots(self, src, dst) -> None:
        s = torch.as_tensor(list(src), dtype=torch.long, device=self.device)
        d = torch.as_tensor(list(dst), dtype=torch.long, device=self.device)
        for t, axis in self._planes():
            t.index_copy_(axis, d, t.index_select(axis, s))

    def size_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t, _ in self._planes())

    def clear(self) -> None:
        self.free_slots = list(range(1, self.size + 1))
        for t, _ in self._planes():
            t.zero_()
