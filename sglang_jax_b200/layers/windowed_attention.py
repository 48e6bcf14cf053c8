"""Grouped-query softmax attention with a sliding window that keeps the sequence's first tokens, all sizes and constants as
parameters, over the paged `PackedKVPool`.

One GEMM produces queries, keys, values and a gate per head; one kernel normalises queries and keys and writes the cache
rows.  A step's tokens then take one of two routes over the same rows: tiles of one sequence's new tokens (prefill,
tcgen05), or every token as a query of its own (decode and short extends).  A layer may read the keys and values that an
earlier layer has written (`own_kv=False`: it projects queries only, and `kv_layer_id` is that layer's)."""

from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..parallel import state as ps
from .extend_plan import extend_plan
from .linear import PackedColumnParallelLinear, RowParallelLinear


class WindowedAttention(nn.Module):
    """`window`: how many keys a query sees, itself included (None: all); `keep_first`: leading keys that stay visible.
    `reduce_results=False` leaves a partial sum under tensor parallelism."""

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, v_dim: int, scale: float, eps: float,
                 kv_layer_id: int, dtype, window: int | None = None, keep_first: int = 0, qk_norm: bool = True,
                 output_gate: bool = True, own_kv: bool = True, reduce_results: bool = True):
        super().__init__()
        tp = ps.tp_size()
        assert num_heads % num_kv_heads == 0 and num_heads % tp == 0, f"{num_heads} heads do not split over {tp} ranks"
        assert num_kv_heads % tp == 0 or tp % num_kv_heads == 0, f"{num_kv_heads} key heads do not split over {tp} ranks"
        self.layer_id, self.own_kv = kv_layer_id, own_kv
        self.heads, self.kv_heads, self.dim, self.v_dim = num_heads // tp, max(num_kv_heads // tp, 1), dim, v_dim
        self.scale, self.eps = float(scale), float(eps)
        self.window, self.keep_first = int(window or 0), int(keep_first or 0)
        self.qk_norm, self.output_gate = qk_norm, output_gate
        shared = max(tp // num_kv_heads, 1)                          # ranks that hold the same key head
        parts = {"q": (num_heads * dim, True)}
        if own_kv:
            parts["k"], parts["v"] = (num_kv_heads * dim, shared), (num_kv_heads * v_dim, shared)
        if output_gate:
            parts["g"] = (num_heads, True)
        self.proj = PackedColumnParallelLinear(hidden_size, parts, dtype)
        self.o_proj = RowParallelLinear(num_heads * v_dim, hidden_size, False, dtype, reduce_results=reduce_results)

    def kv_shape(self) -> tuple[int, int, int]:
        """This rank's `(heads, key width, value width)` for the cache pool."""
        return self.kv_heads, self.dim, self.v_dim

    def load(self, name: str, w: torch.Tensor):
        """One checkpoint tensor: q, k, v, g (projections, as far as this layer has them), o."""
        if name in self.proj.parts:
            self.proj.weight_loader(self.proj.weight, w, name)
        elif name == "o":
            self.o_proj.weight_loader(self.o_proj.weight, w)
        else:
            raise KeyError(name)

    def forward(self, h: torch.Tensor, fb) -> torch.Tensor:
        y = self.proj(h)
        cache = fb.token_to_kv_pool.get_kv_buffer(self.layer_id)
        at = self.proj.offset
        q = ops.attn_prep(y, at("q"), at("k") if self.own_kv else -1, at("v") if self.own_kv else -1, self.heads,
                          self.kv_heads, self.dim, self.v_dim, self.eps, self.qk_norm, fb.out_cache_loc, cache)
        gate = self.proj.part(y, "g") if self.output_gate else None
        return self.o_proj(self._attend(q, gate, cache, fb).flatten(1))

    def _attend(self, q, gate, cache, fb):
        kw = dict(dim=self.dim, v_dim=self.v_dim, scale=self.scale, window=self.window, keep_first=self.keep_first)
        if not ops.use_native_wide(q):
            return ops.reference.window_attention(q, gate, cache, fb, **kw)
        if fb.forward_mode.is_decode():
            return ops.window_attention(q, gate, cache, fb, fb.req_pool_indices, fb.seq_lens, **kw)
        plan = extend_plan(fb, ops.window_extend_supported(q, cache, self.dim, self.v_dim))
        if not plan.long:
            return ops.window_attention(q, gate, cache, fb, plan.token_rows, plan.token_lens, **kw)
        out = torch.empty(q.shape[0], self.heads, self.v_dim, dtype=q.dtype, device=q.device)
        ops.window_extend(q, gate, cache, fb, plan, out, **kw)
        if plan.short_tokens is not None:
            t = plan.short_tokens
            out[t] = ops.window_attention(q[t], gate[t] if gate is not None else None, cache, fb, plan.token_rows[t],
                                          plan.token_lens[t], **kw)
        return out
