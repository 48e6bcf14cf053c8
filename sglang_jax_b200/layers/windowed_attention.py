"""Grouped-query softmax attention with a sliding window that keeps the sequence's first tokens, all sizes and constants as
parameters, over the paged `PackedKVPool`.  Scores may be capped, biased by distance (a slope per head) and joined by a learned
sink in the denominator; values may be mixed with those of an earlier layer.

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
    `qk_norm`: True (per head, without weights), "rows" (over all heads at once, with weights) or False.  `softcap` (None: none),
    `distance_bias` (slopes `2^(-8 (h + 1) / H)`) and `sink` act on the scores.  `value_mix`: "source" hands the layer's values
    on, "mix" replaces a learned share of the layer's own by the source's.  `reduce_results=False` leaves a partial sum under
    tensor parallelism."""

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, v_dim: int, scale: float, eps: float,
                 kv_layer_id: int, dtype, window: int | None = None, keep_first: int = 0, qk_norm: bool | str = True,
                 output_gate: bool = True, own_kv: bool = True, reduce_results: bool = True, softcap: float | None = None,
                 distance_bias: bool = False, sink: bool = False, value_mix: str | None = None):
        super().__init__()
        tp = ps.tp_size()
        assert num_heads % num_kv_heads == 0 and num_heads % tp == 0, f"{num_heads} heads do not split over {tp} ranks"
        assert num_kv_heads % tp == 0 or tp % num_kv_heads == 0, f"{num_kv_heads} key heads do not split over {tp} ranks"
        self.layer_id, self.own_kv = kv_layer_id, own_kv
        self.heads, self.kv_heads, self.dim, self.v_dim = num_heads // tp, max(num_kv_heads // tp, 1), dim, v_dim
        self.scale, self.eps = float(scale), float(eps)
        self.window, self.keep_first = int(window or 0), int(keep_first or 0)
        self.qk_norm, self.output_gate = qk_norm, output_gate
        self.softcap, self.value_mix = float(softcap or 0.0), value_mix
        shared = max(tp // num_kv_heads, 1)                          # ranks that hold the same key head
        self.kv_share = shared
        fp32 = dict(dtype=torch.float32)
        if qk_norm == "rows":
            assert own_kv, "queries and keys are normalised together"
            self.q_norm = nn.Parameter(torch.ones(self.heads * dim, **fp32), requires_grad=False)
            self.k_norm = nn.Parameter(torch.ones(self.kv_heads * dim, **fp32), requires_grad=False)
            self.totals = (num_heads * dim, num_kv_heads * dim)
        assert value_mix is None or qk_norm == "rows"
        slopes = [2.0 ** (-8.0 * (ps.tp_rank() * self.heads + h + 1) / num_heads) for h in range(self.heads)]
        self.register_buffer("slopes", torch.tensor(slopes, **fp32) if distance_bias else None, persistent=False)
        self.sink = nn.Parameter(torch.zeros(self.heads, **fp32), requires_grad=False) if sink else None
        self.v_share = nn.Parameter(torch.zeros(1, **fp32), requires_grad=False) if value_mix == "mix" else None
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
        """One checkpoint tensor: q, k, v, g (projections, as far as this layer has them), o; q.norm, k.norm, sink, vmix."""
        if name in self.proj.parts:
            self.proj.weight_loader(self.proj.weight, w, name)
        elif name == "o":
            self.o_proj.weight_loader(self.o_proj.weight, w)
        elif name == "q.norm":
            self.q_norm.data.copy_(w.narrow(0, ps.tp_rank() * self.q_norm.numel(), self.q_norm.numel()))
        elif name == "k.norm":
            n = self.k_norm.numel()
            self.k_norm.data.copy_(w.narrow(0, ps.tp_rank() // self.kv_share * n, n))
        elif name == "sink":
            self.sink.data.copy_(w.narrow(0, ps.tp_rank() * self.heads, self.heads))
        elif name == "vmix":
            if self.v_share is not None:                             # (the source has no use for it)
                self.v_share.data.fill_(float(w))
        else:
            raise KeyError(name)

    def forward(self, h: torch.Tensor, fb) -> torch.Tensor:
        y = self.proj(h)
        cache = fb.token_to_kv_pool.get_kv_buffer(self.layer_id)
        at = self.proj.offset
        if self.qk_norm == "rows":
            q = self._prep_rows(y, cache, fb)
            return self.o_proj(self._attend(q, self.proj.part(y, "g") if self.output_gate else None, cache, fb).flatten(1))
        q = ops.attn_prep(y, at("q"), at("k") if self.own_kv else -1, at("v") if self.own_kv else -1, self.heads,
                          self.kv_heads, self.dim, self.v_dim, self.eps, self.qk_norm, fb.out_cache_loc, cache)
        gate = self.proj.part(y, "g") if self.output_gate else None
        return self.o_proj(self._attend(q, gate, cache, fb).flatten(1))

    def _prep_rows(self, y, cache, fb):
        squares = mix = None
        if ps.tp_size() > 1:
            squares = torch.stack([self.proj.part(y, "q").float().pow(2).sum(-1),
                                   self.proj.part(y, "k").float().pow(2).sum(-1) / self.kv_share], -1)
            squares = ps.all_reduce(squares)
        if self.value_mix == "source":
            fb.extras["source_values"] = self.proj.part(y, "v")
        elif self.value_mix == "mix":
            mix = fb.extras["source_values"]
        at = self.proj.offset
        return ops.attn_prep_rows(y, at("q"), at("k"), at("v"), self.heads, self.kv_heads, self.dim, self.v_dim, self.eps,
                                  self.q_norm, self.k_norm, fb.out_cache_loc, cache, squares, self.totals, mix, self.v_share)

    def _attend(self, q, gate, cache, fb):
        kw = dict(dim=self.dim, v_dim=self.v_dim, scale=self.scale, window=self.window, keep_first=self.keep_first,
                  softcap=self.softcap, slope=self.slopes, sink=self.sink)
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
