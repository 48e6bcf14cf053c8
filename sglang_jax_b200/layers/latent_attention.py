"""Latent attention with all sizes and constants as parameters, over the latent rows of a paged cache (`MLATokenToKVPool`, or
`PackedKVPool` where other kinds of attention share it).

One GEMM produces queries, latent, shared key part and output gate; one kernel normalises the latent, rotates the key
part and the queries and writes the cache.  Queries may come from a latent of their own (`q_rank`): then the same kernel
normalises that, a second GEMM expands it and a second kernel rotates the result.  From there a step's tokens take one of two
routes that compute the same softmax over the same cache rows:

* absorbed (decode, short extends, every fp32 step): queries are mapped into the latent space with the key up-projection,
  attend to the cache rows themselves, and the value up-projection is applied to the result;
* expanded (long bf16 extends): keys and values of the tokens that the sequence sees are computed from the latents by one
  GEMM, and a tcgen05 flash-attention kernel runs per head.

A step may mix both: the choice is made per sequence from the number of its new tokens."""

from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..parallel import state as ps
from .embeddings import get_rope
from .extend_plan import extend_plan
from .linear import ColumnParallelLinear, PackedColumnParallelLinear, RowParallelLinear


class LatentAttention(nn.Module):
    """`q_rank`: width of the queries' latent (None: none); `window`: how many keys a query sees, itself included (None: all);
    `sink`: a learned entry per head in the softmax's denominator."""

    def __init__(self, hidden_size: int, num_heads: int, dim: int, rot_dim: int, v_dim: int, kv_rank: int, scale: float,
                 rope_base: float, eps: float, max_positions: int, kv_layer_id: int, dtype, output_gate: bool = True,
                 q_rank: int | None = None, window: int | None = None, sink: bool = False):
        super().__init__()
        tp = ps.tp_size()
        assert num_heads % tp == 0, f"{num_heads} heads do not split over {tp} ranks"
        self.layer_id = kv_layer_id
        self.heads, self.dim, self.rot, self.v_dim, self.rank = num_heads // tp, dim, rot_dim, v_dim, kv_rank
        self.scale, self.eps = float(scale), float(eps)
        self.window = int(window or 0)
        parts = {"dq": (q_rank, False)} if q_rank else {"q": (num_heads * (dim + rot_dim), True)}
        if output_gate:
            parts["g"] = (num_heads * v_dim, True)
        parts["dkv"] = (kv_rank + rot_dim, False)
        self.output_gate = output_gate
        self.proj = PackedColumnParallelLinear(hidden_size, parts, dtype)
        self.latent_norm = nn.Parameter(torch.ones(kv_rank, dtype=torch.float32), requires_grad=False)
        self.query_norm = self.query_up = None
        if q_rank:
            self.query_norm = nn.Parameter(torch.ones(q_rank, dtype=torch.float32), requires_grad=False)
            self.query_up = ColumnParallelLinear(q_rank, num_heads * (dim + rot_dim), False, dtype)
        self.sink = nn.Parameter(torch.zeros(self.heads, dtype=torch.float32), requires_grad=False) if sink else None
        # per head: `dim` key rows, then `v_dim` value rows
        self.up = nn.Parameter(torch.empty(self.heads, dim + v_dim, kv_rank, dtype=dtype), requires_grad=False)
        self.o_proj = RowParallelLinear(num_heads * v_dim, hidden_size, False, dtype)
        self.rotary_emb = get_rope(rot_dim, rot_dim, max_positions, rope_base, False, {"rope_type": "exact"}, dtype)

    def kv_shape(self) -> tuple[int, int, int]:
        """`(heads, key width, value width)` of the rows this layer keeps in a `PackedKVPool`."""
        return 1, self.rank + self.rot, 0

    def load(self, name: str, w: torch.Tensor):
        """One checkpoint tensor: q or dq, dq.norm, uq (queries, by way of their latent), g, dkv (latent and key part), dkv.norm,
        uk / uv (key and value up-projection), sink, o."""
        if name in self.proj.parts:
            self.proj.weight_loader(self.proj.weight, w, name)
        elif name == "dkv.norm":
            self.latent_norm.data.copy_(w)
        elif name == "dq.norm" and self.query_norm is not None:
            self.query_norm.data.copy_(w)
        elif name == "uq" and self.query_up is not None:
            self.query_up.weight_loader(self.query_up.weight, w)
        elif name == "sink" and self.sink is not None:
            self.sink.data.copy_(w.narrow(0, ps.tp_rank() * self.heads, self.heads))
        elif name in ("uk", "uv"):
            dst = self.up.data[:, :self.dim] if name == "uk" else self.up.data[:, self.dim:]
            n = self.heads * dst.shape[1]
            dst.copy_(w.narrow(0, ps.tp_rank() * n, n).view(dst.shape))
        elif name == "o":
            self.o_proj.weight_loader(self.o_proj.weight, w)
        else:
            raise KeyError(name)

    # ------------------------------------------------------------------
    def forward(self, h: torch.Tensor, fb) -> torch.Tensor:
        y = self.proj(h)
        cache = fb.token_to_kv_pool.get_latent_buffer(self.layer_id)
        cs = self.rotary_emb.cos_sin_cache
        c_q = ops.latent_prep(y, self.proj.offset("dq" if self.query_up is not None else "q"), self.proj.offset("dkv"),
                              self.heads, self.dim, self.rot, self.rank, self.latent_norm, self.eps, cs, fb.positions,
                              fb.out_cache_loc, cache, self.query_norm)
        q = self.proj.part(y, "q") if self.query_up is None else self.query_up(c_q)
        q = q.unflatten(-1, (self.heads, self.dim + self.rot))
        if self.query_up is not None:
            ops.latent_rotate(q, self.dim, cs, fb.positions)
        o = self._attend(q, cache, fb).flatten(1)
        if self.output_gate:
            o = ops.sigmoid_gate(o, self.proj.part(y, "g"))
        return self.o_proj(o)

    def _attend(self, q, cache, fb):
        if not fb.forward_mode.is_decode():
            plan = extend_plan(fb, self._can_expand(q))
            if plan.long:
                o = torch.empty(q.shape[0], self.heads, self.v_dim, dtype=q.dtype, device=q.device)
                self._expanded(q, cache, fb, plan, o)
                if plan.short_tokens is not None:
                    t = plan.short_tokens
                    o[t] = self._absorbed(q[t], cache, fb, plan.token_rows[t], plan.token_lens[t])
                return o
        return self._absorbed(q, cache, fb)

    def _absorbed(self, q, cache, fb, rows=None, lens=None):
        """Every query token on its own; `rows` / `lens`: its page-table row and the tokens it sees (None: the step's)."""
        T = q.shape[0]
        q_lat = torch.empty(T, self.heads, self.rank, dtype=q.dtype, device=q.device)
        torch.bmm(q[..., :self.dim].transpose(0, 1), self.up[:, :self.dim], out=q_lat.transpose(0, 1))
        o_lat = ops.latent_attention(q_lat, q[..., self.dim:], cache, fb, self.scale, rows, lens, self.window, self.sink)
        o = torch.empty(T, self.heads, self.v_dim, dtype=q.dtype, device=q.device)
        torch.bmm(o_lat.transpose(0, 1), self.up[:, self.dim:].transpose(1, 2), out=o.transpose(0, 1))
        return o

    def _can_expand(self, q) -> bool:
        return ops.latent_extend_supported(q, self.dim, self.rot, self.v_dim, self.rank)

    # bytes of expanded keys and values held at a time: beyond it the heads go in groups
    EXPAND_BYTES = 2 << 30

    def _expanded(self, q, cache, fb, plan, out):
        ctx = plan.context(self.window)
        lat, pe = ops.latent_gather(cache, fb.page_table, plan.rows, ctx.start, ctx.total, self.rank, self.rot, fb.page_size,
                                    ctx.skip)
        per_head = ctx.total * (self.dim + self.v_dim) * lat.element_size()
        step = max(1, min(self.heads, self.EXPAND_BYTES // max(per_head, 1)))
        for h0 in range(0, self.heads, step):
            h1 = min(h0 + step, self.heads)
            kv = ops.linear(lat, self.up[h0:h1].reshape(-1, self.rank))
            ops.latent_extend(q[:, h0:h1], kv, pe, out[:, h0:h1], plan, self.dim, self.v_dim, self.scale, self.window,
                              self.sink[h0:h1] if self.sink is not None else None)
