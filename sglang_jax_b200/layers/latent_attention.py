"""Latent attention with all sizes and constants as parameters, over the paged latent cache (`MLATokenToKVPool`).

One GEMM produces queries, latent, shared key part and output gate; one kernel normalises the latent, rotates the key
part and the queries and writes the cache.  From there a step's tokens take one of two routes that compute the same
softmax over the same cache rows:

* absorbed (decode, short extends, every fp32 step): queries are mapped into the latent space with the key up-projection,
  attend to the cache rows themselves, and the value up-projection is applied to the result;
* expanded (long bf16 extends): keys and values of the sequence's whole context are computed from the latents by one
  GEMM, and a tcgen05 flash-attention kernel runs per head.

A step may mix both: the choice is made per sequence from the number of its new tokens."""

from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..parallel import state as ps
from .embeddings import get_rope
from .extend_plan import extend_plan
from .linear import PackedColumnParallelLinear, RowParallelLinear


class LatentAttention(nn.Module):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, rot_dim: int, v_dim: int, kv_rank: int, scale: float,
                 rope_base: float, eps: float, max_positions: int, kv_layer_id: int, dtype, output_gate: bool = True):
        super().__init__()
        tp = ps.tp_size()
        assert num_heads % tp == 0, f"{num_heads} heads do not split over {tp} ranks"
        self.layer_id = kv_layer_id
        self.heads, self.dim, self.rot, self.v_dim, self.rank = num_heads // tp, dim, rot_dim, v_dim, kv_rank
        self.scale, self.eps = float(scale), float(eps)
        parts = {"q": (num_heads * (dim + rot_dim), True)}
        if output_gate:
            parts["g"] = (num_heads * v_dim, True)
        parts["dkv"] = (kv_rank + rot_dim, False)
        self.output_gate = output_gate
        self.proj = PackedColumnParallelLinear(hidden_size, parts, dtype)
        self.latent_norm = nn.Parameter(torch.ones(kv_rank, dtype=torch.float32), requires_grad=False)
        # per head: `dim` key rows, then `v_dim` value rows
        self.up = nn.Parameter(torch.empty(self.heads, dim + v_dim, kv_rank, dtype=dtype), requires_grad=False)
        self.o_proj = RowParallelLinear(num_heads * v_dim, hidden_size, False, dtype)
        self.rotary_emb = get_rope(rot_dim, rot_dim, max_positions, rope_base, False, {"rope_type": "exact"}, dtype)

    def load(self, name: str, w: torch.Tensor):
        """One checkpoint tensor: q, g, dkv (latent and key part), dkv.norm, uk / uv (key and value up-projection), o."""
        if name in self.proj.parts:
            self.proj.weight_loader(self.proj.weight, w, name)
        elif name == "dkv.norm":
            self.latent_norm.data.copy_(w)
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
        cache = fb.token_to_kv_pool.get_kv_buffer(self.layer_id)
        cs = self.rotary_emb.cos_sin_cache
        ops.latent_prep(y, self.proj.offset("q"), self.proj.offset("dkv"), self.heads, self.dim, self.rot, self.rank,
                        self.latent_norm, self.eps, cs, fb.positions, fb.out_cache_loc, cache)
        q = self.proj.part(y, "q").unflatten(-1, (self.heads, self.dim + self.rot))
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
        o_lat = ops.latent_attention(q_lat, q[..., self.dim:], cache, fb, self.scale, rows, lens)
        o = torch.empty(T, self.heads, self.v_dim, dtype=q.dtype, device=q.device)
        torch.bmm(o_lat.transpose(0, 1), self.up[:, self.dim:].transpose(1, 2), out=o.transpose(0, 1))
        return o

    def _can_expand(self, q) -> bool:
        return ops.latent_extend_supported(q, self.dim, self.rot, self.v_dim, self.rank)

    # bytes of expanded keys and values held at a time: beyond it the heads go in groups
    EXPAND_BYTES = 2 << 30

    def _expanded(self, q, cache, fb, plan, out):
        lat, pe = ops.latent_gather(cache, fb.page_table, plan.rows, plan.ctx_start, plan.ctx_total, self.rank, self.rot,
                                    fb.page_size)
        per_head = plan.ctx_total * (self.dim + self.v_dim) * lat.element_size()
        step = max(1, min(self.heads, self.EXPAND_BYTES // max(per_head, 1)))
        for h0 in range(0, self.heads, step):
            h1 = min(h0 + step, self.heads)
            kv = ops.linear(lat, self.up[h0:h1].reshape(-1, self.rank))
            ops.latent_extend(q[:, h0:h1], kv, pe, out[:, h0:h1], plan, self.dim, self.v_dim, self.scale)
