"""Per-layer token input: a slice of a second, narrow token table gates a bottleneck of the residual stream, and the
normalised result is added to it:  `x <- x + rmsnorm(P (gelu_tanh(G x) * table[token, slice])) * weight`."""

from __future__ import annotations

import torch
from torch import nn

from .. import ops
from .layernorm import PostNormResidual
from .linear import ReplicatedLinear


class TokenSide(nn.Module):
    """`table [vocab, layers * dim]` belongs to the model, `index` selects this layer's slice.  Replicated over tensor
    ranks."""

    def __init__(self, hidden_size: int, dim: int, index: int, eps: float, dtype):
        super().__init__()
        self.dim, self.offset = dim, index * dim
        self.gate = ReplicatedLinear(hidden_size, dim, False, dtype)
        self.proj = ReplicatedLinear(dim, hidden_size, False, dtype)
        self.norm = PostNormResidual(hidden_size, eps, dtype=dtype)

    def load(self, name: str, w: torch.Tensor):
        """One checkpoint tensor: gate, proj or norm."""
        m = getattr(self, name)
        m.weight_loader(m.weight, w)

    def forward(self, h, x, ids, table, next_norm):
        """`x`: the fp32 stream, updated in place; `h`: the same in the model's type.  Returns `next_norm(x)`."""
        y = self.proj(ops.token_side_gate(self.gate(h), table, ids, self.offset))
        return self.norm.then(y, x, next_norm)
