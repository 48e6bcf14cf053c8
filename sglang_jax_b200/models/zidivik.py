"""Zidivik: a decoder whose layers mix tokens either with a delta rule that decays every key channel on its own (recurrent
state) or with windowed attention that keeps the first tokens (paged keys and values, which later layers may share), in
parallel with a routed feed-forward, followed by a per-layer token input.

The residual stream is fp32; both sublayers of a layer read the same normalised copy of it.  Positions enter at the
embedding only.  Sizes may differ from layer to layer."""

from __future__ import annotations

import math

import torch
from torch import nn

from .. import ops
from ..layers.embeddings import ParallelLMHead, VocabParallelEmbedding
from ..layers.layernorm import StreamRMSNorm
from ..layers.linear_attention import ChannelDeltaRule
from ..layers.logits_processor import LogitsProcessor
from ..layers.moe import RoutedFeedForward
from ..layers.token_side import TokenSide
from ..layers.windowed_attention import WindowedAttention
from ..parallel import state as ps
from ..utils.precision_tracer import precision_tracer

POSITION_BASE = 10000.0


class ZidivikLayer(nn.Module):
    """`kv_layers`: cache layer of every attention layer so far, by layer number (extended here)."""

    def __init__(self, config, index: int, entry: dict, dtype, kv_layers: dict[int, int], linear_index: int):
        super().__init__()
        m, width, eps = entry["mixer"], config.hidden_size, config.norm_eps
        self.is_delta = entry["type"] == "channel_delta"
        self.norm1 = StreamRMSNorm(width, eps, dtype=dtype)
        # partial sums under tensor parallelism: the two sublayers are reduced together
        if self.is_delta:
            self.mix = ChannelDeltaRule(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["decay_rank"],
                                        m["gate_rank"], eps, linear_index, dtype, reduce_results=False)
        else:
            source = m.get("kv_from")
            kv_layers[index] = kv_layers[source] if source is not None else len(set(kv_layers.values()))
            mask = m.get("mask") or {}
            self.mix = WindowedAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps,
                                         kv_layers[index], dtype, mask.get("size"), mask.get("keep_first", 0),
                                         own_kv=source is None, reduce_results=False)
        self.mlp = self.side = None
        if entry.get("mlp") is not None:
            r, e = entry["mlp"]["router"], entry["mlp"]["expert"]
            self.mlp = RoutedFeedForward(width, r["experts"], r["top"], e["ff"], dtype, index, act_limit=e["limit"])
        if config.token_side_dim:
            self.side = TokenSide(width, config.token_side_dim, index, eps, dtype)

    def forward(self, h, x, ids, fb, side_table, next_norm):
        """`x`: the fp32 stream, updated in place; `h`: `norm1(x)`.  Returns `next_norm(x)`."""
        y = self.mix(h, fb)
        if self.mlp is not None:
            xt = self.mlp(h, y, x)
        else:
            xt = ops.stream_add(ps.all_reduce(y), x)
        if self.side is not None:
            return self.side(xt, x, ids, side_table, next_norm)
        return next_norm(x)


class ZidivikForCausalLM(nn.Module):
    is_hybrid_linear = True
    kernel_set = "window_delta"            # csrc/build.py

    def __init__(self, config, dtype=torch.bfloat16, quant_config=None):
        super().__init__()
        self.config = config
        self.dtype = dtype
        # library products (low-rank pairs, widths that are not multiples of 8) reduce in fp32, too
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        width = config.hidden_size
        self.embed_tokens = VocabParallelEmbedding(config.vocab_size, width, dtype)
        turns = POSITION_BASE ** (-2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width) / (2 * math.pi)
        self.register_buffer("position_turns", turns, persistent=False)
        self.side_embed = VocabParallelEmbedding(config.vocab_size, len(config.layers) * config.token_side_dim, dtype) \
            if config.token_side_dim else None
        self.layers = nn.ModuleList()
        kv_layers: dict[int, int] = {}
        lin = 0
        for i, entry in enumerate(config.layers):
            layer = ZidivikLayer(config, i, entry, dtype, kv_layers, lin)
            lin += layer.is_delta
            self.layers.append(layer)
        self.norm = StreamRMSNorm(width, config.norm_eps, dtype=dtype)
        self.lm_head = ParallelLMHead(config.vocab_size, width, dtype)
        self.logits_processor = LogitsProcessor(config.vocab_size)
        self.capture_aux_hidden_states = False
        # what the runner needs to size the caches; a model without attention keeps a token-sized placeholder
        self.kv_layer_shapes = [l.mix.kv_shape() for l in self.layers if not l.is_delta and l.mix.own_kv] or [(1, 8, 0)]
        self.num_kv_layers = len(self.kv_layer_shapes)
        states = [l.mix.state_spec() for l in self.layers if l.is_delta]
        self.recurrent_spec = None
        if states:
            same = all(s == states[0] for s in states)
            self.recurrent_spec = dict(num_layers=len(states), **states[0]) if same else dict(layers=states)

    def forward(self, input_ids, fb, input_embeds=None):
        if input_embeds is None:
            x, _ = ops.embed_scaled(input_ids, self.embed_tokens.weight, 1.0, fb.positions, self.position_turns)
        else:
            x = input_embeds.to(torch.float32, copy=True)
        tracing = precision_tracer.enabled
        if tracing:
            precision_tracer.begin_forward()
            precision_tracer.record(x, "embed_tokens", fb.forward_mode.name)
        norms = [l.norm1 for l in self.layers] + [self.norm]
        side = self.side_embed.weight if self.side_embed is not None else None
        h = norms[0](x)
        for i, layer in enumerate(self.layers):
            h = layer(h, x, input_ids, fb, side, norms[i + 1])
            if tracing:
                precision_tracer.record(x, "layer_residual", fb.forward_mode.name, i)
        return self.logits_processor(h, self.lm_head, fb)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        expected = self._expected_tensors()
        for name, w in weights:
            if name not in expected:
                raise RuntimeError(f"unexpected tensor {name} in the checkpoint")
            self._load_one(name, w)
            expected.discard(name)
        if expected:
            raise RuntimeError(f"checkpoint is missing {len(expected)} tensors, e.g. {sorted(expected)[:5]}")
        self.post_load_weights()
        return {n for n, _ in self.named_parameters()}

    def _expected_tensors(self) -> set[str]:
        names = {"embed", "final.norm", "head"}
        if self.side_embed is not None:
            names.add("side.embed")
        delta = ["q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "norm", "a1", "a2", "dt_bias", "g1", "g2", "o"]
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            names.add(p + "norm1")
            attn = (["q", "k", "v"] if not l.is_delta and l.mix.own_kv else ["q"]) + ["g", "o"]
            names |= {f"{p}mix.{n}" for n in (delta if l.is_delta else attn)}
            if l.mlp is not None:
                names |= {p + "mlp.router", p + "mlp.router.b"}
                names |= {f"{p}mlp.e{e}.{n}" for e in range(l.mlp.gate.weight.shape[0]) for n in ("gate", "up", "down")}
            if l.side is not None:
                names |= {f"{p}side.{n}" for n in ("gate", "proj", "norm")}
        return names

    def _load_one(self, name: str, w: torch.Tensor):
        for top, module in (("embed", self.embed_tokens), ("side.embed", self.side_embed), ("head", self.lm_head),
                            ("final.norm", self.norm)):
            if name == top:
                return module.weight_loader(module.weight, w)
        first, rest = name.split(".", 1)
        layer = self.layers[int(first[1:])]
        if rest == "norm1":
            return layer.norm1.weight_loader(layer.norm1.weight, w)
        group, leaf = rest.split(".", 1)
        getattr(layer, group).load(leaf, w)

    def post_load_weights(self):
        for m in self.modules():
            if hasattr(m, "fold"):
                m.fold()


EntryClass = [ZidivikForCausalLM]
