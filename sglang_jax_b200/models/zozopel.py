"""Zozopel: a decoder whose layers mix tokens either with a gated delta rule (recurrent state) or with latent attention
(latent KV cache, gated output), each followed by an optional GELU-gated feed-forward.

The residual stream is fp32 and is read by the sublayers directly; normalisation sits on the sublayer's output only, with
a per-channel layer scale and a residual multiplier.  Sizes may differ from layer to layer."""

from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..layers.activation import GeluAndMul
from ..layers.embeddings import ParallelLMHead, VocabParallelEmbedding
from ..layers.latent_attention import LatentAttention
from ..layers.layernorm import PostNormResidual, StreamRMSNorm
from ..layers.linear_attention import GatedDeltaRule
from ..layers.logits_processor import LogitsProcessor
from ..utils.precision_tracer import precision_tracer
from .llama import DenseMLP


class ZozopelLayer(nn.Module):
    def __init__(self, config, entry: dict, dtype, kv_layer_id: int, linear_index: int):
        super().__init__()
        m, width, eps = entry["mixer"], config.hidden_size, config.norm_eps
        self.is_delta = entry["type"] == "delta"
        if self.is_delta:
            self.mix = GatedDeltaRule(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], eps, linear_index,
                                      dtype)
        else:
            assert m["rot"]["dims"] == m["rot_dim"], "the whole rotary part of a head is rotated"
            self.mix = LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"],
                                       m["rot"]["base"], eps, config.max_position_embeddings, kv_layer_id, dtype)
        self.norm1 = PostNormResidual(width, eps, config.residual_multiplier, True, dtype)
        self.mlp = self.norm2 = None
        if entry.get("mlp") is not None:
            self.mlp = DenseMLP(width, entry["mlp"]["ff"], dtype)
            self.mlp.act_fn = GeluAndMul("tanh")
            self.norm2 = PostNormResidual(width, eps, config.residual_multiplier, True, dtype)

    def forward(self, h, x, fb):
        """`x`: the fp32 stream, updated in place; `h`: the same in the model's type.  Returns the next `h`."""
        h = self.norm1(self.mix(h, fb), x)
        if self.mlp is not None:
            h = self.norm2(self.mlp(h), x)
        return h


class ZozopelForCausalLM(nn.Module):
    is_hybrid_linear = True
    kernel_set = "latent_delta"            # csrc/build.py

    def __init__(self, config, dtype=torch.bfloat16, quant_config=None):
        super().__init__()
        self.config = config
        self.dtype = dtype
        # library products (up-projections of single tokens, widths that are not multiples of 8) reduce in fp32, too
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self.embed_tokens = VocabParallelEmbedding(config.vocab_size, config.hidden_size, dtype)
        self.layers = nn.ModuleList()
        kv = lin = 0
        for entry in config.layers:
            layer = ZozopelLayer(config, entry, dtype, kv, lin)
            kv, lin = (kv, lin + 1) if layer.is_delta else (kv + 1, lin)
            self.layers.append(layer)
        self.norm = StreamRMSNorm(config.hidden_size, config.norm_eps, config.logit_scale, dtype)
        self.lm_head = ParallelLMHead(config.vocab_size, config.hidden_size, dtype)
        self.logits_processor = LogitsProcessor(config.vocab_size)
        self.capture_aux_hidden_states = False
        # what the runner needs to size the caches; a model without latent layers keeps a token-sized placeholder
        self.latent_kv_dims = [(l.mix.rank, l.mix.rot) for l in self.layers if not l.is_delta] or [(8, 0)]
        self.num_kv_layers = len(self.latent_kv_dims)
        states = [l.mix.state_spec() for l in self.layers if l.is_delta]
        self.recurrent_spec = None
        if states:
            same = all(s == states[0] for s in states)
            self.recurrent_spec = dict(num_layers=len(states), **states[0]) if same else dict(layers=states)

    def forward(self, input_ids, fb, input_embeds=None):
        if input_embeds is None:
            x, h = ops.embed_scaled(input_ids, self.embed_tokens.weight, self.config.embedding_scale)
        else:
            x = input_embeds.to(torch.float32, copy=True)
            h = x if self.dtype == torch.float32 else x.to(self.dtype)
        tracing = precision_tracer.enabled
        if tracing:
            precision_tracer.begin_forward()
            precision_tracer.record(x, "embed_tokens", fb.forward_mode.name)
        for i, layer in enumerate(self.layers):
            h = layer(h, x, fb)
            if tracing:
                precision_tracer.record(x, "layer_residual", fb.forward_mode.name, i)
        return self.logits_processor(self.norm(x), self.lm_head, fb)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        expected = self._expected_tensors()
        # a layer without a feed-forward has no use for the second norm, should the file carry one
        unused = {f"l{i}.{n}" for i, l in enumerate(self.layers) if l.mlp is None for n in ("norm2", "ls2")}
        for name, w in weights:
            if name in unused:
                continue
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
        delta = ["q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "a", "A_log", "dt_bias", "norm", "g", "o"]
        latent = ["q", "dkv", "dkv.norm", "uk", "uv", "g", "o"]
        for i, l in enumerate(self.layers):
            names |= {f"l{i}.mix.{n}" for n in (delta if l.is_delta else latent)} | {f"l{i}.norm1", f"l{i}.ls1"}
            if l.mlp is not None:
                names |= {f"l{i}.mlp.{n}" for n in ("gate", "up", "down")} | {f"l{i}.norm2", f"l{i}.ls2"}
        return names

    def _load_one(self, name: str, w: torch.Tensor):
        if name == "embed":
            return self.embed_tokens.weight_loader(self.embed_tokens.weight, w)
        if name == "head":
            return self.lm_head.weight_loader(self.lm_head.weight, w)
        if name == "final.norm":
            return self.norm.weight_loader(self.norm.weight, w)
        first, rest = name.split(".", 1)
        layer = self.layers[int(first[1:])]
        if rest in ("norm1", "norm2"):
            norm = getattr(layer, rest)
            return norm.weight_loader(norm.weight, w)
        if rest in ("ls1", "ls2"):
            norm = layer.norm1 if rest == "ls1" else layer.norm2
            return norm.weight_loader(norm.layer_scale, w)
        group, leaf = rest.split(".", 1)
        if group == "mlp":
            if leaf == "down":
                return layer.mlp.down_proj.weight_loader(layer.mlp.down_proj.weight, w)
            up = layer.mlp.gate_up_proj
            return up.weight_loader(up.weight, w, 0 if leaf == "gate" else 1)
        layer.mix.load(leaf, w)

    def post_load_weights(self):
        self.norm.fold()
        for layer in self.layers:
            layer.norm1.fold()
            if layer.norm2 is not None:
                layer.norm2.fold()


EntryClass = [ZozopelForCausalLM]
