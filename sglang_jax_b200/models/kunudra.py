"""Kunudra: a decoder whose layers mix tokens with latent attention or with grouped-query attention whose scores fall with the
distance, both under a sliding window and with a learned sink, each followed by a dense feed-forward, by routed experts with
identity choices and a gated shared expert, or by none.

The residual stream is fp32 and is read by the sublayers directly; the norm sits behind each residual sum.  Attention layers
may mix their values with those of the first one.  A table of token pairs is added to the embedding.  Sizes may differ from
layer to layer."""

from __future__ import annotations

import torch
from torch import nn

from ..layers.activation import SwiGLU
from ..layers.embeddings import PairEmbedding, ParallelLMHead, VocabParallelEmbedding
from ..layers.latent_attention import LatentAttention
from ..layers.layernorm import StreamRMSNorm, SumNorm
from ..layers.logits_processor import LogitsProcessor
from ..layers.moe import ScoredFeedForward
from ..layers.windowed_attention import WindowedAttention
from ..utils.precision_tracer import precision_tracer
from .llama import DenseMLP


class KunudraLayer(nn.Module):
    """`first_values`: number of the layer whose values the others mix in."""

    def __init__(self, config, index: int, entry: dict, dtype, first_values: int | None):
        super().__init__()
        m, width, eps = entry["mixer"], config.hidden_size, config.norm_eps
        window = (m.get("mask") or {}).get("size")
        if entry["type"] == "latent_attention":
            self.mix = LatentAttention(width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"],
                                       m["rot"]["base"], eps, config.max_position_embeddings, index, dtype,
                                       output_gate=False, q_rank=m["q_rank"], window=window, sink=True)
        else:
            mix = None if not m.get("v_mix") else "source" if index == first_values else "mix"
            self.mix = WindowedAttention(width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps, index, dtype,
                                         window, qk_norm="rows", output_gate=False, softcap=m.get("softcap"),
                                         distance_bias=True, sink=True, value_mix=mix)
        self.norm1 = SumNorm(width, eps, config.residual_alpha, dtype)
        self.mlp = self.norm2 = None
        self.is_moe = False
        if entry.get("mlp") is not None:
            f = entry["mlp"]
            self.is_moe = f["kind"] == "moe"
            if self.is_moe:
                r = f["router"]
                self.mlp = ScoredFeedForward(width, r["experts"], r.get("identity", 0), r["top"], f["expert"]["ff"],
                                             r.get("scale", 1.0), (f.get("shared") or {}).get("ff", 0), dtype, index)
            else:
                self.mlp = DenseMLP(width, f["ff"], dtype)
                self.mlp.act_fn = SwiGLU()
            self.norm2 = SumNorm(width, eps, config.residual_alpha, dtype)

    def forward(self, h, x, fb, then=None):
        """`x`: the fp32 stream, updated in place; `h`: the same in the model's type.  Returns the next `h`, or `then(x)`."""
        h = self.norm1(self.mix(h, fb), x, then if self.mlp is None else None)
        if self.mlp is None:
            return h
        return self.mlp(h, x, self.norm2, then) if self.is_moe else self.norm2(self.mlp(h), x, then)

    def tensors(self) -> set[str]:
        """Checkpoint names without the layer's prefix."""
        names = {"norm1", "ls1"} | ({"norm2", "ls2"} if self.mlp is not None else set())
        if isinstance(self.mix, LatentAttention):
            names |= {f"mix.{n}" for n in ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "sink", "o")}
        else:
            names |= {f"mix.{n}" for n in ("q", "k", "v", "q.norm", "k.norm", "sink", "o")}
            if self.mix.value_mix is not None:
                names.add("mix.vmix")
        three = ("gate", "up", "down")
        if self.is_moe:
            names |= {"mlp.router", "mlp.correction"}
            names |= {f"mlp.e{e}.{n}" for e in range(self.mlp.experts.num_logical_experts) for n in three}
            if self.mlp.shared is not None:
                names |= {f"mlp.shared.{n}" for n in (*three, "sg")}
        elif self.mlp is not None:
            names |= {f"mlp.{n}" for n in three}
        return names

    def unused(self) -> set[str]:
        """Tensors a file may carry for this layer although nothing reads them."""
        names = {"norm2", "ls2"} if self.mlp is None else set()
        if isinstance(self.mix, WindowedAttention) and self.mix.value_mix is None:
            names.add("mix.vmix")
        return names

    def load(self, name: str, w: torch.Tensor):
        if name in ("norm1", "norm2"):
            norm = getattr(self, name)
            return norm.weight_loader(norm.weight, w)
        if name in ("ls1", "ls2"):
            norm = self.norm1 if name == "ls1" else self.norm2
            return norm.weight_loader(norm.layer_scale, w)
        group, leaf = name.split(".", 1)
        if group == "mix" or self.is_moe:
            return getattr(self, group).load(leaf, w)
        if leaf == "down":
            return self.mlp.down_proj.weight_loader(self.mlp.down_proj.weight, w)
        up = self.mlp.gate_up_proj
        up.weight_loader(up.weight, w, 0 if leaf == "gate" else 1)


class KunudraForCausalLM(nn.Module):
    kernel_set = "window_latent"           # csrc/build.py
    kv_token_ids = True                    # the pair embedding reads a portion's predecessor out of the cache

    def __init__(self, config, dtype=torch.bfloat16, quant_config=None):
        super().__init__()
        self.config = config
        self.dtype = dtype
        # library products (up-projections of single tokens, widths that are not multiples of 8) reduce in fp32, too
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        width, pair = config.hidden_size, config.pair_embedding
        self.embed_tokens = VocabParallelEmbedding(config.vocab_size, width, dtype)
        self.pair_embed = PairEmbedding(pair["buckets"], width, pair["mul_prev"], pair["mul_cur"], dtype)
        mixing = [i for i, e in enumerate(config.layers) if e["type"] == "attention" and e["mixer"].get("v_mix")]
        self.layers = nn.ModuleList(KunudraLayer(config, i, e, dtype, mixing[0] if mixing else None)
                                    for i, e in enumerate(config.layers))
        self.norm = StreamRMSNorm(width, config.norm_eps, dtype=dtype, one_plus=True)
        self.lm_head = ParallelLMHead(config.vocab_size, width, dtype)
        self.logits_processor = LogitsProcessor(config.vocab_size)
        self.capture_aux_hidden_states = False
        # what the runner needs to size the cache
        self.kv_layer_shapes = [l.mix.kv_shape() for l in self.layers]
        self.num_kv_layers = len(self.kv_layer_shapes)

    def forward(self, input_ids, fb, input_embeds=None):
        if input_embeds is None:
            x, h = self.pair_embed(input_ids, self.embed_tokens, fb)
        else:
            x = input_embeds.to(torch.float32, copy=True)
            h = x if self.dtype == torch.float32 else x.to(self.dtype)
        tracing = precision_tracer.enabled
        if tracing:
            precision_tracer.begin_forward()
            precision_tracer.record(x, "embed_tokens", fb.forward_mode.name)
        for i, layer in enumerate(self.layers):
            h = layer(h, x, fb, self.norm if i + 1 == len(self.layers) else None)
            if tracing:
                precision_tracer.record(x, "layer_residual", fb.forward_mode.name, i)
        return self.logits_processor(h, self.lm_head, fb)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        expected = {"embed", "bigram", "final.norm"} | {f"l{i}.{n}" for i, l in enumerate(self.layers) for n in l.tensors()}
        unused = {f"l{i}.{n}" for i, l in enumerate(self.layers) for n in l.unused()}
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

    def _load_one(self, name: str, w: torch.Tensor):
        if name == "embed":
            return self.embed_tokens.weight_loader(self.embed_tokens.weight, w)
        if name == "bigram":
            return self.pair_embed.weight_loader(self.pair_embed.weight, w)
        if name == "final.norm":
            return self.norm.weight_loader(self.norm.weight, w)
        first, rest = name.split(".", 1)
        self.layers[int(first[1:])].load(rest, w)

    def post_load_weights(self):
        self.lm_head.tie_to(self.embed_tokens)
        for m in self.modules():
            if hasattr(m, "fold"):
                m.fold()


EntryClass = [KunudraForCausalLM]
