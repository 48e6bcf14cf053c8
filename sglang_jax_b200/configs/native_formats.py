"""Configuration files that are not in the HF layout: `config.json` names its design under `architecture` and has keys
of its own.  A translator turns such a file into the attribute names the framework works with and leaves the design's
own description (layer list, constants) in place for the model class."""

from __future__ import annotations

from typing import Callable

_TRANSLATORS: dict[str, Callable[[dict], dict]] = {}


def native_format(name: str):
    def register(fn):
        _TRANSLATORS[name] = fn
        return fn
    return register


def translate_native_config(d: dict) -> dict:
    name = d["architecture"]
    if name not in _TRANSLATORS:
        raise ValueError(f"unknown architecture {name!r} in config.json; known: {sorted(_TRANSLATORS)}")
    return _TRANSLATORS[name](d)


# positions are computed, not learned, and the file states no limit: the context length used unless one is asked for
DEFAULT_CONTEXT = 32768


@native_format("Zozopel")
def _zozopel(d: dict) -> dict:
    layers = d["layers"]
    known = {"delta": "linear_attention", "latent_attention": "full_attention"}
    for i, e in enumerate(layers):
        if e["type"] not in known:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}; known: {sorted(known)}")
        if e.get("mlp") is not None and e["mlp"]["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {e['mlp']['kind']!r}")
    latent = [e["mixer"] for e in layers if e["type"] == "latent_attention"]
    first = latent[0] if latent else dict(kv_rank=8, rot_dim=0, dim=8, vdim=8, heads=layers[0]["mixer"]["heads"])
    return dict(
        architectures=["ZozopelForCausalLM"], model_type="zozopel", hidden_size=d["width"], vocab_size=d["vocab"],
        num_hidden_layers=len(layers), num_attention_heads=first["heads"], layers=layers,
        layer_types=[known[e["type"]] for e in layers], latent_kv_cache=True, kv_lora_rank=first["kv_rank"],
        qk_rope_head_dim=first["rot_dim"], qk_nope_head_dim=first["dim"], v_head_dim=first["vdim"],
        norm_eps=d["norm"]["eps"], embedding_scale=d["embedding"]["scale"], residual_multiplier=d["residual_mult"],
        logit_scale=d["logit_scale"], max_position_embeddings=DEFAULT_CONTEXT, unbounded_positions=True,
        tie_word_embeddings=False, torch_dtype="bfloat16", eos_token_id=None, bos_token_id=None)
