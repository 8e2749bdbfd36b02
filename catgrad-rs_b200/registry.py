"""From a checkpoint folder (config.json + *.safetensors) to a running decoder.

`load_config` picks the model class by the architecture that config.json names, the way the
reference's drivers pick their graph (catgrad-llm/examples/llama/main.rs:60-117), and
`load_decoder` builds the decoder and loads its weights.  A family is added by registering a
function from the parsed config.json to a configuration object.
"""
from __future__ import annotations

import glob
import json
import os

from .decoder import Decoder
from .layered import LayeredConfig
from .synth import ModelConfig


def _hf(arch: str):
    """Llama-family checkpoints in the Hugging Face layout (field names of
    catgrad-llm/src/legacy/models/utils.rs:52-112)."""
    def build(d: dict) -> ModelConfig:
        gemma = arch == "gemma"
        kw = {}
        if d.get("num_experts", d.get("num_local_experts", 0)):
            kw = dict(num_local_experts=d.get("num_experts", d.get("num_local_experts")), num_experts_per_tok=d["num_experts_per_tok"],
                      moe_intermediate_size=d["moe_intermediate_size"], norm_topk_prob=d.get("norm_topk_prob", False),
                      decoder_sparse_step=d.get("decoder_sparse_step", 1))
        if gemma:
            kw.update(attn_logit_softcap=d.get("attn_logit_softcapping") or 0.0, final_logit_softcap=d.get("final_logit_softcapping") or 0.0,
                      sliding_window=d.get("sliding_window") or 0, qk_norm="Gemma3" in d["architectures"][0],
                      sliding_window_pattern=d.get("sliding_window_pattern") or 0, rope_local_base_freq=d.get("rope_local_base_freq") or 0.0)
        return ModelConfig(d["architectures"][0], d["hidden_size"], d["intermediate_size"], d["num_hidden_layers"], d["num_attention_heads"],
                           d.get("num_key_value_heads", d["num_attention_heads"]), d["vocab_size"], head_dim=d.get("head_dim") or 0,
                           rms_norm_eps=d["rms_norm_eps"], rope_theta=d.get("rope_theta", 10000.0),
                           tie_word_embeddings=d.get("tie_word_embeddings", gemma), dtype="bf16", arch=arch,
                           rope_scaling=d.get("rope_scaling"), **kw)
    return build


ARCHITECTURES = {
    "LlamaForCausalLM": _hf("llama"),
    "Qwen3ForCausalLM": _hf("qwen3"),
    "Qwen3MoeForCausalLM": _hf("qwen3"),
    "Gemma2ForCausalLM": _hf("gemma"),
    "Gemma3ForCausalLM": _hf("gemma"),
    "Ralapel": LayeredConfig.from_json,
    "Segedra": LayeredConfig.from_json,
    "Regupel": LayeredConfig.from_json,
    "Kivorax": LayeredConfig.from_json,
}


def config_from_json(d: dict):
    name = d.get("architecture") or (d.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name](d)


def load_config(folder: str):
    with open(os.path.join(folder, "config.json")) as f:
        return config_from_json(json.load(f))


def runs_in_f32(cfg) -> bool:
    """Whether the decoder has an f32 form of this model (attention-only decoders are bf16)."""
    return isinstance(cfg, LayeredConfig)


def load_decoder(backend, folder: str, max_seq: int, max_batch: int, **switches) -> Decoder:
    dec = Decoder(backend, load_config(folder), max_seq=max_seq, max_batch=max_batch, **switches)
    dec.load_file(*sorted(glob.glob(os.path.join(folder, "*.safetensors"))))
    return dec
