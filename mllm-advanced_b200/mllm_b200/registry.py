"""Model registry: a folder with config.json and *.safetensors becomes a model that runs on the GPU.

config.json names the design ("architecture", or the first of "architectures").  An entry loads it with the runtime
sizes (slots, tokens per slot, tokens per step) and says which runtime it belongs to: "engine" models (LanguageModel)
step over ragged batches and are served by the scheduler; "qwen2" models are the quantized batch-1 decoder."""
import json
import os

import numpy as np

from . import lm, taralix, vupuzen
from .safetensors import Tensors

DTYPES = {"bfloat16": lm.BF16, "float32": lm.F32}


def _load_vupuzen(cfg, folder, dtype, max_seqs, max_ctx, max_rows):
    return vupuzen.load(cfg, Tensors(folder), DTYPES[dtype], max_seqs, max_ctx, max_rows)


def _load_taralix(cfg, folder, dtype, max_seqs, max_ctx, max_rows):
    return taralix.load(cfg, Tensors(folder), DTYPES[dtype], max_seqs, max_ctx, max_rows)


def _load_qwen2(cfg, folder, dtype, max_seqs, max_ctx, max_rows):
    """Weights by their published names, the linears quantized to int4 on the host (W4A32), lm_head in fp16."""
    import torch

    from . import binding as B
    from .decoder import LINEAR_NAMES, Qwen2Decoder
    t = Tensors(folder)
    heads = cfg["num_attention_heads"]
    dec = Qwen2Decoder(dict(layers=cfg["num_hidden_layers"], hidden=cfg["hidden_size"], q_heads=heads, kv_heads=cfg["num_key_value_heads"],
                            head_dim=cfg.get("head_dim") or cfg["hidden_size"] // heads, inter=cfg["intermediate_size"],
                            vocab=cfg["vocab_size"], max_ctx=max_ctx, eps=cfg["rms_norm_eps"], rope_theta=cfg["rope_theta"]))
    for i in range(cfg["num_hidden_layers"]):
        p = f"model.layers.{i}."
        for name in LINEAR_NAMES:
            q = p + ("self_attn." if name in "qkvo" else "mlp.") + name + "_proj."
            bias = t.f32(q + "bias") if q + "bias" in t else None
            dec.set_linear(i, name, B.quant_prepack(t.f32(q + "weight"), bias))
        dec.set_norm(0, i, t.f32(p + "input_layernorm.weight"))
        dec.set_norm(1, i, t.f32(p + "post_attention_layernorm.weight"))
    dec.set_norm(2, 0, t.f32("model.norm.weight"))
    emb = t.f32("model.embed_tokens.weight")
    head = t.f32("lm_head.weight") if "lm_head.weight" in t else emb
    dec.set_tables(torch.from_numpy(emb).cuda(), torch.from_numpy(np.ascontiguousarray(head)).cuda().half())
    return dec


MODELS = {  # design -> (runtime, number formats, loader)
    vupuzen.ARCHITECTURE: ("engine", ("bfloat16", "float32"), _load_vupuzen),
    taralix.ARCHITECTURE: ("engine", ("bfloat16", "float32"), _load_taralix),
    "Qwen2ForCausalLM": ("qwen2", ("w4a32",), _load_qwen2),
}


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def architecture(cfg):
    name = cfg.get("architecture") or (cfg.get("architectures") or [None])[0]
    if name not in MODELS:
        raise ValueError(f"unknown model design {name!r}; known: {', '.join(sorted(MODELS))}")
    return name


def load(folder, dtype=None, max_seqs=8, max_ctx=2048, max_rows=2048):
    """(model, runtime).  dtype: one of the design's number formats, by default the first."""
    cfg = read_config(folder)
    runtime, dtypes, loader = MODELS[architecture(cfg)]
    dtype = dtype or dtypes[0]
    if dtype not in dtypes:
        raise ValueError(f"{architecture(cfg)} runs in {', '.join(dtypes)}, not in {dtype}")
    return loader(cfg, folder, dtype, max_seqs, max_ctx, max_rows), runtime


def generate(model, runtime, prompts, max_new, stop=(), portion=None):
    """Greedy continuations (lists of token ids)."""
    if runtime == "engine":
        from . import scheduler
        return scheduler.generate(model, prompts, max_new, stop, portion)
    out = []
    for p in prompts:
        model.prefill(p)
        if max_new > 1:
            model.decode(max_new - 1)
        toks = [int(x) for x in model.generated(max_new - 1)]
        cut = next((i + 1 for i, x in enumerate(toks) if x in stop), len(toks))
        out.append(toks[:cut])
    return out
