"""The model registry: what it knows, and a Qwen2 folder under its published tensor names against the same decoder filled
by hand."""
import json
import os
import re

import numpy as np
import pytest

import lm_models as M
import test_decoder as td
from mllm_b200 import lm, registry
from mllm_b200.safetensors import save

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_engine_library_exports_every_declared_symbol():
    import ctypes as C
    hdr = open(os.path.join(ROOT, "include", "mllmb200_lm.h")).read()
    names = set(re.findall(r"MLLMB200_API\s+[\w\s\*]+?\b(mllmb200_lm_\w+)\s*\(", hdr))
    assert len(names) >= 12
    L = C.CDLL(lm.lib_path())
    for n in sorted(names):
        assert hasattr(L, n), n


def test_known_designs_and_formats(tmp_path, capsys):
    from mllm_b200 import __main__ as cli
    cli.main(["info", "--model", M.write(tmp_path / "m", M.MIXED, M.weights(M.MIXED, 1))])
    assert "Vupuzen" in capsys.readouterr().out
    assert registry.architecture({"architectures": ["Qwen2ForCausalLM"]}) == "Qwen2ForCausalLM"
    with pytest.raises(ValueError):
        registry.load(str(tmp_path / "m"), dtype="w4a32")


def write_qwen2(folder, cfg, w, raw):
    os.makedirs(folder)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump({"architectures": ["Qwen2ForCausalLM"], "num_hidden_layers": cfg["layers"], "hidden_size": cfg["hidden"],
                   "num_attention_heads": cfg["q_heads"], "num_key_value_heads": cfg["kv_heads"], "head_dim": cfg["head_dim"],
                   "intermediate_size": cfg["inter"], "vocab_size": cfg["vocab"], "rms_norm_eps": cfg["eps"],
                   "rope_theta": cfg["rope_theta"]}, f)
    t = {"model.embed_tokens.weight": w["embedding"], "lm_head.weight": w["lm_head"], "model.norm.weight": w["final_norm"]}
    for l in range(cfg["layers"]):
        t[f"model.layers.{l}.input_layernorm.weight"] = w[f"ln1.{l}"]
        t[f"model.layers.{l}.post_attention_layernorm.weight"] = w[f"ln2.{l}"]
    for l, name, wt, b in raw:
        p = f"model.layers.{l}.{'self_attn' if name in 'qkvo' else 'mlp'}.{name}_proj."
        t[p + "weight"] = wt
        if b is not None:
            t[p + "bias"] = b
    save(os.path.join(folder, "model.safetensors"), {k: ("F32", np.asarray(v, np.float32)) for k, v in t.items()})
    return str(folder)


@pytest.mark.gpu
def test_qwen2_folder_generates_what_the_decoder_does(tmp_path):
    cfg = td.SMALL
    w, raw = td.make_model(cfg, 31)
    model, runtime = registry.load(write_qwen2(tmp_path / "q", cfg, w, raw), max_ctx=cfg["max_ctx"])
    assert runtime == "qwen2"
    prompts = [[3, 17, 999, 0, 5], [42] * 9]
    got = registry.generate(model, runtime, prompts, 8)
    ref = td._gpu_decoder(cfg, w, raw)
    for p, g in zip(prompts, got):
        ref.prefill(p)
        ref.decode(7)
        assert ref.generated(7).tolist() == g
    stop = got[0][3]
    assert registry.generate(model, runtime, prompts[:1], 8, {stop})[0] == got[0][:got[0].index(stop) + 1]
    model.close()
    ref.close()
