"""The Taralix decoder: config.json and tensor names to the engine's layer descriptions.

The norms stand behind the residual sum, norm(alpha x + sublayer(x)), with gains stored as their distance from one.  The
mixer is latent attention: one normed row per position is cached and every head's key and value are made from it; a layer
may use an earlier layer's rows.  Feed-forwards are dense (gelu), mixtures of experts (silu; softmax over the chosen
experts' logits), or absent."""
from . import lm

ARCHITECTURE = "Taralix"


def layers_from_config(cfg):
    out = []
    for i, e in enumerate(cfg["layers"]):
        if e["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        m, f = e["mixer"], e.get("mlp")
        src = m.get("kv_from")
        d = dict(mixer=lm.LATENT, heads=m["heads"], kv_heads=m["heads"], dim=m["dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                 kv_from=-1 if src is None else src, score_scale=m["scale"])
        if f is not None:
            if f["kind"] == "dense":
                d.update(ff=f["ff"], act=lm.GELU)
            elif f["kind"] == "moe":
                d.update(ff=f["expert"]["ff"], act=lm.SILU, experts=f["router"]["experts"], top=f["router"]["top"])
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
        out.append(d)
    return out


def model_config(cfg, max_seqs, max_ctx, max_rows):
    return {"vocab": cfg["vocab"], "width": cfg["width"], "conv_taps": 0, "eps": cfg["norm"]["eps"], "logit_scale": 1.0,
            "norm_place": lm.NORM_POST, "residual_scale": cfg["postln_alpha"], "max_seqs": max_seqs, "max_ctx": max_ctx, "max_rows": max_rows}


def load_layer(model, tensors, i, entry):
    p = f"l{i}."
    bf16 = lambda name, tensor: model.set_tensor(i, name, tensors.bf16(p + tensor))
    gain = lambda name: model.set_tensor(i, name, 1.0 + tensors.f32(p + name))
    gain("norm1")
    for name in ("q", "uk", "uv", "o"):
        bf16(name, "mix." + name)
    if entry["mixer"].get("kv_from") is None:
        bf16("dkv", "mix.dkv")
        model.set_tensor(i, "dkv_norm", tensors.f32(p + "mix.dkv.norm"))
    f = entry.get("mlp")
    if f is None:
        return
    gain("norm2")
    if f["kind"] == "dense":
        for name in ("gate", "up", "down"):
            bf16(name, "mlp." + name)
        return
    bf16("router", "mlp.router")
    model.set_tensor(i, "router_b", tensors.f32(p + "mlp.router.b"))
    for x in range(f["router"]["experts"]):
        for name in ("gate", "up", "down"):
            model.set_expert(i, x, name, tensors.bf16(f"{p}mlp.e{x}.{name}"))


def load(cfg, tensors, dtype, max_seqs, max_ctx, max_rows):
    model = lm.LanguageModel(model_config(cfg, max_seqs, max_ctx, max_rows), layers_from_config(cfg), dtype)
    model.set_tensor(-1, "embed", tensors.bf16("embed"))
    model.set_tensor(-1, "head", tensors.bf16("head"))
    model.set_tensor(-1, "final_norm", 1.0 + tensors.f32("final.norm"))
    for i, e in enumerate(cfg["layers"]):
        load_layer(model, tensors, i, e)
    return model
