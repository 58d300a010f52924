"""The Vupuzen decoder: config.json and tensor names to the engine's layer descriptions.

Every layer wraps its sublayers in norms on both sides (one gain per norm), reads its mixer's input through a causal
convolution, and mixes by attention (no rotation; a learned bias by log-bucketed distance; a sink of score 0) or by
retention (rotated, a fixed decay per head).  The feed-forward is a clamped gated one, or absent.  A layer may use an
earlier layer's tensors."""
import numpy as np

from . import lm

ARCHITECTURE = "Vupuzen"


def layers_from_config(cfg, rel_rows):
    """rel_rows(i): rows of the distance-bias table that layer i uses."""
    out = []
    for i, e in enumerate(cfg["layers"]):
        m, f = e["mixer"], e.get("mlp")
        src = e.get("weights_of")
        d = {"heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "weights_of": -1 if src is None else src}
        if e["type"] == "attention":
            d.update(mixer=lm.ATTENTION, kv_heads=m["kv_heads"], score_scale=m["scale"], sink=1, bias_rows=rel_rows(i), bias_max=m["bias_max"])
        elif e["type"] == "retention":
            rot = m.get("rot") or {"dims": 0, "base": 1.0}
            d.update(mixer=lm.RETENTION, kv_heads=m["heads"], rot_dims=rot["dims"], rot_base=rot["base"])
            if len(m["decay"]) != m["heads"]:
                raise ValueError(f"layer {i}: {len(m['decay'])} decays for {m['heads']} heads")
        else:
            raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
            d.update(ff=f["ff"], ff_limit=f["limit"])
        out.append(d)
    return out


def model_config(cfg, max_seqs, max_ctx, max_rows):
    return {"vocab": cfg["vocab"], "width": cfg["width"], "conv_taps": cfg["canon"]["taps"], "eps": cfg["norm"]["eps"],
            "logit_scale": cfg["logit_scale"], "max_seqs": max_seqs, "max_ctx": max_ctx, "max_rows": max_rows}


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer_tensors(entry):
    """(engine name, tensor name inside the layer) of a layer that has tensors of its own."""
    names = [("norm1", "norm1"), ("norm1b", "norm1b"), ("conv", "canon1")]
    attn = entry["type"] == "attention"
    names += [(n, "mix." + n) for n in (("q", "k", "v", "o", "rel") if attn else ("q", "k", "v", "g", "o"))]
    if entry.get("mlp") is not None:
        names += [("norm2", "norm2"), ("norm2b", "norm2b")] + [(n, "mlp." + n) for n in ("gate", "up", "down")]
    return names


def load(cfg, tensors, dtype, max_seqs, max_ctx, max_rows):
    model = lm.LanguageModel(model_config(cfg, max_seqs, max_ctx, max_rows),
                             layers_from_config(cfg, lambda i: tensors.shape(f"l{owner(cfg, i)}.mix.rel")[0]), dtype)
    model.set_tensor(-1, "embed", tensors.bf16("embed"))
    model.set_tensor(-1, "head", tensors.bf16("head"))
    model.set_tensor(-1, "final_norm", tensors.f32("final.norm"))
    for i, e in enumerate(cfg["layers"]):
        if owner(cfg, i) != i:
            continue
        for name, tensor in layer_tensors(e):
            get = tensors.bf16 if name in lm._LINEARS else tensors.f32
            model.set_tensor(i, name, get(f"l{i}.{tensor}"))
        if e["type"] == "retention":
            model.set_tensor(i, "decay", np.asarray(e["mixer"]["decay"], np.float64))
    return model
