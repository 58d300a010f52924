"""Small random models of the Vupuzen design for the tests: configurations, weights, and the folder a user would have."""
import json
import os

import numpy as np

from mllm_b200.safetensors import bf16_to_f32, f32_to_bf16, save


def attention(heads, kv, dim, vdim, bias_max, scale=None):
    return {"bias_max": bias_max, "dim": dim, "heads": heads, "kv_heads": kv, "scale": scale or 1.3 * dim ** -0.5, "vdim": vdim}


def retention(heads, dim, vdim, rot, decay, base=5000.0):
    assert len(decay) == heads
    return {"decay": decay, "dim": dim, "heads": heads, "rot": {"base": base, "dims": rot}, "vdim": vdim}


def layer(kind, mixer, ff=None, limit=1.5, weights_of=None):
    e = {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(width, vocab, layers, taps=3, eps=1e-5, logit_scale=0.75):
    return {"architecture": "Vupuzen", "canon": {"taps": taps}, "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


def rounded(x):
    """To bf16 and back."""
    return bf16_to_f32(f32_to_bf16(np.asarray(x, np.float32))).reshape(np.shape(x))


def weights(cfg, seed, rel_rows=10, rel_std=1.0):
    """fp32 arrays that bf16 holds exactly, tensor names as in the model files."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, s=1.0: rng.standard_normal((n, k)) * s / np.sqrt(k)
    gain = lambda: np.float32(rng.uniform(0.7, 1.4))
    w = {"embed": rng.standard_normal((V, W)), "head": lin(V, W, 2.0), "final.norm": gain()}
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        m, p = e["mixer"], f"l{i}."
        H, D, DV = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        w.update({p + "norm1": gain(), p + "norm1b": gain(), p + "canon1": rng.standard_normal((W, cfg["canon"]["taps"])) * 0.4})
        w.update({p + "mix.q": lin(H * D, W), p + "mix.k": lin(G * D, W), p + "mix.v": lin(G * DV, W), p + "mix.o": lin(W, H * DV)})
        if e["type"] == "attention":
            w[p + "mix.rel"] = rng.standard_normal((rel_rows, H)) * rel_std
        else:
            w[p + "mix.g"] = lin(H * DV, W)
        if e["mlp"]:
            F = e["mlp"]["ff"]
            w.update({p + "norm2": gain(), p + "norm2b": gain()})
            w.update({p + "mlp.gate": lin(F, W, 1.5), p + "mlp.up": lin(F, W, 1.5), p + "mlp.down": lin(W, F)})
    return {k: rounded(v) for k, v in w.items()}


def write(folder, cfg, w):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save(os.path.join(folder, "model.safetensors"), {k: ("BF16", f32_to_bf16(v)) for k, v in w.items()})
    return str(folder)


# A mix of everything: odd sizes, partial rotation, grouped heads, a layer without a feed-forward, shared weights.
MIXED = config(136, 211, [
    layer("retention", retention(3, 20, 28, 12, [0.9, 0.97, 1.0]), 72),
    layer("attention", attention(4, 2, 24, 40, 37)),
    layer("attention", attention(5, 1, 36, 12, 90), 56, limit=0.6),
    layer("retention", retention(3, 20, 28, 12, [0.9, 0.97, 1.0]), 72, weights_of=0),
    layer("attention", attention(4, 2, 24, 40, 37), weights_of=1),
])
# Heads of 16 .. 256, one head per key, sizes that need no padding, one tap.
WIDE = config(256, 160, [
    layer("attention", attention(3, 3, 128, 256, 50), 128),
    layer("retention", retention(2, 144, 160, 144, [0.995, 0.5]), 64),
    layer("attention", attention(16, 2, 256, 64, 200)),
], taps=1, logit_scale=2.0)
# One layer of each kind, five taps, large groups.
DEEP_CONV = config(72, 97, [
    layer("attention", attention(12, 1, 16, 16, 21), 40, limit=3.0),
    layer("retention", retention(4, 32, 16, 8, [0.8, 0.9, 0.99, 0.999]), None),
], taps=5, eps=1e-6, logit_scale=1.0)
MODELS = {"mixed": MIXED, "wide": WIDE, "deep_conv": DEEP_CONV}
