"""Small random models of the Taralix design for the tests."""
import numpy as np

from lm_models import rounded, write  # noqa: F401  (write: the folder a user would have)


def mixer(heads, dim, vdim, rank, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or 1.1 * dim ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def layer(m, mlp=None):
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, alpha=1.7):
    return {"architecture": "Taralix", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab, "width": width}


def weights(cfg, seed, router_std=5.0):
    """fp32 arrays that bf16 holds exactly, tensor names as in the model files.  Router logits lie far apart, so that few
    tokens are close to a different choice."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda n, k, s=1.0: rng.standard_normal((n, k)) * s / np.sqrt(k)
    around_zero = lambda n: rng.uniform(-0.3, 0.4, n)
    w = {"embed": rng.standard_normal((V, W)), "head": lin(V, W, 2.0), "final.norm": around_zero(W)}
    for i, e in enumerate(cfg["layers"]):
        m, f, p = e["mixer"], e["mlp"], f"l{i}."
        H, D, DV, R = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        w.update({p + "norm1": around_zero(W), p + "mix.q": lin(H * D, W), p + "mix.uk": lin(H * D, R), p + "mix.uv": lin(H * DV, R),
                  p + "mix.o": lin(W, H * DV)})
        if m.get("kv_from") is None:
            w.update({p + "mix.dkv": lin(R, W), p + "mix.dkv.norm": rng.uniform(0.7, 1.4, R)})
        if f is None:
            continue
        w[p + "norm2"] = around_zero(W)
        if f["kind"] == "dense":
            F = f["ff"]
            w.update({p + "mlp.gate": lin(F, W, 1.5), p + "mlp.up": lin(F, W, 1.5), p + "mlp.down": lin(W, F)})
            continue
        F, n = f["expert"]["ff"], f["router"]["experts"]
        w.update({p + "mlp.router": lin(n, W, router_std), p + "mlp.router.b": rng.standard_normal(n) * 2.0})
        for x in range(n):
            q = f"{p}mlp.e{x}."
            w.update({q + "gate": lin(F, W, 1.5), q + "up": lin(F, W, 1.5), q + "down": lin(W, F)})
    return {k: rounded(v) for k, v in w.items()}


# Odd sizes; rows shared with the layer before, with an earlier one, by two layers; a layer without a feed-forward; one
# expert of many, all of few.
MIXED = config(100, 211, [
    layer(mixer(3, 20, 28, 36), experts(7, 3, 24)),
    layer(mixer(5, 24, 12, 52), dense(72)),
    layer(mixer(2, 36, 40, 36, kv_from=0)),
    layer(mixer(3, 8, 16, 36, scale=0.5, kv_from=0), experts(5, 1, 40)),
    layer(mixer(4, 17, 9, 52, kv_from=1), experts(3, 3, 33)),
])
# More heads than an mma tile has rows, sizes that need no padding, a large latent.
WIDE = config(320, 163, [
    layer(mixer(18, 128, 64, 384), experts(40, 6, 48)),
    layer(mixer(33, 16, 32, 384, kv_from=0), dense(192)),
], eps=1e-6, alpha=0.8)
# The largest heads of the prompt kernel and a latent beyond 512.
DEEP = config(72, 97, [
    layer(mixer(2, 256, 256, 600), None),
    layer(mixer(4, 32, 48, 130), experts(2, 1, 16)),
], alpha=3.0)
# Heads beyond the prompt kernel: every row attends through the latent.
HUGE_HEADS = config(64, 61, [layer(mixer(2, 272, 300, 64), dense(64)), layer(mixer(1, 16, 16, 64, kv_from=0), experts(4, 2, 16))])
MODELS = {"mixed": MIXED, "wide": WIDE, "deep": DEEP, "huge_heads": HUGE_HEADS}
