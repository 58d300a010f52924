"""Plain, slow implementation of the Taralix decoder in float64 numpy: one function per mechanism, whole sequences at
once, keys and values written out per head, no cache and no code shared with the product path.

config: the parsed config.json; weights: dict name -> numpy array ([out, in] for the linear maps).
"""
import numpy as np


def rms_unit(x, eps):
    """x over its root mean square (last axis)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_one(x, w, eps):
    """RMS norm whose gain is stored as its distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def latent(h, w, eps):
    """The compressed row every head's keys and values are made from."""
    return rms_unit(h @ w["dkv"].T, eps) * w["dkv.norm"]


def causal_softmax(s):
    """Rows of scores [T, T] to weights over the keys that are not later than the row."""
    s = np.where(np.tri(len(s), dtype=bool), s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_attention(h, c, w, m):
    """h [T, width], c [T, kv_rank]; m: the mixer's sizes."""
    T, H, D, DV = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, D)
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, DV)
    o = np.stack([causal_softmax(q[:, a] @ k[:, a].T * m["scale"]) @ v[:, a] for a in range(H)], axis=1)
    return o.reshape(T, H * DV) @ w["o"].T


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + np.exp(-z))


def gated(x, gate, up, down, act):
    return (act(x @ gate.T) * (x @ up.T)) @ down.T


def route(x, w, b, top):
    """(chosen experts, their weights), each [T, top]: the largest logits, softmax over those alone."""
    z = x @ w.T + b
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    s = np.take_along_axis(z, idx, axis=-1)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return idx, e / e.sum(axis=-1, keepdims=True)


def mixture(x, w, top):
    idx, p = route(x, w["router"], w["router.b"], top)
    y = np.zeros_like(x)
    for t in range(len(x)):
        for e, g in zip(idx[t], p[t]):
            y[t] += g * gated(x[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], silu)
    return y


def feed_forward(x, entry, w):
    if entry["kind"] == "dense":
        return gated(x, w["gate"], w["up"], w["down"], gelu_tanh)
    return mixture(x, w, entry["router"]["top"])


def _part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer_forward(x, i, weights, cfg, latents):
    """latents: the compressed rows of the layers that make their own, by layer; this one's are added."""
    e, eps, a, p = cfg["layers"][i], cfg["norm"]["eps"], cfg["postln_alpha"], f"l{i}."
    mix = _part(weights, p + "mix.")
    src = e["mixer"].get("kv_from")
    if src is None:
        latents[i] = latent(x, mix, eps)
    c = latents[i if src is None else src]
    x = norm_around_one(a * x + latent_attention(x, c, mix, e["mixer"]), weights[p + "norm1"], eps)
    if e.get("mlp"):
        x = norm_around_one(a * x + feed_forward(x, e["mlp"], _part(weights, p + "mlp.")), weights[p + "norm2"], eps)
    return x


def forward(cfg, weights, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    x, latents, layers = w["embed"][np.asarray(tokens)], {}, []
    for i in range(len(cfg["layers"])):
        x = layer_forward(x, i, w, cfg, latents)
        layers.append(x)
    logits = norm_around_one(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
    return (logits, np.stack(layers)) if want_layers else logits


def router_gaps(cfg, weights, tokens):
    """Per token, the smallest distance over all layers between the last chosen and the first rejected router logit."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    x, latents, gap = w["embed"][np.asarray(tokens)], {}, np.full(len(tokens), np.inf)
    for i, e in enumerate(cfg["layers"]):
        if e.get("mlp") and e["mlp"]["kind"] == "moe" and e["mlp"]["router"]["top"] < e["mlp"]["router"]["experts"]:
            mid = layer_forward(x, i, w, dict(cfg, layers=[dict(a, mlp=None) for a in cfg["layers"]]), dict(latents))
            z = np.sort(mid @ w[f"l{i}.mlp.router"].T + w[f"l{i}.mlp.router.b"], axis=-1)[:, ::-1]
            top = e["mlp"]["router"]["top"]
            gap = np.minimum(gap, z[:, top - 1] - z[:, top])
        x = layer_forward(x, i, w, cfg, latents)
    return gap


def greedy(cfg, weights, tokens, steps):
    """Tokens of greedy decoding, recomputing the whole sequence every step (lowest index on ties)."""
    seq = list(tokens)
    for _ in range(steps):
        seq.append(int(np.argmax(forward(cfg, weights, seq)[-1])))
    return seq[len(tokens):]
