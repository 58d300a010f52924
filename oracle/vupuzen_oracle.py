"""Plain, slow implementation of the Vupuzen decoder in float64 numpy: one function per mechanism, whole sequences
at once, no cache and no code shared with the product path.

config: the parsed config.json; weights: dict name -> numpy array ([out, in] for the linear maps).
Retention is evaluated in its recurrent form, attention by writing out every score.
"""
import math

import numpy as np


def rms_unit(x, eps):
    """x over its root mean square (last axis)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_scalar(x, gain, eps):
    """RMS norm whose gain is one number for all coordinates."""
    return rms_unit(x, eps) * float(gain)


def causal_conv(h, taps_w):
    """Depthwise causal convolution over time; h [T, C], taps_w [C, taps]; tap taps-1 meets the current row."""
    T, taps = h.shape[0], taps_w.shape[1]
    y = np.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += taps_w[:, j] * h[s]
    return y


def distance_bucket(n, buckets, max_distance):
    """Exact up to half of the buckets, then logarithmic up to max_distance, then the last one.
    The floor is taken exactly: the largest m with (n / half)^(B - half) >= (D / half)^m, in integers."""
    half = buckets // 2
    if n < half:
        return n
    rest = buckets - half
    m = 0
    while half + m < buckets - 1 and n ** rest * half ** (m + 1) >= max_distance ** (m + 1) * half ** rest:
        m += 1
    return half + m


def distance_bias(rel, bias_max, i, j):
    """Row of the bias table for query position i and key position j (all heads)."""
    return rel[distance_bucket(i - j, rel.shape[0], bias_max)]


def softmax_with_sink(s):
    """exp(s) / (1 + sum exp(s)) along the last axis; -inf marks what is not seen."""
    m = np.maximum(np.max(s, axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def attention(h, w, cfg):
    """Grouped-query causal attention, distance bias, sink of score 0.  w: dict with q, k, v, o, rel."""
    T, H, G, D, DV = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = (h @ w["q"].T).reshape(T, H, D)
    k = (h @ w["k"].T).reshape(T, G, D)
    v = (h @ w["v"].T).reshape(T, G, DV)
    bias = np.stack([distance_bias(w["rel"], cfg["bias_max"], n, 0) for n in range(T)])  # [T, H]
    out = np.zeros((T, H, DV))
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    for a in range(H):
        g = a // (H // G)
        s = (q[:, a] @ k[:, g].T) * cfg["scale"] + bias[np.maximum(dist, 0), a]
        s = np.where(dist >= 0, s, -np.inf)
        out[:, a] = softmax_with_sink(s) @ v[:, g]
    return out.reshape(T, H * DV) @ w["o"].T


def rotate_half_split(x, positions, dims, base):
    """Rotates coordinate i with coordinate i + dims/2, i < dims/2; x [T, heads, D]; the rest passes."""
    y = x.copy()
    for i in range(dims // 2):
        a = positions * base ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        y[:, :, i] = u * c - v * s
        y[:, :, i + dims // 2] = v * c + u * s
    return y


def retention_recurrence(q, k, v, decay):
    """S <- decay S + k v^T, o = S^T q per head; q, k [T, H, D], v [T, H, DV]; returns (o, final state)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = np.asarray(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o, S


def silu(z):
    return z / (1.0 + np.exp(-z))


def retention(h, w, cfg, eps):
    """w: dict with q, k, v, g, o."""
    T, H, D = h.shape[0], cfg["heads"], cfg["dim"]
    DV = w["v"].shape[0] // H
    pos = np.arange(T, dtype=np.float64)
    q = (h @ w["q"].T).reshape(T, H, D)
    k = (h @ w["k"].T).reshape(T, H, D)
    v = (h @ w["v"].T).reshape(T, H, DV)
    rot = cfg.get("rot")
    if rot:
        q = rotate_half_split(q, pos, rot["dims"], rot["base"])
        k = rotate_half_split(k, pos, rot["dims"], rot["base"])
    o, _ = retention_recurrence(q, k * D ** -0.5, v, cfg["decay"])
    return (rms_unit(o, eps).reshape(T, H * DV) * silu(h @ w["g"].T)) @ w["o"].T


def gated_clamped_mlp(h, w, limit):
    """w: dict with gate, up, down."""
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)) @ w["down"].T


def _part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer_forward(x, entry, index, weights, cfg):
    src = entry.get("weights_of")
    p = "l%d." % (index if src is None else src)
    eps = cfg["norm"]["eps"]
    h = rms_norm_scalar(x, weights[p + "norm1"], eps)
    h = h + causal_conv(h, weights[p + "canon1"])
    mix = _part(weights, p + "mix.")
    y = attention(h, mix, entry["mixer"]) if entry["type"] == "attention" else retention(h, mix, entry["mixer"], eps)
    x = x + rms_norm_scalar(y, weights[p + "norm1b"], eps)
    if entry.get("mlp"):
        y = gated_clamped_mlp(rms_norm_scalar(x, weights[p + "norm2"], eps), _part(weights, p + "mlp."), entry["mlp"]["limit"])
        x = x + rms_norm_scalar(y, weights[p + "norm2b"], eps)
    return x


def forward(cfg, weights, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    x = w["embed"][np.asarray(tokens)]
    layers = []
    for i, entry in enumerate(cfg["layers"]):
        x = layer_forward(x, entry, i, w, cfg)
        layers.append(x)
    logits = rms_norm_scalar(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T * cfg["logit_scale"]
    return (logits, np.stack(layers)) if want_layers else logits


def greedy(cfg, weights, tokens, steps):
    """Tokens of greedy decoding, recomputing the whole sequence every step (lowest index on ties)."""
    seq = list(tokens)
    for _ in range(steps):
        seq.append(int(np.argmax(forward(cfg, weights, seq)[-1])))
    return seq[len(tokens):]
