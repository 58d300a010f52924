"""`bench.py --lm`: prefill and decode throughput of a design on the language-model engine (random bf16 weights) beside the
closest other model at equal layer sizes: same width, heads, head size, feed-forward, vocabulary and depth.  Vupuzen stands
beside the quantized Qwen2 decoder, Taralix (`--lm-design taralix`) beside Vupuzen; a mixture of experts is equal to a dense
feed-forward as wide as the experts a token uses.
Device times by CUDA events on the engines' streams; the best of a few repetitions.  Every timed step streams more
weights than L2 holds (the smallest model reads 0.7 GB per step).

Roofline: a prompt against the measured bf16 rate (dense products of the linears, causal attention, chunked retention), a
decode step against the measured copy bandwidth (weights once, every cache and state byte once, states written too; of a
mixture the experts that so many tokens are expected to choose)."""
import numpy as np

SIZES = {
    # layers like published models of this scale; every fourth layer is retention
    "0.5b": dict(width=896, layers=24, heads=14, kv=2, dim=64, ff=4864, vocab=151936),
    "1.5b": dict(width=1536, layers=28, heads=12, kv=2, dim=128, ff=8960, vocab=151936),
    "2048": dict(width=2048, layers=16, heads=16, kv=4, dim=128, ff=8192, vocab=32000),
}


# Every other layer uses the cached rows of the one before it; a mixture of experts in all layers but the first.
TARALIX_SIZES = {
    "0.5b": dict(width=896, layers=24, heads=14, dim=64, rank=256, ff=4864, vocab=151936),
    "1.5b": dict(width=1536, layers=28, heads=12, dim=128, rank=512, ff=8960, vocab=151936),
    "moe": dict(width=2048, layers=16, heads=16, dim=128, rank=512, ff=8448, experts=64, top=6, vocab=32000),
}


def beside(s):
    """Sizes of the Vupuzen model next to a Taralix one."""
    return dict({k: s[k] for k in ("width", "layers", "heads", "dim", "ff", "vocab")}, kv=2 if s["heads"] % 4 else 4)


def build_taralix(torch, lm, s, max_seqs, max_ctx, max_rows, seed=0):
    gen = torch.Generator(device="cuda").manual_seed(seed)
    W, H, D, R, E = s["width"], s["heads"], s["dim"], s["rank"], s.get("experts", 0)
    layers = []
    for i in range(s["layers"]):
        d = dict(mixer=lm.LATENT, heads=H, kv_heads=H, dim=D, vdim=D, kv_rank=R, kv_from=i - 1 if i % 2 else -1, score_scale=D ** -0.5)
        layers.append(dict(d, ff=s["ff"] // s["top"], act=lm.SILU, experts=E, top=s["top"]) if E and i else dict(d, ff=s["ff"], act=lm.GELU))
    m = lm.LanguageModel(dict(vocab=s["vocab"], width=W, conv_taps=0, max_seqs=max_seqs, max_ctx=max_ctx, max_rows=max_rows, eps=1e-6,
                              logit_scale=1.0, norm_place=lm.NORM_POST, residual_scale=2.0), layers)
    rand = lambda n, k, g=1.0: torch.randn((n, k), device="cuda", generator=gen).mul_(g * k ** -0.5).bfloat16()
    emb = torch.randn((s["vocab"], W), device="cuda", generator=gen).bfloat16()
    m.set_tensor(-1, "embed", emb)
    m.set_tensor(-1, "head", emb[torch.randperm(s["vocab"], device="cuda", generator=gen)])
    one = np.ones(W, np.float32)
    m.set_tensor(-1, "final_norm", one)
    for i, d in enumerate(layers):
        for name, n, k in [("q", H * D, W), ("uk", H * D, R), ("uv", H * D, R), ("o", W, H * D)]:
            m.set_tensor(i, name, rand(n, k))
        if d["kv_from"] < 0:
            m.set_tensor(i, "dkv", rand(R, W))
            m.set_tensor(i, "dkv_norm", np.ones(R, np.float32))
        for name in ("norm1", "norm2"):
            m.set_tensor(i, name, one)
        F = d["ff"]
        mlp = [("gate", F, W), ("up", F, W), ("down", W, F)]
        if "experts" not in d:
            for name, n, k in mlp:
                m.set_tensor(i, name, rand(n, k))
            continue
        m.set_tensor(i, "router", rand(E, W))
        m.set_tensor(i, "router_b", np.zeros(E, np.float32))
        for x in range(E):
            for name, n, k in mlp:
                m.set_expert(i, x, name, rand(n, k))
    return m


def taralix_parts(s):
    """Elements of a layer's linears: attention (mean over the layers), a dense feed-forward as wide as what a token uses,
    the router."""
    W, H, D, R = s["width"], s["heads"], s["dim"], s["rank"]
    return 2 * W * H * D + W * R / 2 + 2 * H * D * R, 3 * W * s["ff"], W * s.get("experts", 0)


def taralix_prefill_flops(s, n):
    a, f, r = taralix_parts(s)
    L, E = s["layers"], s.get("experts", 0)
    return 2 * n * (L * (a + f) + (L - 1) * r) + L * 2 * s["heads"] * s["dim"] * n * (n + 1) + 2 * s["vocab"] * s["width"]


def taralix_decode_bytes(s, batch, ctx):
    a, f, r = taralix_parts(s)
    L, E = s["layers"], s.get("experts", 0)
    moe = f / s["top"] * E * (1 - (1 - s["top"] / E) ** batch) + r if E else f  # the experts that `batch` tokens choose
    return 2 * (L * a + f + (L - 1) * moe) + 2 * s["vocab"] * s["width"] + batch * L * s["rank"] * 2 * ctx


def build(torch, lm, s, max_seqs, max_ctx, max_rows, seed=0):
    """A Vupuzen model of these sizes with random weights made on the device."""
    gen = torch.Generator(device="cuda").manual_seed(seed)
    W, H, G, D, F = s["width"], s["heads"], s["kv"], s["dim"], s["ff"]
    layers = []
    for i in range(s["layers"]):
        base = dict(heads=H, dim=D, vdim=D, ff=F, ff_limit=7.0)
        if i % 4 == 3:
            layers.append(dict(base, mixer=lm.RETENTION, kv_heads=H, rot_dims=D, rot_base=1e6))
        else:
            layers.append(dict(base, mixer=lm.ATTENTION, kv_heads=G, score_scale=D ** -0.5, sink=1, bias_rows=32, bias_max=1024))
    m = lm.LanguageModel(dict(vocab=s["vocab"], width=W, conv_taps=4, max_seqs=max_seqs, max_ctx=max_ctx, max_rows=max_rows, eps=1e-6,
                              logit_scale=1.0), layers)
    rand = lambda n, k: torch.randn((n, k), device="cuda", generator=gen).mul_(k ** -0.5).bfloat16()
    emb = torch.randn((s["vocab"], W), device="cuda", generator=gen).bfloat16()
    m.set_tensor(-1, "embed", emb)
    m.set_tensor(-1, "head", emb[torch.randperm(s["vocab"], device="cuda", generator=gen)])  # greedy decoding walks a permutation
    m.set_tensor(-1, "final_norm", np.float32(1))
    for i, d in enumerate(layers):
        attn = d["mixer"] == lm.ATTENTION
        for name, n, k in [("q", H * D, W), ("k", d["kv_heads"] * D, W), ("v", d["kv_heads"] * D, W), ("o", W, H * D), ("gate", F, W),
                           ("up", F, W), ("down", W, F)] + ([] if attn else [("g", H * D, W)]):
            m.set_tensor(i, name, rand(n, k))
        for name in ("norm1", "norm1b", "norm2", "norm2b"):
            m.set_tensor(i, name, np.float32(0.25 if name.endswith("b") else 1))
        m.set_tensor(i, "conv", np.random.default_rng(i).standard_normal((W, 4)).astype(np.float32) * 0.2)
        if attn:
            m.set_tensor(i, "rel", np.random.default_rng(i).standard_normal((32, H)).astype(np.float32) * 0.3)
        else:
            m.set_tensor(i, "decay", 1.0 - 2.0 ** -(5.0 + np.arange(H) * 8.0 / H))
    return m


def mixer_kinds(s):
    ret = s["layers"] // 4
    return s["layers"] - ret, ret


def linear_weights(s):
    """bf16 weights of all layers' linears, in elements."""
    W, H, G, D, F = s["width"], s["heads"], s["kv"], s["dim"], s["ff"]
    a, r = mixer_kinds(s)
    return a * (W * D * (H + 2 * G) + W * H * D) + r * (4 * W * H * D + W * H * D) + s["layers"] * 3 * W * F


def prefill_flops(s, n):
    H, D = s["heads"], s["dim"]
    a, r = mixer_kinds(s)
    attn = a * 2 * 2 * H * D * n * (n + 1) / 2
    ret = r * 2 * n * H * (2 * 64 / 2 * D + 2 * D * D)
    return 2 * n * linear_weights(s) + attn + ret + 2 * s["vocab"] * s["width"]


def decode_bytes(s, batch, ctx):
    H, G, D = s["heads"], s["kv"], s["dim"]
    a, r = mixer_kinds(s)
    return 2 * linear_weights(s) + 2 * s["vocab"] * s["width"] + batch * (a * 2 * G * D * 2 * ctx + r * 2 * H * D * D * 4)


def event_ms(torch, stream, fn):
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    fn()
    b.record(stream)
    stream.synchronize()
    return a.elapsed_time(b)


def time_engine(torch, lm, s, prompts, batches, ctx, steps, hbm, tflops, make=build, flops=prefill_flops, step_bytes=decode_bytes):
    rows = max(prompts)
    m = make(torch, lm, s, max(batches), max(rows, ctx + steps + 8), rows)
    st, rng, out = m.stream(), np.random.default_rng(1), {"prefill": {}, "decode": {}}
    for n in prompts:
        toks, ms = rng.integers(0, s["vocab"], n).tolist(), []
        for _ in range(5):
            slot = m.acquire()
            ms.append(event_ms(torch, st, lambda: m.step([(slot, toks)], sample=True)))
            m.release(slot)
        t, f = min(ms[1:]), flops(s, n)
        out["prefill"][n] = {"ms": t, "tokens_per_s": n / t * 1e3, "tflops": f / t / 1e9, "frac_bf16": f / t / 1e9 / tflops}
    for b in batches:
        slots = [m.acquire() for _ in range(b)]
        for k, slot in enumerate(slots):
            m.step([(slot, rng.integers(0, s["vocab"], ctx - 5 - k % 7).tolist())], sample=True)
        m.decode(slots, 4)
        ms = min(event_ms(torch, st, lambda: m.decode(slots, steps // 4)) for _ in range(4)) / (steps // 4)
        distinct = len({tuple(m.read(x, ctx - 3, steps).tolist()) for x in slots})
        by = step_bytes(s, b, ctx + steps / 2)
        out["decode"][b] = {"ms_per_step": ms, "tokens_per_s": b / ms * 1e3, "context": ctx, "GBs": by / ms / 1e6,
                            "frac_hbm": by / ms / 1e6 / hbm, "sequences_differ": distinct == b}
        for slot in slots:
            m.release(slot)
    m.check_device_status()
    m.close()
    return out


def time_qwen2(torch, mb, bench, s, prompts, batches, ctx, steps, hbm, tflops):
    H, G, D, W, F = s["heads"], s["kv"], s["dim"], s["width"], s["ff"]
    gen = torch.Generator(device="cuda").manual_seed(3)
    cfg = dict(layers=s["layers"], hidden=W, q_heads=H, kv_heads=G, head_dim=D, inter=F, vocab=s["vocab"],
               max_ctx=max(max(prompts) + 1, ctx + steps + 8), eps=1e-6, rope_theta=1e6)
    dec = mb.Qwen2Decoder(cfg)
    shapes = [("q", W, H * D, True), ("k", W, G * D, True), ("v", W, G * D, True), ("o", H * D, W, False), ("gate", W, F, False),
              ("up", W, F, False), ("down", F, W, False)]
    for i in range(s["layers"]):
        for name, k, n, bias in shapes:
            dec.set_linear_tiled(i, name, bench.make_random_weights(mb, torch, n, k, bias, gen))
        dec.set_norm(0, i, np.ones(W, np.float32))
        dec.set_norm(1, i, np.ones(W, np.float32))
    dec.set_norm(2, 0, np.ones(W, np.float32))
    emb = torch.randn((s["vocab"], W), device="cuda", generator=gen) * 16
    dec.set_tables(emb, (emb * 0.02).half())
    st, rng, out = dec.stream(), np.random.default_rng(1), {"prefill": {}, "decode": {}}
    lin = s["layers"] * sum(n * k for _, k, n, _ in shapes)
    for n in prompts:
        toks = torch.from_numpy(rng.integers(0, s["vocab"], n).astype(np.int32)).cuda()
        torch.cuda.synchronize()
        t = min([event_ms(torch, st, lambda: dec.prefill_device(toks)) for _ in range(5)][1:])
        f = 2 * n * lin + s["layers"] * 2 * H * D * n * (n + 1) + 2 * s["vocab"] * W
        out["prefill"][n] = {"ms": t, "tokens_per_s": n / t * 1e3, "tflops": f / t / 1e9, "frac_bf16": f / t / 1e9 / tflops}

    def entry(ms, b):
        by = lin * 0.5625 + 2 * s["vocab"] * W + b * s["layers"] * 2 * G * D * 4 * (ctx + steps / 2)
        return {"ms_per_step": ms, "tokens_per_s": b / ms * 1e3, "context": ctx, "GBs": by / ms / 1e6, "frac_hbm": by / ms / 1e6 / hbm}

    for b in batches:
        if b == 1:
            dec.prefill(rng.integers(0, s["vocab"], ctx))
            dec.decode(4)
            ms = min(event_ms(torch, st, lambda: dec.decode(steps // 4)) for _ in range(4)) / (steps // 4)
        else:
            try:
                bd = mb.Qwen2BatchDecoder(dec, b)
            except mb.MllmB200Error:  # its batched lm_head holds the activations in shared memory: widths up to about 1700
                out["decode"][b] = None
                continue
            bd.set_policy(5)
            for k in range(b):
                bd.prefill(k, tokens=rng.integers(0, s["vocab"], ctx))
            bd.decode(4)
            ms = min(event_ms(torch, st, lambda: bd.decode(steps // 4)) for _ in range(4)) / (steps // 4)
            bd.close()
        out["decode"][b] = entry(ms, b)
    mb.check_device_status(st)
    dec.close()
    return out


def once(torch, mb, bench, which, size, layers):
    """A short untimed run for a profiler's launch list: one prompt, then a few decode steps."""
    from mllm_b200 import lm
    taralix = size in TARALIX_SIZES and which == "taralix"
    s = dict(TARALIX_SIZES[size] if taralix else SIZES[size], layers=layers, vocab=8192)
    if which != "qwen2":
        m = (build_taralix if taralix else build)(torch, lm, s, 64, 1200, 16384)
        rng = np.random.default_rng(0)
        slots = [m.acquire() for _ in range(64)]
        m.step([(slots[0], rng.integers(0, 8192, 1024).tolist())], sample=True)
        for k in range(1, 64, 16):
            m.step([(x, rng.integers(0, 8192, 1024).tolist()) for x in slots[k:k + 16]], sample=True)
        m.decode(slots, 1)
        m.decode(slots[:1], 1)
        for n, x in zip((128, 512), slots):
            m.release(x)
            m.step([(m.acquire(), rng.integers(0, 8192, n).tolist())], sample=True)
        m.synchronize()
        m.check_device_status()
        m.close()
    else:
        time_qwen2(torch, mb, bench, s, [1024], [1], 1024, 4, 1.0, 1.0)


def run(args, bench):
    import torch
    import mllm_b200 as mb
    from mllm_b200 import lm
    torch.cuda.set_device(0)
    if args.lm_once:
        once(torch, mb, bench, args.lm_once, args.lm_size or "1.5b", 4)
        return {"once": args.lm_once}
    hbm, tflops, kind = bench.measured_peaks()
    prompts, batches, ctx, steps = [128, 512, 2048], [1, 8, 64], 512, 64
    taralix = args.lm_design == "taralix"
    sizes = TARALIX_SIZES if taralix else SIZES
    pair = "Taralix beside Vupuzen" if taralix else "Vupuzen beside Qwen2 W4A32"
    out = {"metric": f"language-model engine, {pair} at equal layer sizes", "unit": "tokens/s", "data": "synthetic",
           "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "kind": kind}, "sizes": {}}
    sampler = bench.ClockSampler(0)
    sampler.start()
    import time
    t0 = time.time()
    for name in [args.lm_size] if args.lm_size else sizes:
        s = sizes[name]
        timing = (prompts, batches, ctx, steps, hbm, tflops)
        if taralix:
            out["sizes"][name] = {"config": s, "taralix": time_engine(torch, lm, s, *timing, build_taralix, taralix_prefill_flops, taralix_decode_bytes)}
            if not args.lm_no_compare:
                out["sizes"][name]["vupuzen"] = time_engine(torch, lm, beside(s), *timing)
            torch.cuda.empty_cache()
            continue
        out["sizes"][name] = {"config": s, "vupuzen": time_engine(torch, lm, s, *timing)}
        torch.cuda.empty_cache()
        if not args.lm_no_compare:
            out["sizes"][name]["qwen2_w4a32"] = time_qwen2(torch, mb, bench, s, prompts, batches, ctx, steps, hbm, tflops)
            torch.cuda.empty_cache()
    out["clocks"] = sampler.summary(t0, time.time())
    sampler.stop()
    return out
