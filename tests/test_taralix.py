"""The Taralix design on the language-model engine, against the plain float64 implementation in oracle/taralix_oracle.py.
The 32-bit mode must agree to fp32 rounding; the bf16 mode within the error of bf16 products, on inputs made so that a
wrong key, latent, expert or gain is far outside of it.  In bf16, tokens whose router is near a tie may go either way and
are left out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "oracle"))

import lm_case  # noqa: E402
import taralix_models as M  # noqa: E402
import taralix_oracle as X  # noqa: E402
from lm_case import BAR, DTYPES, residual_after, row_error  # noqa: E402
from mllm_b200 import lm, registry, taralix  # noqa: E402

gpu = pytest.mark.gpu
GAP = {"float32": 1e-3, "bfloat16": 0.25}


class Case(lm_case.Case):
    def __init__(self, folder, cfg, w, dtype, *sizes, **kw):
        super().__init__(M.write(folder, cfg, w), X, cfg, w, dtype, *sizes, **kw)
        self._known = {}

    def oracle(self, tokens):
        """The same prompts come again and again."""
        key = tuple(tokens)
        if key not in self._known:
            self._known[key] = super().oracle(tokens)
        return self._known[key]

    def sure(self, tokens):
        """Tokens whose choice of experts does not hang on a rounding."""
        key = ("gaps",) + tuple(tokens)
        if key not in self._known:
            self._known[key] = X.router_gaps(self.cfg, self.w, tokens) > GAP[self.dtype]
            assert self._known[key].mean() > 0.6 or len(tokens) < 10
        return self._known[key]

    def same(self, got, tokens, places=None):
        want, sure = self.oracle(tokens), self.sure(tokens)
        if places is not None:
            want, sure = want[places], sure[places]
        if sure.any():
            self.check(got, want, sure)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            cfg = M.MODELS[name]
            made[name, dtype] = Case(tmp_path_factory.mktemp("m"), cfg, M.weights(cfg, 7), dtype)
        return made[name, dtype]

    yield get
    for c in made.values():
        c.model.close()


# ------------------------------------------------------------------------------------------ host side
def test_config_becomes_layer_descriptions():
    d = taralix.layers_from_config(M.MIXED)
    assert all(x["mixer"] == lm.LATENT and x["kv_heads"] == x["heads"] for x in d)
    assert [x["kv_from"] for x in d] == [-1, -1, 0, 0, 1] and [x["kv_rank"] for x in d] == [36, 52, 36, 36, 52]
    assert [x.get("experts", 0) for x in d] == [7, 0, 0, 5, 3] and [x.get("top", 0) for x in d] == [3, 0, 0, 1, 3]
    assert [x.get("ff", 0) for x in d] == [24, 72, 0, 40, 33] and d[1]["act"] == lm.GELU and d[0]["act"] == lm.SILU
    m = taralix.model_config(M.MIXED, 2, 30, 20)
    assert m["residual_scale"] == 1.7 and m["norm_place"] == lm.NORM_POST and m["eps"] == 1e-5 and m["conv_taps"] == 0
    for key, value in (("type", "other"), ("mlp", {"kind": "other"})):
        with pytest.raises(ValueError):
            taralix.layers_from_config(dict(M.MIXED, layers=[dict(M.MIXED["layers"][0], **{key: value})]))


class Recorder:
    def __init__(self):
        self.seen = {}

    def set_tensor(self, layer, name, data):
        self.seen[layer, name] = np.asarray(data)

    def set_expert(self, layer, expert, name, data):
        self.seen[layer, expert, name] = np.asarray(data)


def test_every_tensor_is_loaded_once(tmp_path):
    from mllm_b200.safetensors import Tensors, bf16_to_f32
    w = M.weights(M.MIXED, 3)
    t, r = Tensors(M.write(tmp_path / "m", M.MIXED, w)), Recorder()
    for i, e in enumerate(M.MIXED["layers"]):
        taralix.load_layer(r, t, i, e)
    assert len(r.seen) == len([k for k in w if k.startswith("l")])
    assert np.array_equal(r.seen[0, "norm1"], 1 + w["l0.norm1"]) and np.array_equal(r.seen[0, "dkv_norm"], w["l0.mix.dkv.norm"])
    assert (2, "dkv") not in r.seen and np.array_equal(bf16_to_f32(r.seen[3, 4, "down"]), w["l3.mlp.e4.down"])


def test_registry_knows_the_design(tmp_path, capsys):
    from mllm_b200 import __main__ as cli
    cli.main(["info", "--model", M.write(tmp_path / "m", M.DEEP, M.weights(M.DEEP, 1))])
    assert "Taralix" in capsys.readouterr().out


def test_oracle_routing_and_absorbed_scores():
    """The router's softmax is over the chosen logits alone; scores and outputs through the latent are the same numbers."""
    rng = np.random.default_rng(0)
    idx, p = X.route(np.eye(3), np.array([[0.0, 5, 1], [2, 0, 1], [1, 4, 1]]), np.array([0.5, 0, 0]), 2)  # a row per expert
    assert idx.tolist() == [[1, 2], [0, 2], [0, 1]] and np.allclose(p[0], [1 / (1 + np.exp(-1.0)), 1 / (1 + np.exp(1.0))])
    h, c = rng.standard_normal((6, 10)), rng.standard_normal((6, 5))
    m = M.mixer(2, 4, 3, 5)
    w = {"q": rng.standard_normal((8, 10)), "uk": rng.standard_normal((8, 5)), "uv": rng.standard_normal((6, 5)), "o": np.eye(6)}
    q = (h @ w["q"].T).reshape(6, 2, 4)
    out = []
    for a in range(2):
        uk, uv = w["uk"][4 * a:4 * a + 4], w["uv"][3 * a:3 * a + 3]
        out.append(X.causal_softmax((q[:, a] @ uk) @ c.T * m["scale"]) @ c @ uv.T)
    assert np.allclose(np.concatenate(out, axis=1), X.latent_attention(h, c, w, m))


# ------------------------------------------------------------------------------------------ mechanisms alone
MECHANISMS = {
    "latent": M.config(96, 64, [M.layer(M.mixer(6, 40, 24, 80))]),
    "latent_shared": M.config(96, 64, [M.layer(M.mixer(3, 16, 16, 40)), M.layer(M.mixer(2, 24, 32, 40, kv_from=0))]),
    "dense": M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.dense(88))]),
    "experts": M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.experts(9, 4, 40))]),
    "one_expert": M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.experts(1, 1, 40))]),
    "many_experts": M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.experts(70, 3, 16))]),
    "most_experts": M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.experts(33, 32, 16))]),
    "alpha_zero": M.config(96, 64, [M.layer(M.mixer(2, 16, 16, 48), M.dense(32))], alpha=0.0, eps=0.3),
}


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MECHANISMS))
def test_mechanism_alone(name, dtype, tmp_path):
    cfg = MECHANISMS[name]
    w = M.weights(cfg, 1)
    c = Case(tmp_path / "m", cfg, w, dtype)
    toks, last = c.tokens(350), len(cfg["layers"]) - 1
    _, want = X.forward(cfg, w, toks, want_layers=True)
    x0 = cfg["postln_alpha"] * w["embed"][toks]
    for portions in (None, [70, 2, 1, 1, 76, 200]):
        got = residual_after(c, toks, portions, last)
        e = row_error(got, want[last])[c.sure(toks)]
        assert e.max() < (2e-5 if dtype == "float32" else 0.03), (name, float(e.max()), int(e.argmax()))
    assert row_error(x0 / np.sqrt(np.mean(x0 ** 2 + 1e-9)), want[last]).min() > 0.1  # the sublayers matter
    c.model.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chosen", [0, 11, 12])
def test_all_tokens_to_one_expert(dtype, chosen, tmp_path):
    """Several row tiles of one expert, none of the others."""
    cfg = M.config(96, 64, [M.layer(M.mixer(1, 16, 16, 16), M.experts(13, 1, 40))])
    w = M.weights(cfg, 2, router_std=0.5)
    w["l0.mlp.router.b"] = M.rounded(np.where(np.arange(13) == chosen, 40.0, 0.0))
    c = Case(tmp_path / "m", cfg, w, dtype)
    for n in (1, 3, 5, 64, 128, 129, 400):
        toks = c.tokens(n)
        c.check(c.run(toks), c.oracle(toks))
    c.model.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_in_a_sandwich_of_norms(dtype):
    """The mixture and the latent mixer under the other placement of norms, described to the engine directly."""
    cfg = M.config(96, 64, [M.layer(M.mixer(2, 16, 24, 40), M.experts(6, 2, 40))])
    w = M.weights(cfg, 4)
    gains = {"norm1": 0.9, "norm1b": 1.2, "norm2": 1.1, "norm2b": 0.8}
    m = lm.LanguageModel(dict(vocab=64, width=96, conv_taps=0, eps=1e-5, logit_scale=1.0, max_seqs=2, max_ctx=400, max_rows=400),
                         taralix.layers_from_config(cfg), lm.F32 if dtype == "float32" else lm.BF16)
    from mllm_b200.safetensors import f32_to_bf16 as b
    for n in ("embed", "head"):
        m.set_tensor(-1, n, b(w[n]))
    m.set_tensor(-1, "final_norm", np.float32(1))
    for n, g in gains.items():
        m.set_tensor(0, n, np.float32(g))
    for n in ("q", "uk", "uv", "o", "dkv"):
        m.set_tensor(0, n, b(w["l0.mix." + n]))
    m.set_tensor(0, "dkv_norm", w["l0.mix.dkv.norm"])
    m.set_tensor(0, "router", b(w["l0.mlp.router"]))
    m.set_tensor(0, "router_b", w["l0.mlp.router.b"])
    for e in range(6):
        for n in ("gate", "up", "down"):
            m.set_expert(0, e, n, b(w[f"l0.mlp.e{e}.{n}"]))
    w64 = {k: np.asarray(v, np.float64) for k, v in w.items()}
    mix, mlp = X._part(w64, "l0.mix."), X._part(w64, "l0.mlp.")
    for n in (3, 60, 330):
        toks = np.random.default_rng(n).integers(0, 64, n)
        x = w64["embed"][toks]
        h = X.rms_unit(x, 1e-5) * gains["norm1"]
        x = x + X.rms_unit(X.latent_attention(h, X.latent(h, mix, 1e-5), mix, cfg["layers"][0]["mixer"]), 1e-5) * gains["norm1b"]
        h = X.rms_unit(x, 1e-5) * gains["norm2"]
        z = np.sort(h @ mlp["router"].T + mlp["router.b"], axis=-1)
        sure = z[:, -2] - z[:, -3] > GAP[dtype]
        x = x + X.rms_unit(X.mixture(h, mlp, 2), 1e-5) * gains["norm2b"]
        want = X.rms_unit(x, 1e-5) @ w64["head"].T
        s = m.acquire()
        got = m.step([(s, toks.tolist())], list(range(n)))
        m.release(s)
        assert row_error(got, want)[sure].max() < BAR[dtype]
    m.check_device_status()
    m.close()


# ------------------------------------------------------------------------------------------ whole models
@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_prompt_and_portions(cases, name, dtype):
    c = cases(name, dtype)
    toks = c.tokens(333)
    for portions in (None, [64], [2], [37, 2, 3, 65, 1, 1, 2, 130], [128, 1], [1, 63, 65, 7, 3], [16, 17], [5, 300]):
        c.same(c.run(toks, portions), toks)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_token_by_token_and_first_tokens(cases, name, dtype):
    c = cases(name, dtype)
    toks = c.tokens(90, 2)
    c.same(c.run(toks, [1]), toks)
    for n in (1, 2, 3, 5):
        c.same(c.run(toks[:n]), toks[:n])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "deep", "huge_heads"])
def test_mixed_batches_equal_requests_alone(cases, name, dtype):
    """Prompts, portions and single tokens of unequal requests share steps; freed slots are used again."""
    c = cases(name, dtype)
    rng = np.random.default_rng(11)
    reqs = [c.tokens(n, 20 + n) for n in (150, 67, 3, 129, 1, 88, 200)]
    m, waiting, live, got = c.model, list(range(len(reqs))), {}, [[] for _ in reqs]
    while waiting or live:
        while waiting and len(live) < m.max_seqs:
            live[waiting.pop(0)] = [m.acquire(), 0]
        entries, places, row = [], [], 0
        for i, (slot, at) in live.items():
            n = min(int(rng.choice([1, 1, 2, 3, 16, 17, 64, 65])), len(reqs[i]) - at)
            entries.append((slot, reqs[i][at:at + n]))
            places.append((i, n))
        logits = m.step(entries, list(range(sum(n for _, n in places))))
        for i, n in places:
            got[i].append(logits[row:row + n])
            row += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                m.release(live.pop(i)[0])
    m.check_device_status()
    for g, t in zip(got, reqs):
        c.same(np.concatenate(g), t)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_large_ragged_steps(cases, name, dtype):
    """Steps of several hundred rows in which sequences of one, two and hundreds of tokens meet anywhere."""
    c = cases(name, dtype)
    m = c.model
    sizes = [(1, 2, 310, 1, 40, 3), (2, 1, 5, 290, 1, 17), (150, 150, 1, 3, 2, 2)]
    reqs = [c.tokens(sum(s[i] for s in sizes), 60 + i) for i in range(6)]
    slots, at, got = [m.acquire() for _ in reqs], [0] * 6, [[] for _ in reqs]
    for s in sizes:
        logits, row = m.step([(slots[i], reqs[i][at[i]:at[i] + s[i]]) for i in range(6)], list(range(sum(s)))), 0
        for i in range(6):
            got[i].append(logits[row:row + s[i]])
            row, at[i] = row + s[i], at[i] + s[i]
    for i in range(6):
        m.release(slots[i])
        c.same(np.concatenate(got[i]), reqs[i])
    m.check_device_status()


@gpu
def test_long_contexts_that_do_not_fit_one_expansion(tmp_path):
    """Portions of several long sequences in one step: their keys and values are made in more than one pass."""
    cfg = M.config(64, 50, [M.layer(M.mixer(2, 16, 16, 32), M.dense(48)), M.layer(M.mixer(3, 32, 16, 32, kv_from=0))])
    c = Case(tmp_path / "m", cfg, M.weights(cfg, 3), "bfloat16", max_seqs=5, max_ctx=300, max_rows=120)
    m = c.model
    reqs = [c.tokens(300, 70 + i) for i in range(5)]
    slots, got = [m.acquire() for _ in reqs], [[] for _ in reqs]
    for at in range(0, 300, 20):
        logits = m.step([(s, t[at:at + 20]) for s, t in zip(slots, reqs)], list(range(100)))
        for i in range(5):
            got[i].append(logits[20 * i:20 * i + 20])
    for g, t in zip(got, reqs):
        c.same(np.concatenate(g), t)
    m.check_device_status()
    m.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_only(cases, dtype):
    c = cases("mixed", dtype)
    toks = c.tokens(140, 4)
    s = c.model.acquire()
    places = [139, 0, 64, 63]
    got = c.model.step([(s, toks)], places)
    assert c.model.step([(s, toks[:1])]).shape == (0, c.cfg["vocab"])
    c.model.release(s)
    c.same(got, toks, places)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "deep"])
def test_long_decode(cases, name, dtype):
    """Graph-replayed decoding over the edges of the context splits, against the oracle on the tokens it chose."""
    c = cases(name, dtype)
    m, prompt, steps = c.model, c.tokens(200, 6), 330
    s = m.acquire()
    m.step([(s, prompt)], sample=True)
    m.decode([s], steps)
    out = m.read(s, len(prompt) - 1, steps + 1).tolist()
    logits = m.step([(s, out[-1:])], [0])  # after the last token, with the cache that decoding left
    m.release(s)
    seq = prompt + out
    want = c.oracle(seq)
    c.same(logits, seq, [len(seq) - 1])
    rows = want[len(prompt) - 1:-1]
    if dtype == "float32":
        assert [int(x) for x in np.argmax(rows, axis=1)] == out
    else:  # every sure choice is within the error of the best one
        gap = (rows.max(axis=1) - rows[np.arange(len(out)), out])[c.sure(seq)[len(prompt) - 1:-1]]
        assert gap.max() < 6 * BAR[dtype] * np.sqrt(np.mean(rows ** 2))


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decode_equals_each_alone(cases, dtype):
    """Unequal contexts decode together, then one of them goes on alone."""
    c = cases("wide", dtype)
    m = c.model
    prompts = [c.tokens(n, 80 + n) for n in (3, 64, 65, 170, 255)]
    slots = [m.acquire() for _ in prompts]
    m.step([(s, p) for s, p in zip(slots, prompts)], sample=True)
    m.decode(slots, 9)
    m.decode(slots[2:3], 4)
    for i, (s, p) in enumerate(zip(slots, prompts)):
        out = m.read(s, len(p) - 1, 10 + 4 * (i == 2)).tolist()
        got = m.step([(s, out[-1:])], [0])
        c.same(got, p + out, [len(p) + len(out) - 1])
        if dtype == "float32":
            assert out == X.greedy(c.cfg, c.w, p, len(out))
        m.release(s)


@gpu
def test_greedy_generation_through_the_scheduler(cases):
    c = cases("mixed", "float32")
    prompts = [c.tokens(n, 40 + n) for n in (5, 70, 1, 33, 12, 90, 18)]
    got = registry.generate(c.model, "engine", prompts, 7, portion=32)
    assert got == [X.greedy(c.cfg, c.w, p, 7) for p in prompts]
    assert registry.generate(c.model, "engine", prompts[1:2], 7) == got[1:2]


@gpu
def test_command_line_generates(cases, tmp_path, capsys):
    from mllm_b200 import __main__ as cli
    c = cases("deep", "float32")
    folder = M.write(tmp_path / "m", c.cfg, c.w)
    prompts = [c.tokens(9, 1), c.tokens(4, 2)]
    cli.main(["generate", "--model", folder, "--dtype", "float32", "--max-new", "5"] +
             sum([["--tokens", ",".join(map(str, p))] for p in prompts], []))
    lines = capsys.readouterr().out.split()
    assert [cli.ids(x) for x in lines] == [X.greedy(c.cfg, c.w, p, 5) for p in prompts]


@gpu
def test_trace_runner_program(cases, tmp_path):
    c = cases("mixed", "float32")
    folder = M.write(tmp_path / "m", c.cfg, c.w)
    a, b = c.tokens(50, 1), c.tokens(20, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[33:], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b, "want": [19]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "50"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0 and p.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"], p.stderr[-500:]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    read = lambda n: np.fromfile(out / f"{n}.f32", "<f4").reshape(-1, c.cfg["vocab"])
    c.same(read(0), a, [0, 32])
    c.same(read(2), b, [19])


# ------------------------------------------------------------------------------------------ one key that matters
NEEDLE, ASK, FILL = 1, 2, 3


def needle_model(heads, dim, vdim, rank, shared=False, score=12.0):
    """Tokens have latents in directions of their own; only ASK has a query, along the key of NEEDLE, whose score stands
    out among hundreds of fill tokens' zeros."""
    layers = [M.layer(M.mixer(heads, dim, vdim, rank, scale=0.25))]
    if shared:
        layers.append(M.layer(M.mixer(heads, dim, vdim, rank, scale=0.25, kv_from=0)))
    cfg = M.config(64, 8, layers, alpha=1.0)
    w = M.weights(cfg, 9)
    rng = np.random.default_rng(3)
    e, dkv = np.zeros((8, 64)), np.zeros((rank, 64))
    for t in range(8):
        e[t, t] = 4.0
        dkv[t, t] = 1.0
    size = np.sqrt(rank)  # of the one coordinate of a latent after its norm
    w.update({"embed": M.rounded(e), "l0.mix.dkv": M.rounded(dkv), "l0.mix.dkv.norm": np.ones(rank, np.float32)})
    for i in range(len(layers)):
        q, uk = np.zeros((heads * dim, 64)), np.zeros((heads * dim, rank))
        for h in range(heads):
            q[h * dim + h % dim, ASK] = 1.0
            uk[h * dim + h % dim, NEEDLE] = score / 0.25 / 4.0 / size
        uv = rng.standard_normal((heads * vdim, rank)) / size * 2
        w.update({f"l{i}.mix.q": M.rounded(q), f"l{i}.mix.uk": M.rounded(uk), f"l{i}.mix.uv": M.rounded(uv), f"l{i}.norm1": np.zeros(64, np.float32)})
    return cfg, w


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rank,shared", [(4, 32, 24, 48, False), (17, 16, 16, 200, False), (2, 64, 40, 72, True), (3, 16, 16, 256, False),
                                                         (3, 16, 16, 512, False), (1, 16, 16, 640, False), (2, 16, 16, 1024, False)])
def test_one_far_key_at_every_distance(dtype, heads, dim, vdim, rank, shared, tmp_path):
    """NEEDLE at distances around key blocks, row tiles and context splits; ASK in a prompt, in a short portion, and
    decoded; a second NEEDLE right behind ASK must not be seen."""
    cfg, w = needle_model(heads, dim, vdim, rank, shared)
    c = Case(tmp_path / "m", cfg, w, dtype, max_ctx=1100, max_rows=1100)
    blind = c.oracle([FILL] * 300 + [ASK])[-1:]
    for n in (1, 2, 15, 16, 17, 31, 32, 33, 63, 64, 65, 127, 128, 129, 255, 256, 257, 300, 511, 513, 700, 1030):
        for before in (0, 1, 40):
            toks = [FILL] * before + [NEEDLE] + [FILL] * (n - 1) + [ASK]
            want = c.oracle(toks)[-1:]
            assert row_error(want, blind).min() > 3 * BAR["bfloat16"]
            for portions in (None, [len(toks) - 1, 1], [max(1, len(toks) - 3), 3]):
                c.check(c.run(toks, portions)[-1:], want)
    for n in (1, 15, 16, 62, 63, 64, 127, 300):
        toks = [FILL] * n + [ASK, NEEDLE, NEEDLE] + [FILL] * 30
        want = c.oracle(toks)
        for portions in (None, [n, 2, 40], [n + 1, 1], [n + 2, 40]):
            c.check(c.run(toks, portions), want)
    c.model.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_leave_no_trace(dtype, tmp_path):
    """A slot that held needles is used again by a sequence without; neighbours in a step do not see each other."""
    cfg, w = needle_model(3, 16, 24, 40)
    c = Case(tmp_path / "m", cfg, w, dtype, max_seqs=2, max_ctx=400, max_rows=800)
    m = c.model
    for n in (5, 64, 130, 300):
        a, b = m.acquire(), m.acquire()
        m.step([(a, [NEEDLE] * n), (b, [FILL] * n)])
        got = m.step([(a, [ASK]), (b, [ASK])], [0, 1])
        c.check(got[:1], c.oracle([NEEDLE] * n + [ASK])[-1:])
        c.check(got[1:], c.oracle([FILL] * n + [ASK])[-1:])
        m.release(a)
        m.release(b)
        toks = [FILL] * (n // 2) + [ASK] + [FILL] * 20 + [ASK]
        c.check(c.run(toks), c.oracle(toks))
        c.check(c.run(toks, [1]), c.oracle(toks))
    m.close()


# ------------------------------------------------------------------------------------------ linears, errors
@gpu
def test_row_counts_around_every_kernels_limits(tmp_path):
    """One to four rows, padded tiles, several tiles, K splits, the router inside and behind the norm; sizes that leave
    partial tiles on every side."""
    cfg = M.config(328, 523, [M.layer(M.mixer(5, 48, 72, 136), M.experts(11, 3, 200))])
    c = Case(tmp_path / "m", cfg, M.weights(cfg, 5), "bfloat16", max_ctx=700, max_rows=700)
    toks = c.tokens(650)
    want, sure = c.oracle(toks), c.sure(toks)
    for n in (1, 2, 3, 4, 5, 15, 16, 17, 63, 64, 65, 127, 128, 129, 255, 257, 296, 297, 389, 650):
        c.check(c.run(toks[:n]), want[:n], sure[:n])
    c.model.close()


@gpu
def test_errors_come_back_as_statuses(tmp_path):
    sizes = (1, 8, 8)
    make = lambda *layers: lm.LanguageModel(taralix.model_config(M.config(64, 8, []), *sizes), taralix.layers_from_config({"layers": list(layers)}))
    own, bad = M.mixer(2, 16, 16, 32), []
    bad.append([M.layer(dict(own, kv_from=0))])                          # no layer before it
    bad.append([M.layer(own), M.layer(dict(own, kv_rank=16, kv_from=0))])  # another size
    bad.append([M.layer(own), M.layer(dict(own, kv_from=0)), M.layer(dict(own, kv_from=1))])  # layer 1 has no rows of its own
    bad.append([M.layer(own, M.experts(4, 5, 16))])
    bad.append([M.layer(own, M.experts(4, 0, 16))])
    for layers in bad:
        with pytest.raises(lm.EngineError):
            make(*layers)
    m = make(M.layer(own, M.experts(4, 2, 16)), M.layer(dict(own, kv_from=0), M.dense(16)))
    s = m.acquire()
    with pytest.raises(lm.EngineError):
        m.step([(s, [0])])  # nothing loaded
    for call in (lambda: m.set_tensor(0, "k", np.zeros((32, 64), np.uint16)), lambda: m.set_tensor(1, "dkv", np.zeros((32, 64), np.uint16)),
                 lambda: m.set_tensor(0, "gate", np.zeros((16, 64), np.uint16)), lambda: m.set_expert(0, 4, "gate", np.zeros((16, 64), np.uint16)),
                 lambda: m.set_expert(0, 0, "down", np.zeros((16, 64), np.uint16)), lambda: m.set_tensor(0, "norm1b", np.zeros(64, np.float32)),
                 lambda: m.set_expert(1, 0, "gate", np.zeros((16, 64), np.uint16))):
        with pytest.raises(lm.EngineError):
            call()
    m.close()
