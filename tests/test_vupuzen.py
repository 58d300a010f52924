"""The Vupuzen design on the language-model engine, against the plain float64 implementation in oracle/vupuzen_oracle.py.
The 32-bit mode must agree to fp32 rounding; the bf16 mode within the error of bf16 products, on inputs made so that a
wrong key, bias row, tap, state or sink is far outside of it."""
import os
import sys

import numpy as np
import pytest

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, os.path.join(ROOT, "oracle"))

import lm_case  # noqa: E402
import lm_models as M  # noqa: E402
import vupuzen_oracle as V  # noqa: E402
from lm_case import BAR, DTYPES, residual_after, row_error  # noqa: E402
from mllm_b200 import lm, registry, replay, scheduler  # noqa: E402

gpu = pytest.mark.gpu


class Case(lm_case.Case):
    def __init__(self, folder, cfg, w, dtype, *sizes, **kw):
        super().__init__(M.write(folder, cfg, w), V, cfg, w, dtype, *sizes, **kw)


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
def test_distance_buckets_match_the_definition():
    for rows, largest in ((32, 128), (10, 37), (2, 5), (64, 4096), (9, 100), (16, 256)):
        want = [V.distance_bucket(n, rows, largest) for n in range(largest + 40)]
        assert lm.distance_buckets(rows, largest, largest + 40).tolist() == want
        assert want[0] == 0 and want[largest] == rows - 1 and max(want) == rows - 1 and sorted(want) == want
    # powers of two of a power-of-two table lie exactly on its edges
    b = lm.distance_buckets(16, 128, 129)
    assert b[16] == b[15] + 1 and b[32] == b[31] + 1 and b[64] == b[63] + 1


def test_config_becomes_layer_descriptions(tmp_path):
    from mllm_b200 import vupuzen
    d = vupuzen.layers_from_config(M.MIXED, lambda i: 10)
    assert [x["mixer"] for x in d] == [lm.RETENTION, lm.ATTENTION, lm.ATTENTION, lm.RETENTION, lm.ATTENTION]
    assert [x["weights_of"] for x in d] == [-1, -1, -1, 0, 1]
    assert "ff" not in d[1] and d[2]["ff_limit"] == 0.6 and d[0]["rot_dims"] == 12
    bad = M.config(64, 10, [M.layer("attention", M.attention(2, 1, 16, 16, 20))])
    for key, value in (("type", "other"), ("mlp", {"kind": "mixture", "ff": 8, "limit": 1.0})):
        broken = dict(bad, layers=[dict(bad["layers"][0], **{key: value})])
        with pytest.raises(ValueError):
            vupuzen.layers_from_config(broken, lambda i: 10)
    with pytest.raises(ValueError):
        registry.architecture({"architecture": "Unknown"})


def test_safetensors_round_trip(tmp_path):
    from mllm_b200.safetensors import Tensors
    w = M.weights(M.MIXED, 3)
    t = Tensors(M.write(tmp_path / "m", M.MIXED, w))
    assert set(t.names()) == set(w)
    for k, v in w.items():
        assert t.shape(k) == np.shape(v) and np.array_equal(t.f32(k), v)


class FakeModel:
    """Next token = (last token + number of tokens read) mod 50; records its steps."""

    def __init__(self, max_seqs, max_ctx, max_rows):
        self.max_seqs, self.max_ctx, self.max_rows, self.vocab = max_seqs, max_ctx, max_rows, 4
        self.length, self.seen, self.hist, self.steps = [0] * max_seqs, [[] for _ in range(max_seqs)], {}, []
        self.free = list(range(max_seqs))

    def acquire(self):
        return self.free.pop(0) if self.free else None

    def release(self, s):
        self.length[s], self.seen[s] = 0, []
        self.free.append(s)

    def step(self, entries, want=(), sample=False):
        assert sum(len(t) for _, t in entries) <= self.max_rows and len({s for s, _ in entries}) == len(entries)
        self.steps.append([len(t) for _, t in entries])
        rows = []
        for s, t in entries:
            assert len(t) > 0
            for x in t:
                self.seen[s].append(x)
                rows.append([x, self.length[s], s, 0])
                self.length[s] += 1
            self.hist[s, self.length[s] - 1] = (t[-1] + self.length[s]) % 50
        return np.asarray([rows[k] for k in want], np.float32).reshape(len(want), 4)

    def decode(self, slots, steps):
        for s in slots:
            for _ in range(steps):
                self.step([(s, [self.hist[s, self.length[s] - 1]])])

    def read(self, s, first, count):
        return np.array([self.hist[s, first + i] for i in range(count)])


def fake_reference(prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append((seq[-1] + len(seq)) % 50)
    return seq[len(prompt):]


def test_scheduler_batches_portions_and_reuses_slots():
    rng = np.random.default_rng(5)
    m = FakeModel(3, 64, 16)
    prompts = [rng.integers(0, 50, n).tolist() for n in (1, 30, 7, 16, 2, 41, 3)]
    s = scheduler.Scheduler(m, portion=9)
    reqs = [s.submit(p, 3 + 2 * i) for i, p in enumerate(prompts)]
    s.run()
    for i, (r, p) in enumerate(zip(reqs, prompts)):
        assert r.output == fake_reference(p, 3 + 2 * i)
    assert sorted(m.free) == [0, 1, 2]
    assert any(len(x) > 1 and max(x) > 1 and min(x) == 1 for x in m.steps)  # a token and a portion in one step
    stop = fake_reference(prompts[2], 9)[4]
    out = scheduler.generate(m, [prompts[2]], 30, stop={stop})[0]
    assert out == fake_reference(prompts[2], 30)[:len(out)] and out[-1] == stop and stop not in out[:-1]
    with pytest.raises(ValueError):
        s.submit([1] * 60, 10)


def test_replay_cuts_long_steps_and_keeps_the_order():
    m = FakeModel(2, 64, 5)
    r = replay.Replay(m)
    got = r.step([{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}, {"id": "b", "tokens": list(range(10, 19)), "want": [8, 3, 0]}])
    assert got[:, 0].tolist() == [3, 1, 18, 13, 10] and got[:, 1].tolist() == [2, 0, 8, 3, 0]
    got = r.step([{"id": "a", "tokens": [7], "want": [0]}], end=["b"])
    assert got[0, 1] == 3 and list(r.slots) == ["a"]
    r.step([{"id": "c", "tokens": [4], "want": []}])
    with pytest.raises(RuntimeError):
        r.step([{"id": "d", "tokens": [4]}])


def test_command_line_arguments():
    from mllm_b200 import __main__ as cli
    a = cli.parser().parse_args(["generate", "--model", "x", "--tokens", "1,2", "--tokens", "3", "--max-new", "4"])
    assert [cli.ids(t) for t in a.tokens] == [[1, 2], [3]]
    a = cli.parser().parse_args(["trace", "--model", "x", "--out", "o", "--max-tokens", "9"])
    assert a.dtype == "bfloat16" and a.max_tokens == 9


def test_oracle_retention_forms_agree():
    """The recurrence against the sum over all earlier tokens it stands for."""
    rng = np.random.default_rng(0)
    q, k, v = (rng.standard_normal((9, 2, d)) for d in (6, 6, 5))
    o, S = V.retention_recurrence(q, k, v, [0.5, 0.9])
    for h, g in enumerate((0.5, 0.9)):
        a = np.tril((q[:, h] @ k[:, h].T) * g ** np.maximum(np.arange(9)[:, None] - np.arange(9), 0))
        assert np.allclose(a @ v[:, h], o[:, h])


# ------------------------------------------------------------------------------------------ mechanisms alone
def one_layer(kind, mixer, ff=None, taps=1, width=96, vocab=64, seed=1, conv=0.0, rel_rows=10, **kw):
    cfg = M.config(width, vocab, [M.layer(kind, mixer, ff, **kw)], taps=taps)
    w = M.weights(cfg, seed, rel_rows=rel_rows)
    w["l0.canon1"] = M.rounded(np.random.default_rng(seed).standard_normal((width, taps)) * conv)
    return cfg, w


MECHANISMS = {
    "attention": one_layer("attention", M.attention(6, 3, 40, 24, 33)),
    "retention": one_layer("retention", M.retention(3, 24, 40, 16, [0.7, 0.95, 0.999])),
    "retention_unrotated": one_layer("retention", M.retention(2, 16, 16, 0, [0.9, 0.99])),
    "convolution": one_layer("retention", M.retention(1, 16, 16, 16, [0.9]), taps=6, conv=1.0),
    "feed_forward": one_layer("retention", M.retention(1, 16, 16, 16, [0.9]), ff=88, limit=0.4),
    "feed_forward_unclamped": one_layer("attention", M.attention(2, 2, 16, 16, 33), ff=32, limit=50.0),
}


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(MECHANISMS))
def test_mechanism_alone(name, dtype, tmp_path):
    cfg, w = MECHANISMS[name]
    c = Case(tmp_path / "m", cfg, w, dtype)
    toks = c.tokens(150)
    _, want = V.forward(cfg, w, toks, want_layers=True)
    x0 = w["embed"][toks]
    for portions in (None, [70, 2, 1, 1, 76]):
        e = row_error(residual_after(c, toks, portions) - x0, want[0] - x0)
        assert e.max() < (2e-5 if dtype == "float32" else 0.03), (name, float(e.max()), int(e.argmax()))
    c.model.close()


# ------------------------------------------------------------------------------------------ whole models
@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_prompt_and_portions(cases, name, dtype):
    c = cases(name, dtype)
    toks = c.tokens(333)
    want = c.oracle(toks)
    for portions in (None, [64], [2], [37, 2, 3, 65, 1, 1, 2, 130], [128, 1], [1, 63, 65, 7, 3], [5, 300]):
        c.check(c.run(toks, portions), want)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_token_by_token_and_first_tokens(cases, name, dtype):
    c = cases(name, dtype)
    toks = c.tokens(90, 2)
    want = c.oracle(toks)
    c.check(c.run(toks, [1]), want)
    for n in (1, 2, 3, 5):
        c.check(c.run(toks[:n]), want[:n])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "deep_conv"])
def test_mixed_batches_equal_requests_alone(cases, name, dtype):
    """Prompts, portions and single tokens of unequal requests share steps; freed slots are used again."""
    c = cases(name, dtype)
    rng = np.random.default_rng(11)
    reqs = [c.tokens(n, 20 + n) for n in (150, 67, 3, 129, 1, 88, 200)]
    want = [c.oracle(t) for t in reqs]
    m, waiting, live, got = c.model, list(range(len(reqs))), {}, [[] for _ in reqs]
    while waiting or live:
        while waiting and len(live) < m.max_seqs:
            live[waiting.pop(0)] = [m.acquire(), 0]
        entries, places, row = [], [], 0
        for i, (slot, at) in live.items():
            n = min(int(rng.choice([1, 1, 2, 3, 40, 64, 65])), len(reqs[i]) - at)
            entries.append((slot, reqs[i][at:at + n]))
            places.append((i, n))
        logits = m.step(entries, list(range(sum(n for _, n in places))))
        for i, n in places:
            got[i].append(logits[row:row + n])
            row += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                m.release(live.pop(i)[0])
    for g, w in zip(got, want):
        c.check(np.concatenate(g), w)


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.MODELS))
def test_large_ragged_steps(cases, name, dtype):
    """Steps of several hundred rows in which sequences of one, two and hundreds of tokens meet anywhere."""
    c = cases(name, dtype)
    m = c.model
    sizes = [(1, 2, 310, 1, 40, 3), (2, 1, 5, 290, 1, 17), (150, 150, 1, 3, 2, 2)]
    reqs = [c.tokens(sum(s[i] for s in sizes), 60 + i) for i in range(6)]
    want = [c.oracle(t) for t in reqs]
    slots, at, got = [m.acquire() for _ in reqs], [0] * 6, [[] for _ in reqs]
    for s in sizes:
        logits, row = m.step([(slots[i], reqs[i][at[i]:at[i] + s[i]]) for i in range(6)], list(range(sum(s)))), 0
        for i in range(6):
            got[i].append(logits[row:row + s[i]])
            row, at[i] = row + s[i], at[i] + s[i]
    for i in range(6):
        m.release(slots[i])
        c.check(np.concatenate(got[i]), want[i])
    m.check_device_status()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_only(cases, dtype):
    c = cases("mixed", dtype)
    toks = c.tokens(140, 4)
    want = c.oracle(toks)
    s = c.model.acquire()
    places = [139, 0, 64, 63]
    got = c.model.step([(s, toks)], places)
    assert c.model.step([(s, toks[:1])]).shape == (0, c.cfg["vocab"])
    c.model.release(s)
    c.check(got, want[places])


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decode(cases, dtype):
    """Graph-replayed decoding over the edges of the context splits, against the oracle on the tokens it chose."""
    c = cases("deep_conv", dtype)
    m, prompt, steps = c.model, c.tokens(200, 6), 330
    s = m.acquire()
    m.step([(s, prompt)], sample=True)
    m.decode([s], steps)
    out = m.read(s, len(prompt) - 1, steps + 1).tolist()
    logits = m.step([(s, out[-1:])], [0])  # after the last token, with the state that decoding left
    m.release(s)
    seq = prompt + out
    want = c.oracle(seq)
    c.check(logits, want[-1:])
    if dtype == "float32":
        assert [int(x) for x in np.argmax(want[len(prompt) - 1:-1], axis=1)] == out
    else:  # every choice is within the error of the best one
        rows = want[len(prompt) - 1:-1]
        gap = rows.max(axis=1) - rows[np.arange(len(out)), out]
        assert gap.max() < 6 * BAR[dtype] * np.sqrt(np.mean(rows ** 2))


@gpu
def test_greedy_generation_through_the_scheduler(cases):
    c = cases("mixed", "float32")
    prompts = [c.tokens(n, 40 + n) for n in (5, 70, 1, 33, 12, 90)]
    got = registry.generate(c.model, "engine", prompts, 7, portion=32)
    assert got == [V.greedy(c.cfg, c.w, p, 7) for p in prompts]
    assert registry.generate(c.model, "engine", prompts[1:2], 7) == got[1:2]


@gpu
def test_command_line_generates(cases, tmp_path, capsys):
    from mllm_b200 import __main__ as cli
    c = cases("deep_conv", "float32")
    folder = M.write(tmp_path / "m", c.cfg, c.w)
    prompts = [c.tokens(9, 1), c.tokens(4, 2)]
    cli.main(["generate", "--model", folder, "--dtype", "float32", "--max-new", "5"] +
             sum([["--tokens", ",".join(map(str, p))] for p in prompts], []))
    lines = capsys.readouterr().out.split()
    assert [cli.ids(x) for x in lines] == [V.greedy(c.cfg, c.w, p, 5) for p in prompts]


@gpu
def test_trace_runner_program(cases, tmp_path):
    import json
    import subprocess
    c = cases("mixed", "bfloat16")
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
    assert row_error(read(0), c.oracle(a)[[0, 32]]).max() < BAR["float32"]
    assert row_error(read(2), c.oracle(b)[[19]]).max() < BAR["float32"]


# ------------------------------------------------------------------------------------------ one key that matters
NEEDLE, ASK, FILL = 1, 2, 3


def needle_model(bias_rows, bias_max, heads=4, kv=2, dim=32, vdim=24, strength=9.0):
    """One attention layer in which only NEEDLE has a key and only ASK has a query, along one direction per head; fill
    tokens have neither.  The bias differs much between neighbouring rows, so ASK's result tells NEEDLE's distance."""
    cfg = M.config(64, 8, [M.layer("attention", M.attention(heads, kv, dim, vdim, bias_max, scale=0.25))], taps=1, logit_scale=1.0)
    w = M.weights(cfg, 9, rel_rows=bias_rows)
    rng = np.random.default_rng(3)
    e = np.zeros((8, 64))
    for t in range(8):
        e[t, t] = 8.0  # after the norm: one large coordinate per token
    q, k, v = np.zeros((heads * dim, 64)), np.zeros((kv * dim, 64)), np.zeros((kv * vdim, 64))
    for h in range(heads):
        q[h * dim + h // (heads // kv), ASK] = strength ** 0.5 / 8 * 2
    for g in range(kv):
        k[g * dim + g, NEEDLE] = strength ** 0.5 / 8 * 2
        v[g * vdim:(g + 1) * vdim, NEEDLE] = rng.standard_normal(vdim)
    # a matching score is 9: nearly all of the weight in the rows of bias 0, next to none in those of -14
    rel = np.where(np.arange(bias_rows)[:, None] % 2 == 1, 0.0, -14.0) - np.arange(bias_rows)[:, None] * 0.11 + np.arange(heads) * 0.3
    w.update({"embed": M.rounded(e), "l0.mix.q": M.rounded(q), "l0.mix.k": M.rounded(k), "l0.mix.v": M.rounded(v),
              "l0.mix.rel": M.rounded(rel), "l0.canon1": np.zeros((64, 1), np.float32), "l0.norm1": np.float32(1), "l0.norm1b": np.float32(1)})
    return cfg, w


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv", [(4, 2), (3, 3), (6, 1)])
def test_one_far_key_at_every_edge(dtype, heads, kv, tmp_path):
    """NEEDLE at distances around bias rows, key blocks and context splits; ASK in a prompt, in a short portion, and
    decoded.  The norm after the mixer would hide the size of the output, so the mixed direction carries a constant:
    fill tokens have a value too."""
    rows, largest = 12, 90
    cfg, w = needle_model(rows, largest, heads, kv)
    v = w["l0.mix.v"].copy()
    v[:, FILL] = np.random.default_rng(5).standard_normal(v.shape[0])
    w["l0.mix.v"] = M.rounded(v)
    c = Case(tmp_path / "m", cfg, w, dtype, max_ctx=640, max_rows=640)
    b = lm.distance_buckets(rows, largest, largest + 2)
    b_at = lambda n: b[min(n, largest)]
    edges = [n for n in range(1, largest + 1) if b[n] != b[n - 1]]
    distances = sorted(({n + d for n in edges for d in (-1, 0)} | {63, 64, 65, 127, 128, 255, 256, 257, 300, 511, 513}) - {0})
    seen = []
    for n in distances:
        for tail in (0, 1):
            toks = [FILL] * tail + [NEEDLE] + [FILL] * (n - 1) + [ASK]
            want = c.oracle(toks)[-1:]
            if tail == 0:
                seen.append((want[0], n))
            for portions in (None, [len(toks) - 1, 1], [max(1, len(toks) - 3), 3]):
                c.check(c.run(toks, portions)[-1:], want)
    moves = [row_error(a, b) for (a, m), (b, n) in zip(seen, seen[1:]) if n - m == 1 and b_at(n) != b_at(m)]
    assert min(moves) > 3 * BAR["bfloat16"]  # the bias row next to the right one shows
    c.model.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_sink_takes_weight(dtype, tmp_path):
    """Scores far below 0: nearly all weight is the sink's; without it the output would be a mean of values.  The
    post-norm's eps is large, so that the size of the mixed output is seen."""
    cfg, w = needle_model(4, 40)
    cfg = dict(cfg, norm={"eps": 1.0})
    w["l0.mix.rel"] = np.full_like(w["l0.mix.rel"], -6.0)
    c = Case(tmp_path / "m", cfg, w, dtype)
    toks = [NEEDLE] * 5 + [FILL] * 4 + [NEEDLE] * 90
    want = c.oracle(toks)
    for portions in (None, [50, 1]):
        c.check(c.run(toks, portions), want)
    x0 = w["embed"][toks]
    got = residual_after(c, toks) - x0
    _, layers = V.forward(cfg, w, toks, want_layers=True)
    assert row_error(got, layers[0] - x0).max() < BAR[dtype]
    size = np.abs(layers[0] - x0).max(axis=1)
    assert size[0] < 0.2 * size[-1]  # the sink's share shrinks as keys arrive
    c.model.close()


@gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_state_survives_far_and_is_not_shared(dtype, tmp_path):
    """Retention without decay: one early token decides the result hundreds of tokens later; another sequence in the
    same step, and one that had the slot before, leave no trace."""
    cfg = M.config(64, 8, [M.layer("retention", M.retention(2, 32, 16, 16, [1.0, 0.9995]))], taps=1)
    w = M.weights(cfg, 21)
    e = np.zeros((8, 64))
    for t in range(8):
        e[t, t] = 8.0
    w["embed"], w["l0.canon1"] = M.rounded(e), np.zeros((64, 1), np.float32)
    k = w["l0.mix.k"].copy()
    k[:, FILL] = 0.0  # fill tokens write nothing
    w["l0.mix.k"] = k
    c = Case(tmp_path / "m", cfg, w, dtype, max_ctx=700, max_rows=700)
    m = c.model
    for n in (63, 64, 65, 127, 128, 300, 513):
        toks = [NEEDLE] + [FILL] * (n - 1) + [ASK]
        other = [ASK, NEEDLE, 5] * 30
        want, want_o = c.oracle(toks)[-1:], c.oracle(other)[-1:]
        for portions in (None, [n - 1, 1, 1], [2, n - 1]):
            c.check(c.run(toks, portions)[-1:], want)
        a, b = m.acquire(), m.acquire()
        m.step([(b, other[:40]), (a, toks[:n // 2])])
        got = m.step([(a, toks[n // 2:]), (b, other[40:])], [n + 1 - n // 2 - 1, n + 1 - n // 2 + len(other) - 41])
        c.check(got[:1], want)
        c.check(got[1:], want_o)
        m.release(a)
        m.release(b)
    c.model.close()


# ------------------------------------------------------------------------------------------ linears
@gpu
def test_tensor_core_linears_at_many_row_counts(tmp_path):
    """Row counts around every kernel's limits (one to four rows, padded tiles, several tiles, K splits), sizes that
    leave partial tiles on every side."""
    cfg = M.config(328, 523, [M.layer("attention", M.attention(5, 5, 48, 72, 33), 1000)], taps=2)
    w = M.weights(cfg, 5)
    c = Case(tmp_path / "m", cfg, w, "bfloat16", max_ctx=400, max_rows=400)
    toks = c.tokens(389)
    want = c.oracle(toks)
    for n in (1, 2, 3, 4, 5, 15, 16, 17, 63, 64, 65, 127, 128, 129, 255, 256, 257, 389):
        c.check(c.run(toks[:n]), want[:n])
    c.model.close()


@gpu
def test_errors_come_back_as_statuses(cases):
    m = cases("mixed", "float32").model
    s = m.acquire()
    for entries, want in (([(s, [m.vocab])], ()), ([(s, [0]), (s, [1])], ()), ([(99, [0])], ()), ([(s, [0])], [1])):
        with pytest.raises(lm.EngineError):
            m.step(entries, want)
    with pytest.raises(lm.EngineError):
        m.decode([s], 1)  # no current token
    with pytest.raises(lm.EngineError):
        m.step([(s, [0] * (m.max_rows + 1))])
    m.length[s] = 0
    m.release(s)
    with pytest.raises(lm.EngineError):
        m.set_tensor(0, "q", np.zeros((3, 5), np.uint16))
    cfg = M.config(64, 8, [M.layer("attention", M.attention(3, 2, 16, 16, 20))])
    from mllm_b200 import vupuzen
    with pytest.raises(lm.EngineError):
        lm.LanguageModel(vupuzen.model_config(cfg, 1, 8, 8), vupuzen.layers_from_config(cfg, lambda i: 10))
