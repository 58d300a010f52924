"""What the tests of the language-model engine share: a model on the GPU beside its oracle, and error bars."""
import numpy as np

from mllm_b200 import registry

# relative rms error of a row of logits; bf16: a few roundings of 2^-9 per layer.  One row in fifty may reach OUTLIER:
# a head or a residual row that happens to be small enlarges the roundings.
BAR = {"float32": 3e-5, "bfloat16": 0.06}
OUTLIER = {"float32": 1e-4, "bfloat16": 0.2}
DTYPES = ["float32", "bfloat16"]


def row_error(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want ** 2))


class Case:
    """A model on the GPU (read from `folder`) and in the oracle."""

    def __init__(self, folder, oracle, cfg, w, dtype, max_seqs=6, max_ctx=1024, max_rows=1024):
        self.cfg, self.w, self.dtype, self._oracle = cfg, w, dtype, oracle
        self.model, runtime = registry.load(str(folder), dtype, max_seqs, max_ctx, max_rows)
        assert runtime == "engine"

    def oracle(self, tokens):
        return self._oracle.forward(self.cfg, self.w, tokens)

    def tokens(self, n, seed=0):
        return np.random.default_rng(seed + 1000).integers(0, self.cfg["vocab"], n).tolist()

    def run(self, tokens, portions=None, slot=None):
        """Logits of every place, read in the given portions (the last one is repeated)."""
        own = slot is None
        slot = self.model.acquire() if own else slot
        out, at, k = [], 0, 0
        portions = portions or [len(tokens)]
        while at < len(tokens):
            n = min(portions[min(k, len(portions) - 1)], len(tokens) - at)
            out.append(self.model.step([(slot, tokens[at:at + n])], list(range(n))))
            at, k = at + n, k + 1
        if own:
            self.model.release(slot)
        self.model.check_device_status()
        return np.concatenate(out)

    def check(self, got, want, rows=None):
        """rows: which of them count (default all)."""
        e = row_error(got, want)
        e = e if rows is None else e[rows]
        over = int((e >= BAR[self.dtype]).sum())
        assert over <= len(e) // 50 and e.max() < OUTLIER[self.dtype], (float(e.max()), int(e.argmax()), over, len(e))


def residual_after(case, tokens, portions=None, layer=0):
    """Residual stream after a layer, per token."""
    m, out, at = case.model, [], 0
    slot = m.acquire()
    m.keep_residual(True)
    for n in portions or [len(tokens)]:
        m.step([(slot, tokens[at:at + n])])
        out.append(m.residual(layer, n))
        at += n
    m.keep_residual(False)
    m.release(slot)
    assert at == len(tokens)
    return np.concatenate(out)
