"""Replays a trace of steps on a model: given token ids in, logits out, nothing sampled.

A step is one JSON object a line, {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  The logits of the
wanted places go to <out>/<n>.f32 (little-endian fp32 [wanted, vocab], in the order of entries and places), then a line
"done <n>" is printed."""
import json
import os

import numpy as np


class Replay:
    def __init__(self, model):
        self.model, self.slots = model, {}

    def step(self, entries, end=()):
        """Logits of the wanted places.  A step longer than the model's max_rows is cut."""
        m, todo, n_out = self.model, [], 0
        for e in entries:
            places = [(p, n_out + k) for k, p in enumerate(e.get("want", ()))]  # place, row of the result
            n_out += len(places)
            if e["tokens"]:
                if e["id"] not in self.slots:
                    slot = m.acquire()
                    if slot is None:
                        raise RuntimeError(f"more than {m.max_seqs} requests at once")
                    self.slots[e["id"]] = slot
                todo.append((self.slots[e["id"]], e["tokens"], places))
        out = np.zeros((n_out, m.vocab), np.float32)
        while todo:
            part, want, dst, rest, used = [], [], [], [], 0
            for slot, tokens, places in todo:
                n = min(len(tokens), m.max_rows - used)
                if n:
                    part.append((slot, tokens[:n]))
                    want += [used + p for p, _ in places if p < n]
                    dst += [k for p, k in places if p < n]
                    used += n
                if n < len(tokens):
                    rest.append((slot, tokens[n:], [(p - n, k) for p, k in places if p >= n]))
            logits = m.step(part, want)
            if dst:
                out[dst] = logits
            todo = rest
        for i in end:
            if i in self.slots:
                m.release(self.slots.pop(i))
        return out


def run(model, lines, out_dir, emit):
    r = Replay(model)
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = r.step(s["entries"], s.get("end", ()))
        if len(logits):
            logits.astype("<f4").tofile(os.path.join(out_dir, f"{s['step']}.f32"))
        emit(f"done {s['step']}")
