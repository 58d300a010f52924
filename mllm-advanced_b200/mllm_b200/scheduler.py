"""Continuous batching over a LanguageModel: requests wait for a slot, prompts are taken in portions that share steps
with the sequences already decoding, and when no prompt is left to read the running sequences decode together on the
device (one graph replay per token) until one of them is due to end.  Sampling is greedy, on the device."""
from collections import deque


class Request:
    def __init__(self, prompt, max_new, stop=()):
        self.prompt, self.max_new, self.stop = [int(t) for t in prompt], int(max_new), frozenset(stop)
        self.slot, self.done, self.output = None, 0, []  # done: prompt tokens read so far

    @property
    def finished(self):
        return len(self.output) >= self.max_new or bool(self.output and self.output[-1] in self.stop)


class Scheduler:
    def __init__(self, model, portion=None, stop_check=16):
        """portion: most prompt tokens of one request in a step (default: the model's max_rows); stop_check: decode
        steps between looks at the stop tokens."""
        self.model, self.portion, self.stop_check = model, portion or model.max_rows, stop_check
        self.waiting, self.running = deque(), []

    def submit(self, prompt, max_new, stop=()):
        r = Request(prompt, max_new, stop)
        if not r.prompt or r.max_new < 1:
            raise ValueError("a request needs a prompt and at least one new token")
        if len(r.prompt) + r.max_new > self.model.max_ctx:
            raise ValueError(f"{len(r.prompt)} + {r.max_new} tokens do not fit a slot of {self.model.max_ctx}")
        self.waiting.append(r)
        return r

    def _admit(self):
        while self.waiting:
            slot = self.model.acquire()
            if slot is None:
                return
            r = self.waiting.popleft()
            r.slot = slot
            self.running.append(r)

    def _retire(self):
        for r in [r for r in self.running if r.finished]:
            self.running.remove(r)
            self.model.release(r.slot)

    def _mixed_step(self):
        m = self.model
        room, entries, ends = m.max_rows, [], []
        for r in self.running:  # sequences that decode come first, a token each
            if r.done == len(r.prompt) and room:
                entries.append((r.slot, [r.output[-1]]))
                ends.append(r)
                room -= 1
        for r in self.running:
            n = min(len(r.prompt) - r.done, self.portion, room)
            if n > 0:
                entries.append((r.slot, r.prompt[r.done:r.done + n]))
                r.done += n
                room -= n
                if r.done == len(r.prompt):
                    ends.append(r)
        m.step(entries, sample=True)
        for r in ends:
            r.output.append(int(m.read(r.slot, m.length[r.slot] - 1, 1)[0]))

    def _decode(self):
        m = self.model
        steps = min(r.max_new - len(r.output) for r in self.running)
        if any(r.stop for r in self.running):
            steps = min(steps, self.stop_check)
        batch = self.running[:m.max_rows]
        first = {r.slot: m.length[r.slot] for r in batch}
        m.decode([r.slot for r in batch], steps)
        for r in batch:
            for t in m.read(r.slot, first[r.slot], steps):
                if not r.finished:
                    r.output.append(int(t))

    def run(self):
        """Until every submitted request is finished."""
        while self.waiting or self.running:
            self._admit()
            if any(r.done < len(r.prompt) for r in self.running):
                self._mixed_step()
            else:
                self._decode()
            self._retire()


def generate(model, prompts, max_new, stop=(), portion=None):
    """Greedy continuations of all prompts, batched."""
    s = Scheduler(model, portion)
    reqs = [s.submit(p, max_new, stop) for p in prompts]
    s.run()
    return [r.output for r in reqs]
