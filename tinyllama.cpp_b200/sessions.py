"""Sequences over an engine's KV slots: each session owns one slot from its first token until it ends, and its tokens can
arrive in portions of any size. A portion of one token is a decode step, a longer one goes through prompt ingestion."""
import numpy as np


class Sessions:
    def __init__(self, engine):
        self.engine = engine
        self.free = list(range(engine.desc.max_seqs))[::-1]
        self.live = {}  # id -> [slot, tokens held]

    def open(self, sid):
        if sid in self.live:
            raise KeyError(f"session {sid!r} is live already")
        if not self.free:
            raise RuntimeError(f"all {self.engine.desc.max_seqs} slots are in use")
        self.live[sid] = [self.free.pop(), 0]

    def feed(self, sid, tokens, want=()):
        """The session's next tokens; returns the logits [len(want)][vocab] at places `want` among them."""
        if sid not in self.live:
            self.open(sid)
        slot, at = self.live[sid]
        want = list(want)
        if len(tokens) == 1:
            logits, _ = self.engine.decode(tokens, [at], slots=[slot], want_logits=bool(want), want_argmax=False)
            out = logits[[0] * len(want)] if want else np.empty((0, self.engine.vocab), np.float32)
        else:
            out = self.engine.prefill_rows(tokens, want, slot=slot, start_pos=at)
        self.live[sid][1] = at + len(tokens)
        return out

    def generate_greedy(self, sid, prompt, steps):
        """Feeds the prompt and decodes `steps` ids greedily on the device; returns them."""
        first = int(self.feed(sid, prompt, [len(prompt) - 1])[0].argmax())
        if steps <= 1:
            return [first][:steps]
        slot, at = self.live[sid]
        ids, _ = self.engine.generate_greedy([first], [at], steps - 1, slots=[slot])
        self.live[sid][1] = at + steps - 1
        return [first] + [int(t) for t in ids[:, 0]]

    def end(self, sid):
        """Gives the session's slot back; what it holds is cleared."""
        slot, _ = self.live.pop(sid)
        self.engine.kv_reset(slot)
        self.free.append(slot)
