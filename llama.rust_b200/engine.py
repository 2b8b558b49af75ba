"""Serving loop over a decode context: requests come in, every step carries one token of each sequence that is generating and
portions of the prompts that are still being read, up to the context's batch size; finished sequences give their cells and
state slots back.  Next tokens are picked on the device (argmax).  Works for every architecture of the library."""
import collections

import numpy as np


class Request:
    def __init__(self, rid, prompt, max_new, stop=()):
        self.id, self.prompt, self.max_new, self.stop = rid, list(prompt), max_new, frozenset(stop)
        self.out, self.fed, self.seq = [], 0, None

    @property
    def done(self):
        return len(self.out) >= self.max_new or (self.out and self.out[-1] in self.stop)


class Engine:
    """ctx: a Context.  max_seqs: sequences at a time; portion: most prompt tokens of one sequence in a step (None: all that fit)."""

    def __init__(self, ctx, max_seqs=16, portion=None):
        self.ctx, self.portion = ctx, portion
        self.free = collections.deque(range(min(max_seqs, ctx.n_seq)))
        self.waiting, self.running = collections.deque(), []
        self.steps = []   # rows of every step so far, by request id

    def submit(self, request):
        if not request.prompt:
            raise ValueError("a request needs a prompt")
        self.waiting.append(request)

    def plan(self):
        """[(request, first token, count)] of the next step: generating sequences first, then prompts in order of arrival"""
        while self.waiting and self.free:
            r = self.waiting.popleft()
            r.seq = self.free.popleft()
            self.running.append(r)
        room, rows = self.ctx.n_batch, []
        for r in self.running:
            if r.fed >= len(r.prompt) and room > 0:
                rows.append((r, r.fed, 1))
                room -= 1
        for r in self.running:
            left = len(r.prompt) - r.fed
            if left > 0 and room > 0:
                n = min(left, room, self.portion or left)
                rows.append((r, r.fed, n))
                room -= n
        return rows

    def step(self):
        """one decode call; returns the requests that finished with it"""
        rows = self.plan()
        if not rows:
            return []
        tokens, pos, seqs, outs, owners = [], [], [], [], []
        for r, at, n in rows:
            tokens += (r.prompt + r.out)[at:at + n]
            pos += range(at, at + n)
            seqs += [r.seq] * n
            if at + n >= len(r.prompt):
                outs.append(len(tokens) - 1)
                owners.append(r)
        wanted = outs or [len(tokens) - 1]
        _, picked = self.ctx.decode_seqs(tokens, pos, seqs, wanted, logits=False, argmax=True)
        self.steps.append([(r.id, n) for r, _, n in rows])
        for r, _, n in rows:
            r.fed += n
        for r, t in zip(owners, picked):
            r.out.append(int(t))
        finished = [r for r in self.running if r.done]
        for r in finished:
            self.ctx.seq_rm(r.seq)
            self.free.append(r.seq)
            self.running.remove(r)
        return finished

    def run(self):
        """until nothing is left; {request id: tokens}"""
        out = {}
        while self.waiting or self.running:
            for r in self.step():
                out[r.id] = r.out
        return out


def generate(ctx, prompts, max_new, stop=(), max_seqs=16, portion=None):
    """greedy continuations of token-id prompts, one list per prompt"""
    e = Engine(ctx, max_seqs, portion)
    for i, p in enumerate(prompts):
        e.submit(Request(i, p, max_new, stop))
    out = e.run()
    return [out[i] for i in range(len(prompts))]


class Replay:
    """Recorded streams instead of generated ones: tokens and schedule are the caller's, logits come back.  The same decode calls,
    cells and slots as the serving loop."""

    def __init__(self, ctx):
        self.ctx = ctx
        self.free = collections.deque(range(ctx.n_seq))
        self.seq, self.pos = {}, {}

    def step(self, entries):
        """entries: [(id, tokens, wanted places)] -> logits float32 [wanted, n_vocab] in that order"""
        tokens, pos, seqs, wanted = [], [], [], []
        for rid, toks, want in entries:
            if rid not in self.seq:
                self.seq[rid], self.pos[rid] = self.free.popleft(), 0
            wanted += [len(tokens) + w for w in want]
            tokens += toks
            pos += range(self.pos[rid], self.pos[rid] + len(toks))
            seqs += [self.seq[rid]] * len(toks)
            self.pos[rid] += len(toks)
        out = np.empty((len(wanted), self.ctx.n_vocab), dtype=np.float32)
        order = sorted(range(len(wanted)), key=lambda k: wanted[k])
        for lo in range(0, len(tokens), self.ctx.n_batch):
            hi = min(lo + self.ctx.n_batch, len(tokens))
            mine = [k for k in order if lo <= wanted[k] < hi]
            rows = [wanted[k] - lo for k in mine] or [hi - lo - 1]
            got, _ = self.ctx.decode_seqs(tokens[lo:hi], pos[lo:hi], seqs[lo:hi], rows, logits=bool(mine))
            if mine:
                out[mine] = got
        return out

    def end(self, rid):
        if rid in self.seq:
            self.ctx.seq_rm(self.seq[rid])
            self.free.append(self.seq.pop(rid))
            del self.pos[rid]
