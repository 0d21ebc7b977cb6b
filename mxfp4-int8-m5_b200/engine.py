"""Serving loop around a registered model (registry.Bundle): requests own a cache from a pool, a step feeds each of its requests
the next tokens of its sequence - a portion of a prompt through the prefill path, a single token through the decode path - and
a finished request returns its cache.  generate() is greedy decoding of one request."""
import torch


class CachePool:
    """Caches of equal capacity, created on demand and used again after a request has ended."""

    def __init__(self, make, capacity):
        self.make, self.capacity, self.free = make, capacity, []

    def acquire(self):
        if not self.free:
            return self.make(self.capacity)
        cache = self.free.pop()
        for c in cache:
            c.reset()
        return cache

    def release(self, cache):
        self.free.append(cache)


class Engine:
    def __init__(self, bundle, max_tokens, device="cuda"):
        self.bundle, self.device = bundle, device
        self.pool = CachePool(bundle.prefill.make_cache, max(1, max_tokens))
        self.live = {}

    def start(self, rid):
        if rid not in self.live:
            self.live[rid] = self.pool.acquire()
        return self.live[rid]

    def finish(self, rid):
        cache = self.live.pop(rid, None)
        if cache is not None:
            self.pool.release(cache)

    @torch.no_grad()
    def feed(self, rid, tokens, want):
        """The request's next tokens (list of ids) -> float32 logits [len(want), V] at the places `want` among them, or None."""
        cache = self.start(rid)
        ids = torch.tensor(tokens, dtype=torch.long, device=self.device)[None]
        if len(tokens) == 1:
            logits = self.bundle.decode.step(ids, cache)
            return logits[0, [0] * len(want)].float() if want else None
        h = self.bundle.prefill.hidden(ids, cache)
        if not want:
            return None
        rows = torch.tensor(want, dtype=torch.long, device=self.device)
        return self.bundle.prefill.logits(h[:, rows])[0].float()

    def step(self, entries, end=()):
        """entries: [(request id, tokens, wanted places)] -> their logits in order (None where nothing is wanted); the requests in
        `end` give back what they hold afterwards."""
        out = [self.feed(rid, tokens, want) for rid, tokens, want in entries]
        for rid in end:
            self.finish(rid)
        return out

    def generate(self, prompt, n, rid="generate"):
        """n tokens after `prompt` (list of ids), greedy: the prompt through step(), then the decoder's captured graph."""
        assert n >= 1 and len(prompt) + n - 1 <= self.pool.capacity, "prompt and continuation exceed the cache"
        logits = self.step([(rid, prompt, [len(prompt) - 1])])[0]
        first = logits[-1].argmax().reshape(1, 1)
        out = [int(first)]
        if n > 1:
            out += self.bundle.decode.generate(first, self.live[rid], n - 1).tolist()
        self.finish(rid)
        return out
