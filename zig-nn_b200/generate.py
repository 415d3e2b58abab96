"""Token generation over the engines: one prompt, or a queue of requests over an engine's slots."""
from collections import deque

from . import api


def generate(engine, prompt, n_tokens, top_k=None, temperature=1.0, rng=None):
    """n_tokens tokens after `prompt`. Greedy (the arg-max feeds the next step on the device) unless `rng` is given:
    then api.sample_top_k on every step's logits."""
    logits = engine.prefill(prompt)
    if n_tokens == 0:
        return []
    if rng is None:
        first = int(api.argmax(logits).item())
        rest = engine.decode_greedy(first, n_tokens - 1) if n_tokens > 1 else []
        return [first] + [int(t) for t in rest]
    out = [api.sample_top_k(logits, top_k or 0, temperature, rng)]
    while len(out) < n_tokens:
        out.append(api.sample_top_k(engine.decode_next(out[-1]), top_k or 0, temperature, rng))
    return out


class Request:
    def __init__(self, prompt, n_tokens):
        self.prompt, self.n_tokens, self.seq, self.tokens = list(prompt), int(n_tokens), None, []

    @property
    def finished(self):
        return len(self.tokens) >= self.n_tokens


def serve(engine, requests, portion=0):
    """Greedy continuous batching for an engine with slots: waiting requests take free slots in order (their prompts
    run in portions of `portion` tokens, 0 = whole), one batched step advances all running ones, a finished one gives
    its slot back. requests: Request objects; returns them with `tokens` filled."""
    waiting, running = deque(r for r in requests if not r.finished), []
    while waiting or running:
        while waiting:
            seq = engine.acquire()
            if seq is None:
                break
            r = waiting.popleft()
            r.seq = seq
            step = portion or len(r.prompt)
            for t0 in range(0, len(r.prompt), step):
                part = r.prompt[t0:t0 + step]
                last = t0 + step >= len(r.prompt)
                logits = engine.extend(part, [len(part) - 1] if last else [], seq=seq)
            r.tokens.append(int(api.argmax(logits[0]).item()))
            running.append(r)
        for r in [r for r in running if r.finished]:
            engine.release(r.seq)
            running.remove(r)
        if running:
            logits = engine.decode_next_batch([r.seq for r in running], [r.tokens[-1] for r in running])
            for r, t in zip(running, logits.argmax(dim=1).tolist()):
                r.tokens.append(int(t))
    return requests
