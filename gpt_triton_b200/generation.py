"""Token-by-token generation, for every model of this package.

A model that is driven from here offers

    check_capacity(capacity)                     raises if it cannot hold that many positions
    new_cache(batch, capacity)                   whatever it remembers between tokens
    prompt_pass(ids, cache, start, pos, want)    (batch, n) tokens at positions start.. -> final rows at the places `want`
    decode_pass(ids, cache, pos)                 one token per sequence at the device-side position pos[0] -> final rows
    pick(rows, temperature, top_k, seed, pos)    final rows -> next ids
    head_logits(rows)                            final rows -> logits

`rows` is opaque here.  No counterpart in the reference, which lists "KV cache + sampling" as not built (README.md:55).
"""

import gc

import torch

from . import kernels as K
from .module_base import _OperandCache


class GenerationSession:
    """The state of a fixed number of sequences that advance together: the model's cache, the device-side position
    counter and, after the first two decode steps, a CUDA graph of one decode step that is replayed for every further
    token of this and later generations (any prompt length: the position lives in device memory).  Prompt + generated
    tokens - 1 must fit `capacity`."""

    EAGER_STEPS = 2  # decode steps run eagerly before the capture (kernel attributes, allocator pools)

    def __init__(self, model, batch, capacity, max_new_tokens=1, temperature=0.0, top_k=0, seed=0, use_cuda_graph=True):
        model.check_capacity(capacity)
        assert temperature >= 0.0 and top_k >= 0 and max_new_tokens >= 1
        dev = next(model.parameters()).device
        self.model, self.batch, self.capacity = model, batch, max(int(capacity), 1)
        self.temperature, self.top_k, self.seed, self.use_cuda_graph = float(temperature), int(top_k), int(seed), use_cuda_graph
        self.cache = model.new_cache(batch, self.capacity)
        self.length = 0  # tokens of every sequence that the cache holds (kept on the host between calls)
        self.pos = torch.zeros(2, device=dev, dtype=torch.int32)  # {tokens in the cache, prompt length}
        self.tokens = torch.zeros((batch, max_new_tokens), device=dev, dtype=torch.int64)
        self.feedback = torch.zeros((batch,), device=dev, dtype=torch.int64)  # the ids the next decode step embeds
        self.graph = None
        self._sig = self._signature()

    @property
    def kv(self):
        return self.cache

    def _signature(self):
        return tuple(_OperandCache._tag(p) for p in self.model.parameters())

    def stale(self):
        """True once a parameter has been reloaded, cast or moved: a captured step holds the old operands."""
        return self._signature() != self._sig

    def reset(self):
        """Forget the sequences; the cache's memory is used again by the next ones."""
        self.length = 0

    def _check_device(self):
        code = K.device_status(self.pos.device)
        if code:
            raise RuntimeError(f"generation stopped by a device-side check (code {code}): cache or token buffer out of room")

    @torch.no_grad()
    def extend(self, ids, want=None):
        """The next tokens of every sequence, ids (batch, n): any portion of a prompt, or one given token.  Returns the
        model's final rows at the places `want` of this portion (None: the last), in sequence order: what `pick` or
        `head_logits` take.  One token behind earlier ones runs the decode step, anything else the prompt pass."""
        B, n = ids.shape
        assert B == self.batch and n >= 1 and self.length + n <= self.capacity, "the tokens do not fit this session's cache"
        assert not self.stale(), "the model's parameters changed: make a new session"
        if n == 1 and self.length > 0:
            self.pos[:1].fill_(self.length)
            self.feedback.copy_(ids[:, 0])
            rows = self.model.decode_pass(self.feedback, self.cache, self.pos)
        else:
            rows = self.model.prompt_pass(ids, self.cache, self.length, self.pos, want)
        self.length += n
        return rows

    def _step(self):
        m = self.model
        rows = m.decode_pass(self.feedback, self.cache, self.pos)
        ids = m.pick(rows, self.temperature, self.top_k, self.seed, self.pos)
        K.decode_append(ids, self.tokens, self.pos, advance=True, feedback=self.feedback)

    @torch.no_grad()
    def generate(self, ids, max_new_tokens, portion=0):
        """Continuations (batch, max_new_tokens) of the prompts ids (batch, n); ``portion`` > 0 runs the prompt in pieces
        of at most that many tokens (bounds the activation memory of a long prompt)."""
        m = self.model
        B, L0 = ids.shape
        assert B == self.batch and L0 >= 1 and 1 <= max_new_tokens <= self.tokens.shape[1]
        assert L0 + max_new_tokens - 1 <= self.capacity, "prompt + generated tokens do not fit this session's cache"
        self.reset()
        step = portion if portion > 0 else L0
        for t in range(0, L0, step):
            last = self.extend(ids[:, t:t + step].contiguous())
        self.pos.copy_(torch.tensor([L0, L0], dtype=torch.int32), non_blocking=False)
        first = m.pick(last, self.temperature, self.top_k, self.seed, self.pos)
        K.decode_append(first, self.tokens, self.pos, advance=False, feedback=self.feedback)
        steps = max_new_tokens - 1
        done = 0
        if self.graph is None:
            while done < min(steps, self.EAGER_STEPS):
                self._step()
                done += 1
            if self.use_cuda_graph and done < steps:
                torch.cuda.synchronize(self.pos.device)
                gc.collect()  # a dead session's graph that is freed while a capture runs would invalidate the capture
                self.graph = torch.cuda.CUDAGraph()
                with torch.cuda.graph(self.graph):
                    self._step()
        for _ in range(steps - done):
            if self.graph is not None:
                self.graph.replay()
            else:
                self._step()
        self.length = L0 + steps
        self._check_device()
        return self.tokens[:, :max_new_tokens].clone()


class GeneratesTokens:
    """Mixin: ``generate`` on top of GenerationSession, sessions kept on the model."""

    @torch.no_grad()
    def generate(self, ids, max_new_tokens, temperature=0.0, top_k=0, seed=0, use_cuda_graph=True, portion=0):
        """ids (batch, prompt_len) -> (batch, max_new_tokens) int64 continuation, one token per step with the model's
        cache.  temperature 0: greedy; > 0: draws from softmax(logits / temperature) over the top_k largest logits (0 =
        all), reproducible for a given seed.  The sessions (cache, captured decode step) are kept on the model per
        (batch, temperature, top_k, seed) and re-used by later calls that fit them."""
        B, L0 = ids.shape
        need = L0 + max_new_tokens - 1
        prm = next(self.parameters())
        key = (B, temperature, top_k, seed, use_cuda_graph, prm.dtype, prm.device)
        sessions = self.__dict__.setdefault("_sessions", {})
        session = sessions.get(key)
        if session is None or session.capacity < need or session.tokens.shape[1] < max_new_tokens or session.stale():
            sessions.pop(key, None)
            while len(sessions) >= 4:  # every session holds a cache: keep a few
                sessions.pop(next(iter(sessions)))
            sessions[key] = session = GenerationSession(self, B, capacity=need, max_new_tokens=max_new_tokens, temperature=temperature,
                                                        top_k=top_k, seed=seed, use_cuda_graph=use_cuda_graph)
        return session.generate(ids, max_new_tokens, portion=portion)
