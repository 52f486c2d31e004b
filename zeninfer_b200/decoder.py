"""What every decoder shares: the sequence's state, the step graphs, the prompt in blocks, generation and sampling.

A model class supplies the launches (`_enqueue_layers`, `_enqueue_head`, `prefill`, `_block_logits`); everything that orders
them over a sequence is here, and nothing here computes on the host.  A decoder serves one sequence at a time: `reset` gives
back what the last one held, `feed` continues the live one by any number of tokens, `generate` runs a whole request.
"""
from __future__ import annotations

import numpy as np

from .backend import Backend


class SequenceState:
    """The device buffers that carry a sequence from step to step, fp32.  A buffer indexed by position (a KV cache) is simply
    overwritten by the next sequence, because nothing reads past the positions written so far; a recurrent one is added with
    start_zero and cleared when a sequence begins."""

    def __init__(self, torch, dev) -> None:
        self.torch, self.dev = torch, dev
        self.buffers: dict[str, "torch.Tensor"] = {}
        self._zero: list["torch.Tensor"] = []

    def add(self, name: str, shape: tuple[int, ...], start_zero: bool = False):
        if name in self.buffers:
            raise ValueError(f"state buffer {name!r} exists")
        t = self.buffers[name] = self.torch.zeros(shape, dtype=self.torch.float32, device=self.dev)
        if start_zero:
            self._zero.append(t)
        return t

    def clear(self) -> None:
        """On the current stream."""
        for t in self._zero:
            t.zero_()

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.buffers.values())


class Decoder:
    PREFILL_CHUNK = 512     # tokens per block (buffers are sized for it)
    PREFILL_MIN = 16        # shorter blocks go token by token
    rank, world, group = 0, 1, None

    def _init_runtime(self, backend: Backend, vocab: int, max_positions: int, device=None) -> None:
        import torch
        self.torch, self.be = torch, backend
        self.dev = device if device is not None else torch.device("cuda", torch.cuda.current_device())
        self.vocab, self.max_positions = vocab, max_positions
        self.stream = torch.cuda.Stream(device=self.dev)
        self.sequence = SequenceState(torch, self.dev)
        self.logits = torch.zeros(vocab, dtype=torch.float32, device=self.dev)
        self.pos = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self.token = torch.zeros(1, dtype=torch.int64, device=self.dev)
        self.host_token = torch.zeros(1, dtype=torch.int64).pin_memory()   # generate() feeds every step from the host, as the reference does
        self.graph_layers = self.graph_head = None
        self.fed = 0            # tokens feed() has taken since the last reset

    # ---- what a model supplies ----
    def _enqueue_layers(self) -> None:
        """The token in self.token at position self.pos through the layers; pos advances."""
        raise NotImplementedError

    def _enqueue_head(self) -> None:
        """The last token's logits into self.logits and the greedy pick into self.token."""
        raise NotImplementedError

    def prefill(self, d_tokens, count: int) -> None:
        """`count` tokens (device int64) through the layers as one block, ready for _enqueue_head and _block_logits."""
        raise NotImplementedError

    def _block_logits(self, rows: list[int]):
        """Logits [len(rows)][vocab] (device fp32) of rows of the last prefill block."""
        raise NotImplementedError

    def _prompt_token(self, last: bool) -> None:
        """A prompt token that goes alone."""
        self.step(want_token=last)

    def can_prefill_blocks(self) -> bool:
        return self.world == 1

    def sync_ranks(self) -> None:
        """Where several processes share the model: they begin a sequence of steps together."""

    # ---- steps ----
    def capture(self) -> None:
        """Runs one throw-away step (kernel attributes are set on first launch), then captures the two graphs."""
        torch = self.torch
        self.sync_ranks()
        with torch.cuda.stream(self.stream):
            self.reset()
            self._enqueue_layers()
            self._enqueue_head()
            self.stream.synchronize()
            self.graph_layers, self.graph_head = torch.cuda.CUDAGraph(), torch.cuda.CUDAGraph()
            # with collectives in the graph, other threads of the process (the collective library's watchdog) may call
            # the runtime during the capture: only this thread's calls belong to it
            mode = dict(capture_error_mode="thread_local") if self.world > 1 else {}
            with torch.cuda.graph(self.graph_layers, stream=self.stream, **mode):
                self._enqueue_layers()
            with torch.cuda.graph(self.graph_head, stream=self.stream, **mode):
                self._enqueue_head()
            self.stream.synchronize()
        self.reset()

    def reset(self) -> None:
        """Begins a new sequence."""
        with self.torch.cuda.stream(self.stream):
            self.pos.zero_()
            self.token.zero_()
            self.sequence.clear()
        self.stream.synchronize()
        self.fed = 0

    def step(self, want_token: bool) -> None:
        """Consumes the token in self.token at position self.pos; with want_token the pick replaces self.token."""
        with self.torch.cuda.stream(self.stream):
            if self.graph_layers is not None:
                self.graph_layers.replay()
                if want_token:
                    self.graph_head.replay()
            else:
                self._enqueue_layers()
                if want_token:
                    self._enqueue_head()

    def feed(self, tokens: list[int], want: list[int] = ()) -> np.ndarray:
        """Continues the live sequence by `tokens` (any number of them) and returns the logits [len(want)][vocab] after the
        tokens at the places `want` of this call.  Blocks of at least PREFILL_MIN tokens go through prefill(), others token
        by token; nothing but the state earlier calls left is carried over."""
        torch = self.torch
        if any(not 0 <= w < len(tokens) for w in want):
            raise ValueError("feed: a wanted place is not among the tokens")
        if self.fed + len(tokens) > self.max_positions:
            raise ValueError("feed: the sequence does not fit the configured positions")
        if any(not 0 <= t < self.vocab for t in tokens):
            raise ValueError("feed: a token id is outside the vocabulary")
        rows: dict[int, np.ndarray] = {}
        with torch.cuda.stream(self.stream):
            d_ids = torch.tensor(tokens, dtype=torch.int64).pin_memory().to(self.dev, non_blocking=True)
            done = 0
            while done < len(tokens):
                n = min(self.PREFILL_CHUNK, len(tokens) - done)
                if n >= self.PREFILL_MIN and self.can_prefill_blocks():
                    self.prefill(d_ids[done:done + n], n)
                    mine = sorted({w for w in want if done <= w < done + n})
                    if mine:
                        for w, row in zip(mine, self._block_logits([w - done for w in mine]).cpu().numpy()):
                            rows[w] = row
                else:
                    n = 1
                    self.token.copy_(d_ids[done:done + 1])
                    self._prompt_token(last=done in want)
                    if done in want:
                        rows[done] = self.logits.cpu().numpy()
                done += n
                self.fed += n
        self.be.dev_check(self.stream.cuda_stream)
        return np.stack([rows[w] for w in want]) if len(want) else np.zeros((0, self.vocab), np.float32)

    # ---- generation ----
    def feed_prompt(self, prompt: list[int], batched_prefill: bool | None = None) -> None:
        """Enqueues the whole prompt from position self.pos on, ending with the first pick (left in self.token).  Blocks of
        at least PREFILL_MIN tokens go through prefill() when batched_prefill (default: wherever can_prefill_blocks()), the
        rest token by token."""
        torch = self.torch
        ids = torch.tensor(prompt, dtype=torch.int64).pin_memory()
        if batched_prefill is None:
            batched_prefill = self.can_prefill_blocks()
        with torch.cuda.stream(self.stream):
            done = 0
            if batched_prefill and len(prompt) >= self.PREFILL_MIN:
                d_ids = ids.to(self.dev, non_blocking=True)
                while len(prompt) - done >= self.PREFILL_MIN:
                    n = min(self.PREFILL_CHUNK, len(prompt) - done)
                    self.prefill(d_ids[done:done + n], n)
                    done += n
                if done == len(prompt):
                    self._enqueue_head()      # the first pick, from the last prompt token's hidden state
            for i in range(done, len(prompt)):
                self.token.copy_(ids[i:i + 1], non_blocking=True)
                last = i + 1 == len(prompt)
                self._prompt_token(last)

    def _sample(self, temperature: float, top_k: int, top_p: float, u: float) -> None:
        """Replaces the greedy pick in self.token by a draw from the filtered distribution of self.logits."""
        self.be.dev_sample(self.logits.data_ptr(), self.vocab, temperature, top_k, top_p, u, self.token.data_ptr(), self.stream.cuda_stream)

    def generate(self, prompt: list[int], max_new: int, on_token=None, batched_prefill: bool | None = None, temperature: float = 0.0,
                 top_k: int = 0, top_p: float = 1.0, seed: int = 0) -> list[int]:
        """Generation: the prompt, then max_new picks (each read back, as the reference's per-token callback does).  With
        temperature <= 0 the picks are greedy; otherwise every token is drawn on the device from the temperature / top-k /
        top-p distribution of the step's logits (GenerationOptions, sample_logits :391-418), with one uniform number per
        token from a host generator seeded with `seed` (the generator stays on the host, as the reference's does).  The
        prompt goes through prefill() in blocks (in the prompt's activation mode) on one GPU and on a column-cut sharded
        decoder with an NCCL group, token by token otherwise; batched_prefill overrides the choice.
        Raises when the context would overflow."""
        torch = self.torch
        if not prompt or len(prompt) + max_new > self.max_positions:
            raise ValueError("prompt + max_new exceeds the configured positions")
        self.reset()
        self.sync_ranks()
        out: list[int] = []
        rng = np.random.default_rng(seed) if temperature > 0.0 else None
        with torch.cuda.stream(self.stream):
            self.feed_prompt(prompt, batched_prefill)
            for n in range(max_new):
                if rng is not None:               # the step left the greedy pick in self.token: draw instead
                    self._sample(temperature, top_k, top_p, float(rng.random()))
                tok = int(self.token.item())      # device -> host read of the step's result
                out.append(tok)
                if on_token:
                    on_token(tok)
                if n + 1 < max_new:
                    self.host_token[0] = tok      # host -> device: the next step's input comes from the caller's side
                    self.token.copy_(self.host_token, non_blocking=True)
                    self.step(want_token=True)
        self.be.dev_check(self.stream.cuda_stream)
        return out

    def last_logits(self) -> np.ndarray:
        self.stream.synchronize()
        return self.logits.cpu().numpy()

    def close(self) -> None:
        self.stream.synchronize()
        self.graph_layers = self.graph_head = None
