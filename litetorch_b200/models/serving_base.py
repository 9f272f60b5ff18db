"""The part of cached serving that does not depend on the model: prompt chunks and batched decode steps over a paged cache
(and, for models with recurrent layers, per-sequence state slots), CUDA-graph replay of the decode step, sampling, and
`generate`.

A model supplies four pieces of device work and inherits the rest:

    _prompt_hidden(tokens, start, block_ids, slot)  hidden rows of a prompt chunk; writes the cache and the state
    _decode_hidden(d, S, width)                     hidden rows of one token of S sequences, from the packed input block
    _logits(hidden, rows)                           logits of the given rows (None: all)
    new_serving(...)                                on the engine: how to make the serving model (see `models.registry`)

The packed int64 input block of a decode step is [5 + width, S]: token, position, cache slot, context length, state slot
of every sequence, then its block table (transposed).
"""
from __future__ import annotations

from typing import List, Optional, Sequence

import torch


class ServingModel:
    state_slots = 0                          # > 0: the scheduler passes every sequence's state slot along

    def __init__(self, engine, block_size: int, graphs: bool):
        self.e = engine
        self.block_size = block_size
        self.graphs = graphs                 # record the decode step per (batch size, table width) and replay it
        self._graphs = {}
        self.sampler = None                  # None: greedy on the device; else a callable logits [rows, vocab] -> tokens
        self.last_logits = None              # [rows, vocab] of the newest step (kept for inspection and tests)
        self.prefill_tokens_computed = 0
        self.prefill_tokens_reused = 0

    # ------------------------------------------------------------------ the model's part
    def _prompt_hidden(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], slot: int):
        raise NotImplementedError

    def _decode_hidden(self, d: torch.Tensor, S: int, width: int):
        raise NotImplementedError

    def _logits(self, hidden, rows: Optional[List[int]] = None) -> torch.Tensor:
        raise NotImplementedError

    def _warm_input(self, host: torch.Tensor) -> torch.Tensor:
        """The input block of the pass that runs a step before it is recorded; a model whose step changes more than the
        cache cells that the replay writes again points it at scratch."""
        return host

    # ------------------------------------------------------------------ tokens from logits
    def _pick(self, logits: torch.Tensor) -> torch.Tensor:
        self.last_logits = logits
        if self.sampler is not None:
            return self.sampler(logits.float())
        return logits.float().argmax(-1)

    # ------------------------------------------------------------------ prompt chunks
    @torch.no_grad()
    def prefill_chunk(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], want_token: bool, slot: int = 0) -> int:
        """Run prompt positions [start, start + len(tokens)) of one sequence.  Returns the next token when `want_token` (the
        chunk completes the prompt), else -1."""
        self.prefill_tokens_computed += len(tokens)
        x = self._prompt_hidden(tokens, start, block_ids, slot)
        if not want_token:
            return -1
        return int(self._pick(self._logits(x, [len(tokens) - 1])).item())

    @torch.no_grad()
    def score_chunk(self, tokens: Sequence[int], start: int, block_ids: Sequence[int], rows: Sequence[int], slot: int = 0) -> torch.Tensor:
        """The same pass; returns the fp32 logits [len(rows), vocab] at the given places among `tokens`."""
        self.prefill_tokens_computed += len(tokens)
        x = self._prompt_hidden(tokens, start, block_ids, slot)
        return self._logits(x, list(rows)).float()

    # ------------------------------------------------------------------ one token for every running sequence
    def _decode_body(self, d: torch.Tensor, S: int, width: int):
        logits = self._logits(self._decode_hidden(d, S, width))
        return logits, self._pick(logits)

    def _run_decode(self, last_tokens, positions, block_tables, slots):
        """(logits [S, vocab], next tokens [S]).  On a GPU the step's launches are recorded once per (batch size,
        block-table width) into a CUDA graph and replayed: the step then costs its kernels, not their launch overhead.  The
        inputs of a replay are copied into the graph's static input block first."""
        dev = self.e.device
        S = len(last_tokens)
        bs = self.block_size
        width = max((p + bs) // bs for p in positions)
        use_graph = self.graphs and dev.type == "cuda"
        if use_graph:
            width = (width + 15) // 16 * 16                     # fewer distinct graphs: table widths in steps of 16 blocks
        host = torch.zeros(5 + width, S, dtype=torch.int64)
        host[0] = torch.tensor(list(last_tokens), dtype=torch.int64)
        host[1] = torch.tensor(list(positions), dtype=torch.int64)
        for s in range(S):
            p = positions[s]
            host[2, s] = block_tables[s][p // bs] * bs + p % bs
            row = block_tables[s][:width]
            host[5:5 + len(row), s] = torch.tensor(list(row), dtype=torch.int64)
        host[3] = host[1] + 1
        if slots is not None:
            host[4] = torch.tensor(list(slots), dtype=torch.int64)
        if not use_graph:
            return self._decode_body(host.to(dev, non_blocking=True), S, width)
        entry = self._graphs.get((S, width))
        if entry is None:
            static_in = self._warm_input(host).to(dev)
            side = torch.cuda.Stream(device=dev)
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):                        # eager run on the capture stream: workspaces, caches
                self._decode_body(static_in, S, width)
            torch.cuda.current_stream().wait_stream(side)
            torch.cuda.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=side):
                static_out = self._decode_body(static_in, S, width)
            entry = self._graphs[S, width] = (g, static_in, static_out)
            # the eager pass wrote this step's cache cells already; the replay below rewrites the same ones
        g, static_in, static_out = entry
        static_in.copy_(host, non_blocking=True)
        g.replay()
        self.last_logits = static_out[0]
        return static_out

    @torch.no_grad()
    def decode_batch(self, last_tokens: Sequence[int], positions: Sequence[int], block_tables: List[Sequence[int]],
                     slots: Optional[Sequence[int]] = None) -> List[int]:
        """last_tokens[s] sits at position positions[s] of sequence s and is not in the cache yet: run it and return the next
        token of every sequence."""
        return self._run_decode(last_tokens, positions, block_tables, slots)[1].tolist()

    @torch.no_grad()
    def decode_logits(self, last_tokens: Sequence[int], positions: Sequence[int], block_tables: List[Sequence[int]],
                      slots: Optional[Sequence[int]] = None) -> torch.Tensor:
        """The same step; returns its fp32 logits [S, vocab]."""
        return self._run_decode(last_tokens, positions, block_tables, slots)[0].float().clone()

    # ------------------------------------------------------------------ helpers
    def _slots(self, block_ids: Sequence[int], start: int, n: int) -> torch.Tensor:
        bs = self.block_size
        p = torch.arange(start, start + n)
        return (torch.tensor(list(block_ids), dtype=torch.int64)[p // bs] * bs + p % bs).to(torch.int32)

    @staticmethod
    def _splits_for(ctas: int, keys: int) -> int:
        """Splits of the key range per (sequence, KV head): about four CTAs per SM, at least 256 keys per split."""
        return max(1, min(32, keys // 256, (148 * 4 + ctas - 1) // max(ctas, 1)))


class Sampler:
    """Temperature / top-k / nucleus sampling of next tokens from logits [rows, vocab] with its own random generator, so
    that a run is reproducible from its seed.  `temperature == 0` (or `top_k == 1`) is greedy."""

    def __init__(self, temperature: float = 1.0, top_k: int = 0, top_p: float = 1.0, seed: int = 0, device="cpu"):
        self.temperature, self.top_k, self.top_p = float(temperature), int(top_k), float(top_p)
        self.gen = torch.Generator(device=device).manual_seed(int(seed))

    def __call__(self, logits: torch.Tensor) -> torch.Tensor:
        if self.temperature <= 0.0 or self.top_k == 1:
            return logits.argmax(-1)
        z = logits / self.temperature
        if self.top_k > 0 and self.top_k < z.shape[-1]:
            kth = z.topk(self.top_k, -1).values[..., -1:]
            z = z.masked_fill(z < kth, float("-inf"))
        if self.top_p < 1.0:
            order = z.sort(-1, descending=True)
            p = torch.softmax(order.values, -1)
            before = p.cumsum(-1) - p                     # probability mass ahead of each token, in sorted order
            drop = before >= self.top_p                   # the first token always stays
            z = z.masked_fill(torch.zeros_like(drop).scatter(-1, order.indices, drop), float("-inf"))
        return torch.multinomial(torch.softmax(z, -1), 1, generator=self.gen).squeeze(-1)


@torch.no_grad()
def generate(engine, prompts: Sequence[Sequence[int]], max_new_tokens: int, *, temperature: float = 0.0,
             top_k: int = 0, top_p: float = 1.0, seed: int = 0, eos_id: int = -1, block_size: int = 16,
             max_num_seqs: int = 64, max_num_batched_tokens: int = 4096, kv_dtype=None,
             prefix_cache_bytes: int = 0) -> List[List[int]]:
    """Continue every prompt by up to `max_new_tokens` tokens (stopping at `eos_id`) with continuous batching on a paged KV
    cache sized for the request, and return the new tokens per prompt.  Greedy by default (the decode step is replayed
    from CUDA graphs on a GPU); with `temperature > 0` the next tokens are drawn by `Sampler` (eager decode steps).
    `engine`: any engine of `models.registry`."""
    from ..serving import Request, ServingScheduler
    from .registry import new_serving
    need = sum((len(p) + max_new_tokens + block_size - 1) // block_size for p in prompts)
    greedy = temperature <= 0.0 or top_k == 1
    model = new_serving(engine, num_blocks=need + 1, block_size=block_size, max_num_seqs=max_num_seqs, kv_dtype=kv_dtype,
                        graphs=greedy, prefix_cache_bytes=prefix_cache_bytes)  # prompts of one call that share a prefix reuse its blocks
    if not greedy:
        model.sampler = Sampler(temperature, top_k, top_p, seed, device=engine.device)
    sched = ServingScheduler(num_blocks=need + 1, block_size=block_size, max_num_seqs=max_num_seqs,
                             max_num_batched_tokens=max_num_batched_tokens, eos_id=eos_id)
    limit = engine.cfg.max_seq                            # None: the model's positions have no end
    reqs = [Request(i, list(p), max_new_tokens=max_new_tokens) for i, p in enumerate(prompts)]
    for r in reqs:
        if limit and len(r.prompt_tokens) + max_new_tokens > limit:
            raise ValueError("prompt %d: %d tokens + %d new exceed the model's %d positions" %
                             (r.id, len(r.prompt_tokens), max_new_tokens, limit))
        sched.add_request(r)
    finished, guard = 0, 0
    while finished < len(reqs):
        finished += len(sched.step(model))
        guard += 1
        if guard > 4 * (max_new_tokens + len(reqs)) + 64 + sum(len(p) for p in prompts):
            raise RuntimeError("the schedule did not finish")
    return [list(r.generated_tokens) for r in reqs]
