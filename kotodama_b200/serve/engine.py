"""Serving engine: paged KV cache (16-token pages), continuous batching, greedy / sampled
decoding on the device.

The reference server (``serve.py:322-391``) handles one request at a time with a contiguous KV
cache grown by ``torch.cat``.  Here any number of requests run concurrently: a request is
prefilled in one pass over its prompt (writing post-norm, post-RoPE keys and values straight
into its pages; requests admitted in the same step share that pass, packed back to back with
the attention kernel taking the sequence boundaries), then joins the decode batch, where every step advances all running requests
by one token with the split-KV paged attention kernel.  Pages return to the free list when a
request finishes.

AttnRes needs no cross-token state at inference: the sources of a routing call are that
token's own block summaries, rebuilt layer by layer (``src/model/llama.py:718-763``), so only
keys and values are cached.

The engine is the scheduler, the page accounting, the decode graphs and the sampling; the layer pipeline and
the contents of the cache belong to the model family's runner (``serve/runners.py``, chosen by
``models/registry.py``).  A family that can continue a cached sequence also takes prompts in portions
(``prefill_portion``) and sequences whose tokens the caller supplies (``open`` / ``feed`` / ``close``): both
go through the same two passes as generation, ``_extend`` (several tokens per request) and ``_decode_pass``
(one token per request).  Sampling follows the reference order repetition penalty ->
temperature -> top-k -> top-p -> multinomial, greedy at temperature 0 (``serve.py:266-304``).
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import Any, Optional

import numpy as np
import torch

from ..ops import get_ops
from .cache import PAGE, PagedKVCache, PagePool  # noqa: F401  (the engine module re-exports its cache)
from .runners import Batch, make_runner


@dataclass
class SamplingParams:
    max_new_tokens: int = 256
    temperature: float = 0.7
    top_k: int = 50
    top_p: float = 0.0
    repetition_penalty: float = 1.0
    eos_token_id: Optional[int] = None
    seed: Optional[int] = None           # of the sampler's random draws; None: derived from the request id


@dataclass
class Request:
    rid: int
    prompt: list[int]
    params: SamplingParams
    pages: list[int] = field(default_factory=list)
    generated: list[int] = field(default_factory=list)
    ctx_len: int = 0
    finished: bool = False
    finish_reason: str = ""
    slot: int = -1                       # row of the engine's seen-token bitmap (repetition penalty)
    prev: int = -1                       # the last token that is in the cache (-1: none): part of the sequence's state
    state: int = -1                      # slot of the recurrent layers' states (families that have them)
    freed: int = 0                       # leading pages that were given back because no later token sees them


def request_seed(r: Request) -> int:
    return r.params.seed if r.params.seed is not None else (0x9E3779B1 * (r.rid + 1) + 12345) & 0x7FFFFFFF


def sample_tokens(logits: torch.Tensor, reqs: list[Request], ops: Any, seen: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Next token per row of ``logits[B,V]``.  All-greedy batches use the argmax kernel; anything else
    goes to the batched sampler of the ops backend (on CUDA one kernel for the whole batch, with
    per-request parameters, seeds and seen-token bitmaps): repetition penalty -> temperature -> top-k
    -> top-p -> multinomial, the reference's order (``serve.py:266-304``)."""
    if all(r.params.temperature == 0 and r.params.repetition_penalty == 1.0 for r in reqs):
        return ops.argmax(logits)
    ps = [r.params for r in reqs]
    slots = [max(r.slot, 0) for r in reqs]
    if seen is None and any(p.repetition_penalty != 1.0 for p in ps):
        # no engine-owned bitmaps (direct use): build them from the requests' token lists
        import numpy as np
        words = np.zeros((len(reqs), (logits.shape[1] + 31) // 32), dtype=np.uint32)
        for b, r in enumerate(reqs):                     # generated tokens only, as the reference's server counts them
            ids = np.unique(np.asarray(r.generated, dtype=np.int64))
            np.bitwise_or.at(words[b], ids >> 5, (np.uint32(1) << (ids & 31).astype(np.uint32)))
        seen = torch.from_numpy(words.view(np.int32)).to(logits.device)
        slots = list(range(len(reqs)))
    return ops.sample(logits, [p.temperature for p in ps], [p.top_k for p in ps], [p.top_p for p in ps],
                      [p.repetition_penalty for p in ps], [request_seed(r) for r in reqs],
                      [len(r.generated) for r in reqs], seen, slots)


class ServingEngine:
    def __init__(self, model: Any, *, device: torch.device | str = "cpu",
                 dtype: torch.dtype = torch.float32, max_batch: int = 64, num_pages: Optional[int] = None,
                 max_ctx: Optional[int] = None, ops: Any = None, tp: Any = None,
                 prefill_batch_tokens: int = 8192, prefill_portion: int = 0) -> None:
        self.device = torch.device(device)
        self.dtype = dtype
        self.model = model.eval()
        self.cfg = model.config
        self.ops = ops or get_ops(self.device)
        self.tp = tp                                  # tensor-parallel helper (``serve.tp``) or None
        self.max_batch = max_batch
        self.max_ctx = max_ctx or self.cfg.max_position_embeddings
        self.runner = make_runner(self)
        self.arena = getattr(self.runner, "arena", None)
        self.H, self.KV = getattr(self.runner, "H", None), getattr(self.runner, "KV", None)     # local heads, where one number describes all layers
        cfg = self.cfg
        if prefill_portion and not self.runner.continues:
            raise ValueError(f"{type(self.runner).__name__} prefills whole prompts only")
        self.prefill_portion = prefill_portion        # most tokens of one prompt per prefill pass; 0: the whole prompt
        pages = num_pages or max_batch * ((self.max_ctx + PAGE - 1) // PAGE)
        self.cache = self.runner.make_cache(pages)
        self.max_pages_per_req = (self.max_ctx + PAGE - 1) // PAGE
        self.waiting: list[Request] = []
        self.running: list[Request] = []
        self._next_id = 0
        # one bitmap row per batch slot: the tokens a request has generated so far, for the repetition penalty of
        # the device sampler (the reference's server penalises generated tokens only, ``serve.py:266-283,345-373``;
        # ``penalise_prompt`` adds the prompt's tokens, the convention of other serving stacks)
        self.penalise_prompt = False
        self.seen_words = (cfg.vocab_size + 31) // 32
        self.seen = torch.zeros(max_batch, self.seen_words, dtype=torch.int32, device=self.device)
        self._free_slots = list(range(max_batch - 1, -1, -1))
        self._dec_states: dict[int, dict] = {}
        self.use_cuda_graphs = True          # decode steps are replayed from captured graphs on CUDA
        # captured decode kernels start while the kernel before them drains (KOTODAMA_DEPENDENT_LAUNCH=0: plain order)
        self.dependent_launch = os.environ.get("KOTODAMA_DEPENDENT_LAUNCH", "1") != "0"
        self.graph_ms: Optional[list[float]] = None      # set to a list to collect the device time of every decode replay
        self._graph_events: list = []
        # when a list: every pass appends ([request ids], fp32 logits on the host) - for tests that compare
        # two engines by logits rather than by sampled tokens
        self.logit_trace: Optional[list] = None
        self.prefill_batch_tokens = prefill_batch_tokens     # tokens of one packed prefill pass over several prompts; 0: one prompt per pass
        self.stats = {"prefill_tokens": 0, "decode_tokens": 0, "prefill_s": 0.0, "decode_s": 0.0, "steps": 0,
                      "prefill_passes": 0}

    # ------------------------------------------------------------------ requests
    def add_request(self, prompt: list[int], params: Optional[SamplingParams] = None) -> Request:
        params = params or SamplingParams()
        if len(prompt) == 0:
            raise ValueError("empty prompt")
        if len(prompt) + 1 > self.max_ctx:
            raise ValueError(f"prompt of {len(prompt)} tokens does not fit the context of {self.max_ctx}")
        need = self.cache.pages_for(min(len(prompt) + params.max_new_tokens, self.max_ctx))
        if need > self.cache.num_pages:
            raise ValueError(f"request needs {need} KV pages, the cache has {self.cache.num_pages}")
        r = Request(self._next_id, list(prompt), params)
        self._next_id += 1
        self.waiting.append(r)
        return r

    def cancel(self, rid: int) -> bool:
        """Ends request ``rid`` now (a client went away, a stop string matched): it leaves the waiting
        queue or the decode batch and its KV pages return to the free list.  Call between steps."""
        for lst in (self.waiting, self.running):
            for r in lst:
                if r.rid == rid:
                    lst.remove(r)
                    self._release(r)
                    r.finished, r.finish_reason = True, "cancelled"
                    return True
        return False

    def has_work(self) -> bool:
        return bool(self.waiting or self.running)

    # ------------------------------------------------------------------ model passes
    @torch.no_grad()
    def _extend(self, parts: list[tuple[Request, list[int]]], rows: Optional[list[int]] = None) -> torch.Tensor:
        """One pass over the next tokens of several requests (a prompt, or a portion of one), packed back to back
        (no padding): the attention takes the sequence boundaries, every other op is per token.  Returns the logits
        at ``rows`` of the packed tokens (default: each request's last)."""
        ns = [len(t) for _, t in parts]
        total = sum(ns)
        ids = torch.empty(total, dtype=torch.long)
        slots = torch.empty(total, dtype=torch.long)
        pos = torch.empty(total, dtype=torch.int32)
        prev = torch.empty(total, dtype=torch.int32)
        cu = [0]
        for (r, toks), n in zip(parts, ns):
            at = cu[-1]
            ids[at:at + n] = torch.tensor(toks, dtype=torch.long)
            prev[at] = r.prev
            prev[at + 1:at + n] = ids[at:at + n - 1].to(torch.int32)
            t = torch.arange(r.ctx_len, r.ctx_len + n)
            slots[at:at + n] = torch.tensor(r.pages, dtype=torch.long)[t // PAGE] * PAGE + t % PAGE
            pos[at:at + n] = t.to(torch.int32)
            cu.append(at + n)
        dev = self.device
        last = torch.tensor(rows if rows is not None else [c - 1 for c in cu[1:]], dtype=torch.long)
        batch = Batch(ids=ids.to(dev), positions=pos.to(dev), slots=slots.to(dev), rows=last.to(dev), prev=prev.to(dev),
                      cu_seqlens=torch.tensor(cu, dtype=torch.int32).to(dev), max_seqlen=max(ns))
        if self.runner.continues:
            ctx = [r.ctx_len + n for (r, _), n in zip(parts, ns)]
            table = np.zeros((len(parts), self.max_pages_per_req), dtype=np.int32)
            for i, (r, _) in enumerate(parts):
                table[i, : len(r.pages)] = r.pages
            batch.page_table = torch.from_numpy(table).to(dev)
            batch.ctx_lens = torch.tensor(ctx, dtype=torch.int32).to(dev)
            batch.cu_context = torch.tensor([0] + np.cumsum(ctx).tolist(), dtype=torch.int32).to(dev)
            batch.total_context = sum(ctx)
            batch.max_ctx = max(ctx)
            batch.spans = [(r.ctx_len, n) for (r, _), n in zip(parts, ns)]
        if self.cache.num_states:
            batch.states = torch.tensor([r.state for r, _ in parts], dtype=torch.int32).to(dev)
        logits = self.runner.forward(batch)
        for (r, toks), n in zip(parts, ns):
            r.ctx_len += n
            r.prev = int(toks[-1])
            self._trim(r)
        self.stats["prefill_tokens"] += total
        self.stats["prefill_passes"] += 1
        return logits

    # ------------------------------------------------------------------ scheduling
    def _prefill(self, parts: list[tuple[Request, list[int]]]) -> None:
        """One prefill pass; requests whose prompt it completes get their first token."""
        logits = self._extend(parts)
        done = [i for i, (r, _) in enumerate(parts) if r.ctx_len >= len(r.prompt)]
        if not done:
            return
        if len(done) < len(parts):
            logits = logits[torch.tensor(done, device=logits.device)]
        reqs = [parts[i][0] for i in done]
        if self.logit_trace is not None:
            self.logit_trace.append(([r.rid for r in reqs], logits.float().cpu()))
        toks = sample_tokens(logits, reqs, self.ops, self.seen).tolist()
        if self.tp is not None:
            toks = self.tp.sync_tokens(toks, self.device)
        for r, tok in zip(reqs, toks):
            self._accept(r, int(tok))

    def _admit(self) -> list[list[tuple[Request, list[int]]]]:
        """Moves the waiting requests that fit (batch slots, pages) to ``running`` and groups the prompt tokens that
        are due - the next portion of every request that is not prefilled yet - into passes of at most
        ``prefill_batch_tokens`` packed tokens (0: one request per pass)."""
        while self.waiting and len(self.running) < self.max_batch:
            r = self.waiting[0]
            need = self.cache.pages_for(min(len(r.prompt) + r.params.max_new_tokens, self.max_ctx))
            if not self.cache.can_allocate(need) or not self.cache.can_take_state():
                break
            # pages are handed out in admission order, which is also the order of the decode batch:
            # neighbouring requests of a decode step then read neighbouring pages
            r.pages = self.cache.allocate(need)
            r.slot = self._free_slots.pop()
            r.state = self.cache.take_state()
            if r.params.repetition_penalty != 1.0:
                self._init_seen(r)
            self.waiting.pop(0)
            self.running.append(r)
        groups: list[list[tuple[Request, list[int]]]] = []
        cur: list[tuple[Request, list[int]]] = []
        for r in self.running:
            if r.ctx_len >= len(r.prompt):
                continue
            n = len(r.prompt) - r.ctx_len
            if self.prefill_portion:
                n = min(n, self.prefill_portion)
            if cur and sum(len(t) for _, t in cur) + n > self.prefill_batch_tokens:
                groups.append(cur)
                cur = []
            cur.append((r, r.prompt[r.ctx_len: r.ctx_len + n]))
        if cur:
            groups.append(cur)
        return groups

    def _init_seen(self, r: Request) -> None:
        """A fresh bitmap row for the request's slot: empty (the sampler sets a bit per generated token), or the
        prompt's tokens when ``penalise_prompt`` is on."""
        words = np.zeros(self.seen_words, dtype=np.uint32)
        if self.penalise_prompt:
            ids = np.unique(np.asarray(r.prompt, dtype=np.int64))
            np.bitwise_or.at(words, ids >> 5, (np.uint32(1) << (ids & 31).astype(np.uint32)))
        self.seen[r.slot].copy_(torch.from_numpy(words.view(np.int32)), non_blocking=True)

    def _trim(self, r: Request) -> None:
        """Gives back the pages in front of everything that later tokens of the sequence can see (their numbers stay in
        the page table, where nothing reads them)."""
        first = self.runner.first_visible(r.ctx_len) // PAGE if self.runner.continues else 0
        if first > r.freed:
            self.cache.release(r.pages[r.freed:first])
            r.freed = first

    def _release(self, r: Request) -> None:
        if r.pages:
            self.cache.release(r.pages[r.freed:])
            r.pages, r.freed = [], 0
        if r.state >= 0:
            self.cache.give_state(r.state)
            r.state = -1
        if r.slot >= 0:
            self._free_slots.append(r.slot)
            r.slot = -1

    def _accept(self, r: Request, tok: int) -> None:
        r.generated.append(tok)
        p = r.params
        if p.eos_token_id is not None and tok == p.eos_token_id:
            r.finished, r.finish_reason = True, "eos"
        elif len(r.generated) >= p.max_new_tokens:
            r.finished, r.finish_reason = True, "length"
        elif r.ctx_len + 1 >= self.max_ctx:
            r.finished, r.finish_reason = True, "context"

    def _decode_inputs(self, reqs: list[Request], tokens: list[int]):
        """Static device buffers for a decode step; the page table is rebuilt only when the set of
        running requests (or the pages they hold) changes."""
        B = len(reqs)
        key = tuple((r.rid, len(r.pages)) for r in reqs)
        # static buffers and captured graphs are kept per batch size: a batch size that comes back
        # (requests of unequal length retire one by one) replays its old graphs
        st = self._dec_states.get(B)
        if st is None:
            # ids | slots (int64), pos | ctx (int32) and, for families whose embedding looks at it, the token before
            # (int32) and, for families with recurrent layers, the state slot (int32) live in ONE device buffer with a
            # pinned host twin: a decode step costs one host -> device copy of 24 (28, 32) bytes per request
            dev = self.device
            at_prev = 24 if self.runner.needs_prev else None
            at_state = (28 if self.runner.needs_prev else 24) if self.cache.num_states else None
            width = 24 + 4 * (at_prev is not None) + 4 * (at_state is not None)
            packed = torch.zeros(width * B, dtype=torch.uint8, device=dev)
            host = torch.zeros(width * B, dtype=torch.uint8, pin_memory=dev.type == "cuda")
            cut = lambda t, lo, hi, dt: t[lo * B: hi * B].view(dt)
            st = {"B": B, "key": None, "packed": packed, "host": host,
                  "ids": cut(packed, 0, 8, torch.long), "slots": cut(packed, 8, 16, torch.long),
                  "pos": cut(packed, 16, 20, torch.int32), "ctx": cut(packed, 20, 24, torch.int32),
                  "h_ids": cut(host, 0, 8, torch.long).numpy(), "h_slots": cut(host, 8, 16, torch.long).numpy(),
                  "h_pos": cut(host, 16, 20, torch.int32).numpy(), "h_ctx": cut(host, 20, 24, torch.int32).numpy(),
                  "prev": cut(packed, at_prev, at_prev + 4, torch.int32) if at_prev else None,
                  "h_prev": cut(host, at_prev, at_prev + 4, torch.int32).numpy() if at_prev else None,
                  "states": cut(packed, at_state, at_state + 4, torch.int32) if at_state else None,
                  "h_states": cut(host, at_state, at_state + 4, torch.int32).numpy() if at_state else None,
                  "table": torch.zeros(B, self.max_pages_per_req, dtype=torch.int32, device=dev),
                  "rows": torch.arange(B, device=dev), "idx": np.arange(B), "graphs": {}}
            self._dec_states[B] = st
        if st["key"] != key:
            table = np.zeros((B, self.max_pages_per_req), dtype=np.int32)
            for i, r in enumerate(reqs):
                table[i, : len(r.pages)] = r.pages
            st["table"].copy_(torch.from_numpy(table), non_blocking=True)
            st["host_table"] = table
            st["key"] = key
        lens = np.fromiter((r.ctx_len for r in reqs), dtype=np.int64, count=B)
        st["h_ids"][:] = tokens
        st["h_slots"][:] = st["host_table"][st["idx"], lens // PAGE].astype(np.int64) * PAGE + lens % PAGE
        st["h_pos"][:] = lens
        st["h_ctx"][:] = lens + 1
        if st["h_prev"] is not None:
            st["h_prev"][:] = np.fromiter((r.prev for r in reqs), dtype=np.int32, count=B)
        if st["h_states"] is not None:
            st["h_states"][:] = np.fromiter((r.state for r in reqs), dtype=np.int32, count=B)
        st["packed"].copy_(st["host"], non_blocking=True)
        return st

    @torch.no_grad()
    def _decode_pass(self, reqs: list[Request], tokens: list[int]) -> tuple[torch.Tensor, Optional[torch.Tensor]]:
        """One token per request against the cache, on CUDA as the replay of a captured graph.  Returns the logits and
        (from a graph) the argmax tokens.  The caller reads something back before the next pass (the host
        twin of the inputs is reused)."""
        st = self._decode_inputs(reqs, tokens)
        max_ctx = max(r.ctx_len for r in reqs) + 1
        # grid of the split-KV kernel, where the family's attention kernel is launched for a context size
        bucket = min(self.max_ctx, ((max_ctx + 511) // 512) * 512) if self.runner.context_buckets else self.max_ctx
        batch = Batch(ids=st["ids"], positions=st["pos"], slots=st["slots"], rows=st["rows"], prev=st["prev"],
                      states=st["states"], page_table=st["table"], ctx_lens=st["ctx"], max_ctx=bucket, decode=True)
        toks = None
        if self.device.type == "cuda" and self.use_cuda_graphs:
            g = st["graphs"].get(bucket)
            if g is None:
                # one eager pass first: lazy initialisation must not happen under capture.  It must not advance the
                # recurrent states either: they are detached (slot -1) until the replay
                if st["states"] is not None:
                    st["states"].fill_(-1)
                self.runner.forward(batch)
                torch.cuda.synchronize()
                st["packed"].copy_(st["host"])
                graph = torch.cuda.CUDAGraph()
                # the captured launches are programmatic dependents of one another (the graph keeps the edges)
                with torch.cuda.graph(graph), self.ops.dependent_launch(self.dependent_launch):
                    logits = self.runner.forward(batch)
                    toks = self.ops.argmax(logits)
                g = st["graphs"][bucket] = (graph, logits, toks)
            if self.graph_ms is not None:            # device time of the replay alone (what the host adds is wall - this)
                ev = (torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True))
                ev[0].record()
                g[0].replay()
                ev[1].record()
                self._graph_events.append(ev)
            else:
                g[0].replay()
            logits, toks = g[1], g[2]
        else:
            logits = self.runner.forward(batch)
        for r, t in zip(reqs, tokens):
            r.ctx_len += 1
            r.prev = int(t)
            self._trim(r)
        self.stats["decode_tokens"] += len(reqs)
        return logits, toks

    def _decode(self, reqs: list[Request]) -> None:
        B = len(reqs)
        greedy = all(r.params.temperature == 0 and r.params.repetition_penalty == 1.0 for r in reqs)
        logits, toks = self._decode_pass(reqs, [r.generated[-1] for r in reqs])
        if toks is None or not greedy:
            toks = sample_tokens(logits, reqs, self.ops, self.seen)
        if self.logit_trace is not None:
            self.logit_trace.append(([r.rid for r in reqs], logits[:B].float().cpu()))
        # one device -> host read per step (under tensor parallelism: of rank 0's tokens, broadcast on the device)
        toks = self.tp.sync_tokens(toks, self.device) if self.tp is not None else toks.tolist()
        if self.graph_ms is not None and self._graph_events:
            self.graph_ms += [a.elapsed_time(b) for a, b in self._graph_events]     # the token read above synchronised
            self._graph_events.clear()
        for r, t in zip(reqs, toks):
            self._accept(r, int(t))

    # ------------------------------------------------------------------ sequences fed by the caller
    def open(self) -> Request:
        """A sequence whose tokens the caller supplies through :meth:`feed`; it holds cache pages until :meth:`close`."""
        if not self.runner.continues:
            raise ValueError(f"{type(self.runner).__name__} cannot continue a cached sequence token by token")
        r = Request(self._next_id, [], SamplingParams())
        self._next_id += 1
        return r

    def feed(self, entries: list[tuple[Request, list[int], list[int]]]) -> list[torch.Tensor]:
        """Advances opened sequences by their next tokens, from the cache that earlier calls left.  An entry is
        ``(sequence, tokens, places)``; returns per entry the fp32 logits on the host, ``[len(places), vocab]``.  A single
        further token takes the decode pass, anything else the packed pass of a prompt."""
        for r, toks, places in entries:
            if not toks:
                raise ValueError("an entry without tokens")
            bad = [t for t in toks if not 0 <= t < self.cfg.vocab_size]
            if bad or any(not 0 <= p < len(toks) for p in places):
                raise ValueError(f"token ids outside the vocabulary ({bad[:3]}) or places outside the tokens")
            n = r.ctx_len + len(toks)
            if n > self.max_ctx:
                raise ValueError(f"sequence of {n} tokens does not fit the context of {self.max_ctx}")
            more = self.cache.pages_for(n) - len(r.pages)
            if more > 0:
                r.pages = r.pages + self.cache.allocate(more)
            if r.state < 0:
                r.state = self.cache.take_state()
        out: list[Any] = [None] * len(entries)
        single = [i for i, (r, toks, _) in enumerate(entries) if len(toks) == 1 and r.ctx_len > 0]
        packed = [i for i in range(len(entries)) if i not in set(single)]
        if single:
            logits, _ = self._decode_pass([entries[i][0] for i in single], [entries[i][1][0] for i in single])
            logits = logits.float().cpu()
            for k, i in enumerate(single):
                out[i] = logits[k:k + 1][[0] * len(entries[i][2])]
        while packed:
            group = [packed.pop(0)]
            while packed and sum(len(entries[i][1]) for i in group + packed[:1]) <= self.prefill_batch_tokens:
                group.append(packed.pop(0))
            rows, at = [], 0
            for i in group:
                rows += [at + p for p in entries[i][2]]
                at += len(entries[i][1])
            logits = self._extend([entries[i][:2] for i in group], rows or [at - 1]).float().cpu()
            at = 0
            for i in group:
                n = len(entries[i][2])
                out[i] = logits[at:at + n]
                at += n
        return out

    def close(self, r: Request) -> None:
        self._release(r)
        r.finished, r.finish_reason = True, "closed"

    def step(self) -> list[Request]:
        """Admit and prefill what fits, advance every running request by one token, retire the
        finished.  Returns the requests that finished in this step."""
        import time
        t0 = time.perf_counter()
        for group in self._admit():
            self._prefill(group)
        t1 = time.perf_counter()
        done = [r for r in self.running if r.finished]
        self.running = [r for r in self.running if not r.finished]
        ready = [r for r in self.running if r.generated]            # the others are still being prefilled
        if ready:
            self._decode(ready)
        done += [r for r in self.running if r.finished]
        self.running = [r for r in self.running if not r.finished]
        for r in done:
            self._release(r)
        self.stats["prefill_s"] += t1 - t0
        self.stats["decode_s"] += time.perf_counter() - t1
        self.stats["steps"] += 1
        return done

    def generate(self, prompts: list[list[int]], params: Optional[SamplingParams] = None) -> list[list[int]]:
        """Convenience: run a set of prompts to completion; returns the generated ids per prompt."""
        reqs = [self.add_request(p, params) for p in prompts]
        while self.has_work():
            self.step()
        return [r.generated for r in reqs]
