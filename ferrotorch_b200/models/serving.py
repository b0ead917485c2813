"""Serving engine for decoder models with a paged row cache and recurrent state slots: ragged batches of prompts, portions of prompts and single tokens through one step
function, a captured decode step, a small continuous-batching scheduler, and an adapter that gives the sampling functions of ``llama_gen`` (greedy,
nucleus, beam, speculative, streaming) the cached-model interface they expect.

A model plugs in with

* ``vocab``, ``dtype``, ``device``, ``cache_rows`` (row length per layer),
* optionally ``state_sizes`` (f32 values of recurrent state per sequence and layer, 0 for none),
* ``prepare(max_positions)``,
* ``forward_rows(batch, cache) -> logits of batch.want``,
* ``decode_supported()``, ``decode_begin(max_batch, max_tokens)`` and ``decode(state, batch_size, cache) -> logits`` (capturable: it reads everything that
  changes from the state's device tensors).

Reference parity: ferrotorch-llama/src/generation.rs:110-404 (generation loop), ferrotorch-nn/src/paged_attention.rs:59-518 (page bookkeeping).
"""
from __future__ import annotations

import weakref
from collections import deque
from dataclasses import dataclass, field
from typing import Callable, Deque, Dict, Iterable, List, Optional, Sequence, Tuple

import torch

from .. import _lib
from ..errors import InvalidArgument
from ..nn.extras import PagedRowCache, PagePool, StateSlots
from .llama_gen import GenerationConfig, sample_next

PAGE = 16
DECODE_ROWS = 16
MEMORY_CHUNK = 128                   # tokens that a recurrent layer takes at once
SEGMENT_MIN, SEGMENT_CTAS = 256, 148


@dataclass
class StepEntry:
    """The next tokens of one sequence and the places among them whose logits are wanted."""
    id: object
    tokens: Sequence[int]
    want: Sequence[int] = ()


@dataclass
class MemoryPlan:
    """How recurrent layers go over the new tokens of a batch. ``segments`` ``[n, 8]``: first row, rows, state slot, sequence, flags (1 the only segment, 2 the last, 4 the
    sequence starts), scratch state; ``inner``: those that are not last (``None`` if there are none); ``chains`` ``[sequences, 4]``: first scratch state, segments, slot,
    whether the sequence starts; ``spans`` ``[sequences, 4]``: first row, rows, slot, whether the sequence starts; ``scratch``: number of scratch states."""
    segments: torch.Tensor
    inner: Optional[torch.Tensor]
    chains: torch.Tensor
    spans: torch.Tensor
    sequences: int
    scratch: int


class RowBatch:
    """Device tables of a ragged batch: one row per new token (``ids``, ``positions``, cache ``slots``, ``seq_of``), the page table of its sequences, and the
    dense context layout that prompt attention over gathered rows uses (``ctx_rows`` of the new tokens, ``past_slots`` -> ``past_rows`` of the cached ones)."""

    def __init__(self, entries: Sequence[StepEntry], cache: PagedRowCache, device, max_blocks: int):
        self.device = device
        ids, pos, slots, seq_of, ctx_rows, past_slots, past_rows, want = [], [], [], [], [], [], [], []
        self._spans: List[Tuple[int, int, int, int]] = []              # first row, rows, position of the first, first context row
        base = 0
        for i, e in enumerate(entries):
            start, n = cache.lengths[e.id], len(e.tokens)
            self._spans.append((len(ids), n, start, base))
            want.extend(len(ids) + w for w in e.want)
            ids.extend(int(t) for t in e.tokens)
            pos.extend(range(start, start + n))
            slots.extend(cache.slots(e.id, start, n))
            seq_of.extend([i] * n)
            ctx_rows.extend(range(base + start, base + start + n))
            if start:
                past_slots.extend(cache.slots(e.id, 0, start))
                past_rows.extend(range(base, base + start))
            base += start + n
        self.rows, self.ctx_total = len(ids), base
        self.single = all(len(e.tokens) == 1 for e in entries)
        self.ids = torch.tensor(ids, dtype=torch.int64).to(device)
        packed = torch.tensor(pos + slots + seq_of + ctx_rows + past_slots + past_rows, dtype=torch.int32).to(device)
        n, m = self.rows, len(past_slots)
        self.positions, self.slots, self.seq_of, self.ctx_rows, ps, pr = torch.split(packed, [n, n, n, n, m, m])
        self.past_slots, self.past_rows = (ps, pr) if m else (None, None)
        self.block_table = cache.block_table([e.id for e in entries], max_blocks).to(device)
        self.want = torch.tensor(want, dtype=torch.int64).to(device) if want else None
        self._state_slots = [cache.states.slot[e.id] for e in entries] if cache.states is not None else []
        self._tiles: Dict[int, torch.Tensor] = {}
        self._query_tiles: Dict[int, torch.Tensor] = {}
        self._plans: Dict[int, MemoryPlan] = {}

    def tiles_for(self, dims) -> Optional[torch.Tensor]:
        """Query tiles ``[tiles, 4]`` (first row, rows, first position, first context row), longest context first; ``None`` when the layer's sizes do not fit
        the tiled prompt kernel."""
        size = dims.flash_tile()
        if size == 0:
            return None
        if size not in self._tiles:
            t = [(r0 + m, min(size, n - m), start + m, base) for r0, n, start, base in self._spans for m in range(0, n, size)]
            t.sort(key=lambda x: -(x[1] + x[2]))
            self._tiles[size] = torch.tensor(t, dtype=torch.int32).to(self.device)
        return self._tiles[size]

    def query_tiles(self, size: int) -> torch.Tensor:
        """Query tiles of up to ``size`` tokens for attention over the pages: ``[tiles, 4]`` (first row, tokens, first position, row of ``block_table``), longest
        context first."""
        if size not in self._query_tiles:
            t = [(r0 + m, min(size, n - m), start + m, i) for i, (r0, n, start, _) in enumerate(self._spans) for m in range(0, n, size)]
            t.sort(key=lambda x: -(x[1] + x[2]))
            self._query_tiles[size] = torch.tensor(t, dtype=torch.int32).to(self.device)
        return self._query_tiles[size]

    def memory_plan(self, ctas: int) -> MemoryPlan:
        """Segments of the new tokens for recurrent layers whose walk takes ``ctas`` CTAs per segment: as many as fill the GPU, none shorter than ``SEGMENT_MIN`` tokens.
        ``ctas`` 0: one segment per sequence."""
        if ctas not in self._plans:
            segs, inner, chains, spans = [], [], [], []
            # an equal share of all new tokens per segment, as many segments as the GPU takes at once
            share = max(SEGMENT_MIN, -(-self.rows // max(1, SEGMENT_CTAS // ctas) // MEMORY_CHUNK) * MEMORY_CHUNK) if ctas else 0
            scratch = 0
            for i, (r0, n, start, _) in enumerate(self._spans):
                size = share or n
                count, slot, fresh = -(-n // size), self._state_slots[i], int(start == 0)
                base = scratch if count > 1 else 0
                for j in range(count):
                    flags = (count == 1) * 1 + (j + 1 == count) * 2 + fresh * 4
                    row = (r0 + j * size, min(size, n - j * size), slot, i, flags, base + j, 0, 0)
                    segs.append(row)
                    if j + 1 < count:
                        inner.append(row)
                chains.append((base, count, slot, fresh))
                spans.append((r0, n, slot, fresh))
                scratch += count if count > 1 else 0
            packed = torch.tensor([x for t in (segs, inner, chains, spans) for r in t for x in r], dtype=torch.int32).to(self.device)
            a, b, c, d = torch.split(packed, [8 * len(segs), 8 * len(inner), 4 * len(chains), 4 * len(spans)])
            self._plans[ctas] = MemoryPlan(a.view(-1, 8), b.view(-1, 8) if inner else None, c.view(-1, 4), d.view(-1, 4), len(chains), scratch)
        return self._plans[ctas]


class DecodeState:
    """Device inputs of the captured decode step; a step advances them, so consecutive greedy steps need nothing from the host."""

    def __init__(self, device, max_blocks: int):
        self.tokens = torch.zeros(DECODE_ROWS, device=device, dtype=torch.int64)
        self._ints = torch.zeros(3 * DECODE_ROWS + DECODE_ROWS * max_blocks, device=device, dtype=torch.int32)
        self.positions, self.seq_lens, self.slots = self._ints[: 3 * DECODE_ROWS].view(3, DECODE_ROWS)
        self.block_table = self._ints[3 * DECODE_ROWS:].view(DECODE_ROWS, max_blocks)
        self.picked = torch.zeros(DECODE_ROWS, device=device, dtype=torch.int64)

    def load(self, tokens: Sequence[int], positions: Sequence[int], block_table: torch.Tensor, slots: Optional[Sequence[int]] = None) -> None:
        B = len(tokens)
        host = torch.zeros(3, DECODE_ROWS, dtype=torch.int32)
        host[0, :B] = torch.tensor(list(positions), dtype=torch.int32)
        host[1, :B] = host[0, :B] + 1
        if slots is not None:
            host[2, :B] = torch.tensor(list(slots), dtype=torch.int32)
        used = block_table.reshape(-1)
        self._ints[: 3 * DECODE_ROWS + used.numel()].copy_(torch.cat([host.reshape(-1), used]))
        self.tokens[:B].copy_(torch.tensor(list(tokens), dtype=torch.int64))


class ServingEngine:
    """``engine.step(entries)`` runs the tokens it is given on top of what earlier steps left in the cache; ``engine.generate(prompts, config)`` schedules whole
    requests. ``max_tokens`` bounds the tokens of all live sequences together."""

    def __init__(self, model, max_tokens: int = 4096, max_sequences: int = 64, use_graph: bool = True, prefill_chunk: int = 8192):
        if max_tokens < 1 or max_sequences < 1:
            raise InvalidArgument("ServingEngine: max_tokens and max_sequences must be positive")
        self.model, self.device = model, torch.device(model.device)
        self.max_tokens, self.max_sequences, self.prefill_chunk = max_tokens, max_sequences, prefill_chunk
        self.max_blocks = -(-max_tokens // PAGE)
        # a sequence wastes at most one page beyond its tokens
        self.pool = PagePool(self.max_blocks + max_sequences, PAGE)
        sizes = getattr(model, "state_sizes", ())
        self.states = StateSlots(max_sequences, sizes, self.device) if any(sizes) else None
        self.cache = PagedRowCache(self.pool, model.cache_rows, self.device, model.dtype, self.states)
        self._fed: Dict[object, List[int]] = {}               # tokens of live sequences, kept where a state can only be rebuilt from them
        model.prepare(self.max_blocks * PAGE)
        self.use_graph = use_graph
        self.graphs: Dict[int, Tuple[torch.cuda.CUDAGraph, torch.Tensor]] = {}
        self.fast_decode = model.decode_supported()
        if self.fast_decode:
            self.state = DecodeState(self.device, self.max_blocks)
            model.decode_begin(DECODE_ROWS, self.max_blocks * PAGE)

    # -- sequences -------------------------------------------------------------
    def __contains__(self, seq_id) -> bool:
        return seq_id in self.cache.tables

    def length(self, seq_id) -> int:
        return self.cache.lengths[seq_id]

    def release(self, seq_id) -> None:
        """Gives back what a finished sequence holds."""
        self.cache.free_sequence(seq_id)
        self._fed.pop(seq_id, None)

    def fork(self, src, dst) -> None:
        """A new sequence ``dst`` that continues from where ``src`` is: pages are shared until one of them writes, recurrent state is copied."""
        self.cache.fork(src, dst)
        if src in self._fed:
            self._fed[dst] = list(self._fed[src])

    def truncate(self, seq_id, n: int) -> None:
        """Forgets every token from position ``n`` on. Recurrent state cannot step back: its remaining tokens are run again."""
        if self.states is None or not 0 < n < self.length(seq_id):
            self.cache.truncate(seq_id, n)
            if seq_id in self._fed:
                del self._fed[seq_id][n:]
            return
        tokens = self._fed.pop(seq_id)[:n]
        self.cache.truncate(seq_id, 0)
        self.step([StepEntry(seq_id, tokens)])

    # -- steps -----------------------------------------------------------------
    def _admit(self, entries: Sequence[StepEntry]) -> None:
        seen = set()
        for e in entries:
            if e.id in seen:
                raise InvalidArgument(f"step: sequence {e.id!r} appears twice")
            seen.add(e.id)
            if len(e.tokens) == 0:
                raise InvalidArgument(f"step: no tokens for sequence {e.id!r}")
            if min(e.tokens) < 0 or max(e.tokens) >= self.model.vocab:
                raise InvalidArgument(f"step: token outside the vocabulary ({self.model.vocab})")
            if any(w < 0 or w >= len(e.tokens) for w in e.want):
                raise InvalidArgument("step: wanted place outside the entry's tokens")
        need = 0
        for e in entries:
            total = (self.cache.lengths[e.id] if e.id in self else 0) + len(e.tokens)
            if total > self.max_blocks * PAGE:
                raise InvalidArgument(f"step: sequence {e.id!r} would grow to {total} tokens, the cache holds {self.max_blocks * PAGE}")
            need += self.cache.pages_for(e.id, total)
        if need > self.pool.num_free():
            raise InvalidArgument(f"step: {need} more cache pages needed, {self.pool.num_free()} free")
        if self.states is not None and sum(e.id not in self for e in entries) > self.states.num_free():
            raise InvalidArgument(f"step: more new sequences than free state slots ({self.states.num_free()})")
        for e in entries:
            if e.id not in self:
                self.cache.add_sequence(e.id)
            self.cache.reserve(e.id, self.cache.lengths[e.id] + len(e.tokens))

    @torch.no_grad()
    def step(self, entries: Sequence[StepEntry], end: Iterable = (), taps: Optional[list] = None) -> Optional[torch.Tensor]:
        """Logits ``[wanted, vocab]`` (f32) in the order of the entries and of their ``want``, or ``None`` when nothing is wanted. Sequences named in
        ``end`` are released afterwards. ``taps`` (a list) collects the residual after every layer instead of using the captured decode step."""
        entries = list(entries)
        self._admit(entries)
        out = None
        if entries:
            if self.fast_decode and taps is None and all(len(e.tokens) == 1 for e in entries):
                parts = [self._decode(entries[i: i + DECODE_ROWS]) for i in range(0, len(entries), DECODE_ROWS)]
                parts = [p for p in parts if p is not None]
                out = torch.cat(parts) if parts else None
            else:
                batch = RowBatch(entries, self.cache, self.device, self.max_blocks)
                out = self.model.forward_rows(batch, self.cache, taps)
            for e in entries:
                self.cache.lengths[e.id] += len(e.tokens)
                if self.states is not None:
                    self._fed.setdefault(e.id, []).extend(int(t) for t in e.tokens)
        for s in end:
            self.release(s)
        return out

    def _decode(self, entries: Sequence[StepEntry]) -> Optional[torch.Tensor]:
        B = len(entries)
        self._load_state([e.id for e in entries], [e.tokens[0] for e in entries])
        logits = self._decode_launch(B)
        rows = [i for i, e in enumerate(entries) for _ in e.want]
        if not rows:
            return None
        return logits[:B].clone() if rows == list(range(B)) else logits[torch.tensor(rows, device=self.device)]

    def _load_state(self, ids: Sequence, tokens: Sequence[int]) -> None:
        slots = None if self.states is None else [self.states.slot[s] for s in ids]
        self.state.load(tokens, [self.cache.lengths[s] for s in ids], self.cache.block_table(ids, self.max_blocks), slots)

    def _decode_body(self, B: int) -> torch.Tensor:
        """One decode step of the first ``B`` rows of the state. Its kernels are launched as programmatic dependents (each is scheduled while its
        predecessor drains and waits for it on the device)."""
        prev = _lib.kernels().ft_set_pdl(1)
        try:
            logits = self.model.decode(self.state, B, self.cache)
        finally:
            _lib.kernels().ft_set_pdl(prev)
        s = self.state
        torch.argmax(logits[:B], -1, out=s.picked[:B])
        s.tokens[:B].copy_(s.picked[:B])
        s.positions[:B] += 1
        s.seq_lens[:B] += 1
        return logits

    def _decode_launch(self, B: int) -> torch.Tensor:
        if not self.use_graph:
            return self._decode_body(B)
        if B not in self.graphs:
            s = self.state
            saved = [t.clone() for t in (s.tokens, s._ints)]
            if self.states is not None:
                s.slots.fill_(self.states.spare)                # the first run below must not advance anybody's state
            side = torch.cuda.Stream(self.device)
            side.wait_stream(torch.cuda.current_stream())
            with torch.cuda.stream(side):                       # lazy initialisation outside the capture; its cache write is simply redone
                self._decode_body(B)
            torch.cuda.current_stream().wait_stream(side)
            torch.cuda.synchronize(self.device)
            s.tokens.copy_(saved[0]); s._ints.copy_(saved[1])
            graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(graph):
                logits = self._decode_body(B)
            self.graphs[B] = (graph, logits)
        graph, logits = self.graphs[B]
        graph.replay()
        return logits

    @torch.no_grad()
    def decode_greedy(self, seq_ids: Sequence, tokens: Sequence[int], steps: int) -> List[List[int]]:
        """``steps`` greedy tokens for up to sixteen live sequences, fed back on the device: the host only launches."""
        if len(seq_ids) > DECODE_ROWS or not self.fast_decode:
            raise InvalidArgument(f"decode_greedy takes up to {DECODE_ROWS} sequences of a model with a captured decode step")
        need = sum(self.cache.pages_for(s, self.cache.lengths[s] + steps) for s in seq_ids)
        if need > self.pool.num_free() or any(self.cache.lengths[s] + steps > self.max_blocks * PAGE for s in seq_ids):
            raise InvalidArgument("decode_greedy: not enough cache pages")
        for s in seq_ids:
            self.cache.reserve(s, self.cache.lengths[s] + steps)
        B = len(seq_ids)
        self._load_state(seq_ids, tokens)
        out = torch.empty(steps, B, device=self.device, dtype=torch.int64)
        for i in range(steps):
            self._decode_launch(B)
            out[i].copy_(self.state.picked[:B])
        rows = out.t().tolist()
        for s, t, row in zip(seq_ids, tokens, rows):
            self.cache.lengths[s] += steps
            if self.states is not None:
                self._fed[s].extend([int(t), *row[:-1]])
        return rows

    # -- whole requests --------------------------------------------------------
    def generate(self, prompts: Sequence[Sequence[int]], config: Optional[GenerationConfig] = None, streamer: Optional[Callable[[int, int], None]] = None) -> List[List[int]]:
        """New tokens of every prompt (the stop token included). Prompts of any lengths; more than fit at once wait for their turn."""
        sched = Scheduler(self, config or GenerationConfig(), streamer)
        for p in prompts:
            sched.submit([int(t) for t in p])
        return sched.run()

    def as_cached_model(self) -> "CachedEngineModel":
        return CachedEngineModel(self)

    def check(self) -> None:
        st = _lib.read_status()
        if st:
            from ..errors import Timeout
            raise Timeout(message=f"device-side wait timed out (status {st:#x})")


@dataclass
class _Request:
    index: int
    prompt: List[int]
    fed: int = 0
    out: List[int] = field(default_factory=list)
    gen: Optional[torch.Generator] = None

    @property
    def key(self):
        return ("request", id(self), self.index)


class Scheduler:
    """Continuous batching: waiting prompts are admitted while the cache can hold them to their last token, prefilled in portions of at most
    ``prefill_chunk`` tokens a step, and decoded together with everything that is already running."""

    def __init__(self, engine: ServingEngine, config: GenerationConfig, streamer: Optional[Callable[[int, int], None]] = None):
        if config.num_beams > 1:
            raise InvalidArgument("beam search runs through generate(engine.as_cached_model(), ...)")
        self.engine, self.config, self.streamer = engine, config, streamer
        self.waiting: Deque[_Request] = deque()
        self.prefilling: List[_Request] = []
        self.running: List[_Request] = []
        self.finished: Dict[int, List[int]] = {}
        self.reserved = 0                                     # pages promised to admitted requests
        self.count = 0
        self.stops = set(config.stop_ids())

    def submit(self, prompt: List[int]) -> int:
        if not prompt:
            raise InvalidArgument("generate: a prompt must not be empty")
        r = _Request(self.count, list(prompt))
        if self._pages(r) > self.engine.max_blocks:
            raise InvalidArgument(f"generate: prompt {r.index} and its new tokens do not fit the cache ({self.engine.max_tokens} tokens)")
        if self.config.do_sample:
            r.gen = torch.Generator(device=self.engine.device).manual_seed((self.config.seed or 0) + r.index)
        self.count += 1
        self.waiting.append(r)
        return r.index

    def _pages(self, r: _Request) -> int:
        return -(-(len(r.prompt) + self.config.max_new_tokens) // PAGE)

    def _live(self) -> int:
        return len(self.prefilling) + len(self.running)

    def _take(self, r: _Request, token: int) -> bool:
        """Records a new token; True while the request goes on."""
        r.out.append(token)
        if self.streamer is not None:
            self.streamer(r.index, token)
        if token in self.stops or len(r.out) >= self.config.max_new_tokens:
            self.engine.release(r.key)
            self.reserved -= self._pages(r)
            self.finished[r.index] = r.out
            return False
        return True

    def _sample(self, reqs: List[_Request], logits: torch.Tensor) -> List[int]:
        c = self.config
        if not c.do_sample and c.repetition_penalty == 1.0:
            return logits.argmax(-1).tolist()
        out = []
        for i, r in enumerate(reqs):
            seq = torch.tensor([r.prompt + r.out], device=logits.device)
            out.append(int(sample_next(logits[i: i + 1], seq, c, r.gen)))
        return out

    def tick(self) -> None:
        """One round: admit, one prompt step, one decode step."""
        eng = self.engine
        while self.waiting and self._live() < eng.max_sequences and self.reserved + self._pages(self.waiting[0]) <= eng.max_blocks:
            r = self.waiting.popleft()
            self.reserved += self._pages(r)
            self.prefilling.append(r)
        decoding = list(self.running)
        if self.prefilling:
            room, entries, done = eng.prefill_chunk, [], []
            for r in list(self.prefilling):
                if room <= 0:
                    break
                part = r.prompt[r.fed: r.fed + room]
                room -= len(part)
                r.fed += len(part)
                last = r.fed == len(r.prompt)
                entries.append(StepEntry(r.key, part, [len(part) - 1] if last else []))
                if last:
                    done.append(r)
                    self.prefilling.remove(r)
            logits = eng.step(entries)
            if done:
                for r, t in zip(done, self._sample(done, logits)):
                    if self._take(r, t):
                        self.running.append(r)
        if decoding:
            c = self.config
            left = min(c.max_new_tokens - len(r.out) for r in decoding)
            simple = not self.stops and self.streamer is None and not c.do_sample and c.repetition_penalty == 1.0
            if simple and eng.fast_decode and not self.waiting and not self.prefilling and len(self.running) == len(decoding) <= DECODE_ROWS and left > 1:
                rows = eng.decode_greedy([r.key for r in decoding], [r.out[-1] for r in decoding], left)
                kept = [r for r, row in zip(decoding, rows) if all([self._take(r, t) for t in row])]
            else:
                logits = eng.step([StepEntry(r.key, [r.out[-1]], [0]) for r in decoding])
                kept = [r for r, t in zip(decoding, self._sample(decoding, logits)) if self._take(r, t)]
            self.running = kept + [r for r in self.running if r not in decoding]

    def run(self) -> List[List[int]]:
        if self.config.max_new_tokens < 1:
            return [[] for _ in range(self.count)]
        try:
            while self.waiting or self.prefilling or self.running:
                self.tick()
        finally:
            for r in self.prefilling + self.running:
                self.engine.release(r.key)
        return [self.finished[i] for i in range(self.count)]


class EngineCache:
    """Cache handle for the cached-model interface: the sequences of one batch in an engine's page cache, released with the handle."""

    def __init__(self, engine: ServingEngine):
        self._engine = engine
        self.ids: List[object] = []
        self._token = object()
        self._serial = 0
        self._held: List[object] = []
        weakref.finalize(self, EngineCache._free, engine, self._held)

    @staticmethod
    def _free(engine, held) -> None:
        for s in held:
            engine.release(s)

    def _new_ids(self, n: int) -> List[object]:
        self._serial += 1
        ids = [("cache", id(self._token), self._serial, i) for i in range(n)]
        self._held.extend(ids)
        return ids

    def open(self, n: int) -> None:
        if not self.ids:
            self.ids = self._new_ids(n)
        elif len(self.ids) != n:
            raise InvalidArgument(f"the cache holds {len(self.ids)} sequences, the batch has {n}")

    def len(self) -> int:  # noqa: A003
        return self._engine.length(self.ids[0]) if self.ids and self.ids[0] in self._engine else 0

    def truncate(self, n: int) -> None:
        for s in self.ids:
            self._engine.truncate(s, n)

    def _replace(self, sources: List[object]) -> None:
        new = self._new_ids(len(sources))
        for d, s in zip(new, sources):
            self._engine.fork(s, d)
        for s in self.ids:
            self._engine.release(s)
            self._held.remove(s)
        self.ids = new

    def expand(self, n: int) -> None:
        self._replace([self.ids[0]] * n)

    def reorder(self, index: torch.Tensor) -> None:
        self._replace([self.ids[i] for i in index.tolist()])


class CachedEngineModel:
    """``model(ids [B, S], cache) -> logits [B, S, vocab]`` over a :class:`ServingEngine`, the interface of :class:`CachedLlama`: what ``generate``,
    ``generate_with_streamer``, ``beam_search`` and the speculative decoders take."""

    def __init__(self, engine: ServingEngine):
        self.engine, self.device, self.cfg = engine, engine.device, engine.model.cfg

    def new_cache(self) -> EngineCache:
        return EngineCache(self.engine)

    def __call__(self, ids: torch.Tensor, cache: EngineCache) -> torch.Tensor:
        B, S = ids.shape
        cache.open(B)
        rows = ids.tolist()
        out = self.engine.step([StepEntry(s, rows[i], range(S)) for i, s in enumerate(cache.ids)])
        return out.view(B, S, -1)


class CachedModelEngine:
    """The step interface over a cached model ``model(ids, cache)`` with a cache of its own per sequence (e.g. :class:`CachedLlama`)."""

    def __init__(self, model, vocab: int, device="cpu"):
        self.model, self.vocab, self.device = model, vocab, torch.device(device)
        self._caches: Dict[object, object] = {}

    def __contains__(self, seq_id) -> bool:
        return seq_id in self._caches

    def length(self, seq_id) -> int:
        return self._caches[seq_id].len()

    def release(self, seq_id) -> None:
        self._caches.pop(seq_id, None)

    @torch.no_grad()
    def step(self, entries: Sequence[StepEntry], end: Iterable = ()) -> Optional[torch.Tensor]:
        out = []
        for e in entries:
            c = self._caches.setdefault(e.id, None) or self.model.new_cache()
            self._caches[e.id] = c
            logits = self.model(torch.tensor([list(e.tokens)], dtype=torch.long, device=self.device), c)[0]
            out.extend(logits[w] for w in e.want)
        for s in end:
            self.release(s)
        return torch.stack(out).float() if out else None

    def generate(self, prompts: Sequence[Sequence[int]], config: Optional[GenerationConfig] = None) -> List[List[int]]:
        from .llama_gen import generate
        out = []
        for p in prompts:
            ids = torch.tensor([list(p)], dtype=torch.long, device=self.device)
            out.append(generate(self.model, self.model.new_cache, ids, config)[0, len(p):].tolist())
        return out

    def as_cached_model(self):
        return self.model
