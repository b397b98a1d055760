"""Serving: cache and state slots, scheduling, one model step, sampling.

``CacheManager`` hands out K/V pages and state slots, ``Scheduler`` decides which sequences advance by how many tokens,
``ModelRunner`` turns that into a ``StepBatch`` and runs the model (steps of decoding sequences only are replayed from a
CUDA graph per batch size), ``sample`` picks tokens.  ``Engine`` ties them together:

    engine = Engine(load_model(folder))
    engine.generate([[1, 5, 7], [2, 2]], SamplingParams(max_new_tokens=32))

    engine.feed([("a", [5, 17, 3], [0, 2])])        # given tokens, logits at given places, nothing sampled
    engine.release("a")
"""

from collections import deque
from dataclasses import dataclass, field

import numpy as np
import torch

TILE_ROWS = 128                       # query rows of one tensor-core tile


# ---- one step's input ------------------------------------------------------------------------------------------------
@dataclass
class RowGroup:
    """Sequences of a step that take the same kernels: the decoding ones (one row each) or the prompt portions.
    Device tensors; row numbers are relative to the group's first row."""
    rows: slice                       # the group's rows in the step
    n_seqs: int
    max_rows: int
    total_rows: int
    cu_rows: torch.Tensor             # (n_seqs + 1,) int32
    start_pos: torch.Tensor           # (n_seqs,) int32 position of a sequence's first row; negative = padded
    slots: torch.Tensor               # (n_seqs,) int64 state slot; negative = padded
    block_tables: torch.Tensor        # (n_seqs, max_blocks) int32
    row_seq: torch.Tensor = None      # (total_rows,) int32 (prompt portions)
    tile_seq: torch.Tensor = None     # 128-row query tiles: sequence and first row inside it
    tile_row: torch.Tensor = None
    lengths: tuple = ()               # host copies of the portions' lengths and slots
    host_slots: tuple = ()


@dataclass
class StepBatch:
    ids: torch.Tensor                 # (rows,) int32; decoding sequences first
    prev: torch.Tensor                # (rows,) int32 the token before, -1 at a sequence's start
    positions: torch.Tensor           # (rows,) int32
    slot_mapping: torch.Tensor        # (rows,) int64 cache row, -1 = none
    decode: RowGroup = None
    prefill: RowGroup = None
    logit_rows: torch.Tensor = None   # (n,) int64 rows whose logits are asked for, None = none


# ---- sequences, pages and slots --------------------------------------------------------------------------------------
@dataclass
class SamplingParams:
    max_new_tokens: int = 16
    temperature: float = 0.0          # 0 = greedy
    top_k: int = 0                    # 0 = all
    top_p: float = 1.0
    stop_ids: tuple = ()
    seed: int = None


@dataclass
class Sequence:
    name: object
    tokens: list
    params: SamplingParams = field(default_factory=SamplingParams)
    prompt_len: int = 0
    done: int = 0                     # tokens whose keys and state are in the cache
    slot: int = -1
    pages: list = field(default_factory=list)     # page of every block of tokens, -1 = given back
    dropped: int = 0                  # blocks below this one have been looked at for giving back
    promised_blocks: int = 0          # blocks of tokens admitted for, 0 = no promise
    reserved: int = 0                 # pages promised and not taken yet
    generator: torch.Generator = None

    @property
    def output(self):
        return self.tokens[self.prompt_len:]


class OutOfCache(RuntimeError):
    pass


class CacheManager:
    """Free lists of K/V pages and state slots.  Nothing is cleared on release: a sequence's first token starts its state
    from zero and only keys at its own positions are read.

    ``reach`` = (window, first): no layer looks back past a position's last ``window`` keys except at the first ``first``
    ones, so a sequence gives back the pages in between as it grows and holds at most ``live_pages`` at a time when it
    advances by up to ``max_portion`` tokens a step (None: every key stays)."""

    def __init__(self, num_blocks, block_size, max_seqs, max_blocks_per_seq, reach=None, max_portion=None):
        self.num_blocks, self.block_size, self.max_seqs, self.max_blocks_per_seq = num_blocks, block_size, max_seqs, max_blocks_per_seq
        self.reach, self.max_portion = reach, max_portion
        self.free_pages, self.free_slots = deque(range(num_blocks)), deque(range(max_seqs))
        self.promised = 0

    def pages_for(self, tokens):
        return -(-tokens // self.block_size)

    def live_pages(self, total_tokens):
        """The most pages that a sequence of ``total_tokens`` holds at any time."""
        need = self.pages_for(total_tokens)
        if self.reach is None or self.max_portion is None:
            return need
        window, first = self.reach
        return min(need, self.pages_for(first) + self.pages_for(window + self.max_portion) + 1)

    def admit(self, seq, total_tokens=0):
        """A slot, and the promise of pages for ``total_tokens``; False if there is no room."""
        blocks, need = self.pages_for(total_tokens), self.live_pages(total_tokens)
        if blocks > self.max_blocks_per_seq:
            raise ValueError(f"a sequence of {total_tokens} tokens exceeds the longest one this cache serves "
                             f"({self.max_blocks_per_seq * self.block_size})")
        if not self.free_slots or need > len(self.free_pages) - self.promised:
            return False
        seq.slot = self.free_slots.popleft()
        seq.promised_blocks, seq.reserved = blocks, need
        self.promised += need
        return True

    def _drop_unseen(self, seq):
        """Gives back the pages that no token after the first ``seq.done`` can see; what a promise still needs of them
        stays promised."""
        window, first = self.reach
        keep, end = self.pages_for(first), max(seq.done + 1 - window, 0) // self.block_size       # blocks in [keep, end) are out of sight
        for b in range(max(seq.dropped, keep), min(end, len(seq.pages))):
            self.free_pages.append(seq.pages[b])
            seq.pages[b] = -1
            if seq.reserved < seq.promised_blocks - len(seq.pages):
                seq.reserved += 1
                self.promised += 1
        seq.dropped = max(seq.dropped, end)

    def extend(self, seq, tokens):
        """Pages for the sequence's first ``tokens`` tokens, of which ``seq.done`` are in the cache."""
        if self.reach is not None:
            self._drop_unseen(seq)
        need = self.pages_for(tokens)
        if need > self.max_blocks_per_seq:
            raise OutOfCache(f"a sequence of {tokens} tokens exceeds {self.max_blocks_per_seq * self.block_size}")
        while len(seq.pages) < need:
            if seq.reserved > 0:
                seq.reserved -= 1
                self.promised -= 1
            elif len(self.free_pages) <= self.promised:
                raise OutOfCache("no free page")
            seq.pages.append(self.free_pages.popleft())

    def release(self, seq):
        self.free_pages.extend(p for p in seq.pages if p >= 0)
        self.promised -= seq.reserved
        seq.reserved = seq.promised_blocks = seq.dropped = 0
        if seq.slot >= 0:
            self.free_slots.append(seq.slot)
        seq.pages, seq.slot = [], -1


class Scheduler:
    """First come, first served.  Every running sequence that has its prompt behind it decodes one token; what is left of
    the step's token budget goes to prompts, in portions if the model allows it."""

    def __init__(self, cache, max_step_tokens, chunked_prefill, mixed_batches):
        self.cache, self.max_step_tokens = cache, max_step_tokens
        self.chunked, self.mixed = chunked_prefill, mixed_batches
        self.waiting, self.running = deque(), []

    def add(self, seq):
        self.waiting.append(seq)

    def _admit(self):
        while self.waiting:
            seq = self.waiting[0]
            if not self.cache.admit(seq, seq.prompt_len + seq.params.max_new_tokens):
                if not self.running:
                    raise OutOfCache("the cache is too small for one sequence")
                return
            self.running.append(self.waiting.popleft())

    def schedule(self):
        """[(sequence, new tokens)]: one-token entries first, then longer prompt portions."""
        self._admit()
        decoding = [s for s in self.running if len(s.tokens) - s.done == 1]
        prompts = [s for s in self.running if len(s.tokens) - s.done > 1]
        if not self.chunked:                                # a one-token prompt is a prompt too
            prompts += [s for s in decoding if s.done == 0]
            decoding = [s for s in decoding if s.done > 0]
        plan = []
        if prompts and not self.mixed:
            decoding = []
        budget = self.max_step_tokens
        for s in decoding:
            if budget > 0:
                plan.append((s, 1))
                budget -= 1
        for s in prompts:
            n = len(s.tokens) - s.done
            if n > budget and (self.chunked or not plan):
                n = budget if self.chunked else n           # a model without portions takes an oversized prompt alone
            if n <= 0 or n > max(budget, 0) and plan:
                continue
            plan.append((s, n))
            budget -= n
        if self.chunked:
            plan.sort(key=lambda e: e[1] != 1)              # a portion of one token runs like a decoding sequence
        return plan

    def finish(self, seq):
        self.running.remove(seq)
        self.cache.release(seq)


# ---- running the model -----------------------------------------------------------------------------------------------
class ModelRunner:
    def __init__(self, model, cache, state, graphs=True):
        self.model, self.cache, self.state, self.device = model, cache, state, model.device
        self.graphs = {} if graphs and model.graph_decode else None

    # -- building a step ------------------------------------------------------------------------------------------
    def _group_ints(self, plan, width):
        """Host arrays of one group: (cu, start, block table rows)."""
        lens = np.array([n for _, n in plan], np.int64)
        cu = np.zeros(len(plan) + 1, np.int64)
        np.cumsum(lens, out=cu[1:])
        start = np.array([s.done for s, _ in plan], np.int64)
        tables = np.zeros((len(plan), width), np.int64)
        for i, (s, _) in enumerate(plan):
            tables[i, :len(s.pages)] = s.pages                             # -1 where a page was given back: never read
        return lens, cu, start, tables

    def build(self, plan, want_rows, pad_decode_to=None):
        """plan: [(sequence, new tokens)] with one-token entries first; want_rows: step rows whose logits are wanted.
        ``pad_decode_to``: fill a step of decoding sequences up with padded ones."""
        bs = self.cache.block_size
        as_decode = lambda s, n: n == 1 and (self.model.chunked_prefill or s.done > 0)
        n_dec = 0
        while n_dec < len(plan) and as_decode(*plan[n_dec]):
            n_dec += 1
        if any(as_decode(*e) for e in plan[n_dec:]):
            raise ValueError("decoding sequences come first in a step")
        width = self.cache.max_blocks_per_seq if pad_decode_to is not None else max(max((len(s.pages) for s, _ in plan), default=1), 1)
        lens, cu, start, tables = self._group_ints(plan, width)
        total = int(cu[-1])
        ids, prev = np.empty(total, np.int64), np.empty(total, np.int64)
        for i, (s, n) in enumerate(plan):
            ids[cu[i]:cu[i + 1]] = s.tokens[s.done:s.done + n]
            prev[cu[i]] = s.tokens[s.done - 1] if s.done > 0 else -1
            prev[cu[i] + 1:cu[i + 1]] = s.tokens[s.done:s.done + n - 1]
        seq_of = np.repeat(np.arange(len(plan)), lens)
        pos = start[seq_of] + np.arange(total) - cu[:-1][seq_of]
        slot_map = tables[seq_of, pos // bs] * bs + pos % bs
        slots = np.array([s.slot for s, _ in plan], np.int64)
        pad = 0 if pad_decode_to is None else pad_decode_to - n_dec
        if pad > 0:
            z, neg = np.zeros(pad, np.int64), np.full(pad, -1, np.int64)
            ids, prev, pos, slot_map = (np.concatenate(p) for p in ((ids, z), (prev, neg), (pos, neg), (slot_map, neg)))
            start, slots = np.concatenate((start, neg)), np.concatenate((slots, neg))
            tables = np.concatenate((tables, np.zeros((pad, width), np.int64)))
            n_dec = total = pad_decode_to

        parts32, parts64 = [ids, prev, pos], [slot_map, slots]
        shapes = {}
        nd = n_dec
        if nd:
            parts32 += [np.arange(nd + 1), start[:nd], tables[:nd].reshape(-1)]
        n_pre = len(slots) - nd
        if n_pre:
            pl = lens[nd:]
            tiles = -(-pl // TILE_ROWS)
            t_seq = np.repeat(np.arange(n_pre), tiles)
            first = np.concatenate(([0], np.cumsum(tiles)))[:-1]
            t_row = (np.arange(int(tiles.sum())) - first[t_seq]) * TILE_ROWS
            order = np.argsort(-(start[nd:][t_seq] + t_row), kind="stable")        # the tiles with the most keys first
            parts32 += [cu[nd:] - cu[nd], start[nd:], tables[nd:].reshape(-1), np.repeat(np.arange(n_pre), pl), t_seq[order], t_row[order]]
        parts64.append(np.asarray(want_rows, np.int64))
        d32, d64 = self._upload(parts32, np.int32), self._upload(parts64, np.int64)
        batch = StepBatch(ids=d32[0], prev=d32[1], positions=d32[2], slot_mapping=d64[0], logit_rows=d64[2] if len(want_rows) else None)
        at = 3
        if nd:
            batch.decode = RowGroup(slice(0, nd), nd, 1, nd, d32[at], d32[at + 1], d64[1][:nd], d32[at + 2].view(nd, width))
            at += 3
        if n_pre:
            r0 = int(cu[nd]) if nd else 0
            batch.prefill = RowGroup(slice(r0, total), n_pre, int(pl.max()), total - r0, d32[at], d32[at + 1], d64[1][nd:],
                                     d32[at + 2].view(n_pre, width), d32[at + 3], d32[at + 4], d32[at + 5], tuple(int(n) for n in pl),
                                     tuple(int(s) for s in slots[nd:]))
        return batch

    def _upload(self, parts, dtype):
        """One host-to-device copy for several index arrays; each starts on a 16-byte boundary."""
        unit = 16 // np.dtype(dtype).itemsize
        offs, at = [], 0
        for p in parts:
            offs.append(at)
            at += -(-max(p.size, 1) // unit) * unit
        host = np.zeros(at, dtype)
        for o, p in zip(offs, parts):
            host[o:o + p.size] = p
        t = torch.from_numpy(host)
        dev = t.to(self.device) if self.device.type != "cuda" else t.pin_memory().to(self.device, non_blocking=True)
        return [dev[o:o + p.size] for o, p in zip(offs, parts)]

    # -- running it --------------------------------------------------------------------------------------------------
    def step(self, plan, want_rows):
        """Runs one step and advances the sequences.  Returns fp32 logits of ``want_rows`` (None if there are none)."""
        for s, n in plan:
            self.cache.extend(s, s.done + n)
        decode_only = all(n == 1 and (self.model.chunked_prefill or s.done > 0) for s, n in plan)
        if decode_only and self.graphs is not None:
            logits = self._graph_step(plan)
            if len(want_rows) != logits.shape[0] or list(want_rows) != list(range(logits.shape[0])):
                logits = logits[torch.as_tensor(list(want_rows), dtype=torch.int64, device=logits.device)] if len(want_rows) else None
        else:
            logits = self.model.forward(self.build(plan, want_rows), self.state)
        for s, n in plan:
            s.done += n
        return logits

    def _graph_step(self, plan):
        bucket = 1
        while bucket < len(plan):
            bucket *= 2
        bucket = min(bucket, max(self.cache.max_seqs, len(plan)))
        batch = self.build(plan, range(bucket), pad_decode_to=bucket)
        entry = self.graphs.get(bucket)
        if entry is None:
            entry = self.graphs[bucket] = _CapturedStep(self.model, self.state, batch)
        return entry.run(batch)[:len(plan)]


class _CapturedStep:
    """A step of ``n`` decoding sequences in a CUDA graph.  The warm-up runs on padded sequences only, so that nothing of
    the caches or states changes before the first real replay."""

    FIELDS = ("ids", "prev", "positions", "slot_mapping", "logit_rows")

    def __init__(self, model, state, like):
        self.static = StepBatch(**{f: getattr(like, f).clone() for f in self.FIELDS})
        g = like.decode
        self.static.decode = RowGroup(g.rows, g.n_seqs, 1, g.total_rows, g.cu_rows.clone(), torch.full_like(g.start_pos, -1),
                                      torch.full_like(g.slots, -1), torch.zeros_like(g.block_tables))
        self.static.positions.fill_(-1)
        self.static.slot_mapping.fill_(-1)
        side = torch.cuda.Stream(device=model.device)
        side.wait_stream(torch.cuda.current_stream(model.device))
        with torch.cuda.stream(side):
            for _ in range(2):
                model.forward(self.static, state)
        torch.cuda.current_stream(model.device).wait_stream(side)
        torch.cuda.synchronize(model.device)
        self.graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(self.graph):
            self.logits = model.forward(self.static, state)

    def run(self, batch):
        s = self.static
        for f in self.FIELDS:
            getattr(s, f).copy_(getattr(batch, f))
        for f in ("start_pos", "slots", "block_tables"):
            getattr(s.decode, f).copy_(getattr(batch.decode, f))
        self.graph.replay()
        return self.logits


# ---- sampling --------------------------------------------------------------------------------------------------------
def sample(logits, sequences):
    """One token per row of fp32 logits, by each sequence's parameters."""
    out = logits.argmax(-1)
    rest = [i for i, s in enumerate(sequences) if s.params.temperature > 0]
    for i in rest:
        p, seq = sequences[i].params, sequences[i]
        row = logits[i].float() / p.temperature
        if p.top_k > 0 and p.top_k < row.numel():
            row = row.masked_fill(row < row.topk(p.top_k).values[-1], float("-inf"))
        prob = torch.softmax(row, -1)
        if p.top_p < 1.0:
            sorted_p, order = prob.sort(descending=True)
            drop = sorted_p.cumsum(-1) - sorted_p >= p.top_p          # keeps the token that crosses the threshold
            prob = prob.scatter(0, order, sorted_p.masked_fill(drop, 0.0))
        if p.seed is not None and seq.generator is None:
            seq.generator = torch.Generator(device=logits.device).manual_seed(p.seed)
        out[i] = torch.multinomial(prob, 1, generator=seq.generator)[0]
    return out.tolist()


# ---- the engine --------------------------------------------------------------------------------------------------------
class Engine:
    """``max_tokens``: tokens whose keys live sequences hold at most (sizes the K/V cache); ``max_model_len``: the longest
    sequence (None = max_tokens; more than that where the model only looks back a window)."""

    def __init__(self, model, *, max_tokens=32768, max_seqs=64, block_size=256, max_model_len=None, max_step_tokens=8192, graphs=True):
        reach, limit = getattr(model, "cache_reach", None), getattr(model, "max_positions", None)
        max_model_len = max_model_len or max_tokens
        if reach is None:
            max_model_len = min(max_model_len, max_tokens)
        if limit is not None:
            max_model_len = min(max_model_len, limit)
        per_seq = -(-max_model_len // block_size)
        self.max_len = per_seq * block_size if limit is None else min(per_seq * block_size, limit)
        num_blocks = -(-max_tokens // block_size) + max_seqs          # every live sequence may leave a page unfilled
        self.model = model
        self.cache = CacheManager(num_blocks, block_size, max_seqs, per_seq, reach, max_step_tokens)
        state = model.new_state(max_seqs, num_blocks, block_size, per_seq * block_size)
        self.runner = ModelRunner(model, self.cache, state, graphs)
        self.scheduler = Scheduler(self.cache, max_step_tokens, model.chunked_prefill, model.mixed_batches)
        self.fed = {}
        self._names = 0

    def _check_ids(self, tokens):
        if any(not 0 <= int(t) < self.model.vocab for t in tokens):
            raise ValueError(f"token ids must lie in 0..{self.model.vocab - 1}")

    # -- generation ----------------------------------------------------------------------------------------------------
    def add_request(self, tokens, params=None):
        tokens = [int(t) for t in tokens]
        if not tokens:
            raise ValueError("an empty prompt")
        self._check_ids(tokens)
        params = params or SamplingParams()
        if params.max_new_tokens < 1:
            raise ValueError("max_new_tokens must be at least 1")
        self._names += 1
        seq = Sequence(self._names, tokens, params, len(tokens))
        if len(tokens) + params.max_new_tokens > self.max_len:
            raise ValueError(f"prompt and new tokens exceed the longest sequence served ({self.max_len})")
        self.scheduler.add(seq)
        return seq

    def has_work(self):
        return bool(self.scheduler.waiting or self.scheduler.running)

    def step(self):
        """One scheduling decision, one model step, one token for every sequence whose tokens are all in the cache.
        Returns the sequences that finished."""
        plan = self.scheduler.schedule()
        rows, sampled, at = [], [], 0
        for s, n in plan:
            at += n
            if s.done + n == len(s.tokens):
                rows.append(at - 1)
                sampled.append(s)
        logits = self.runner.step(plan, rows)
        finished = []
        if sampled:
            for s, tok in zip(sampled, sample(logits, sampled)):
                s.tokens.append(tok)
                if len(s.output) >= s.params.max_new_tokens or tok in s.params.stop_ids:
                    self.scheduler.finish(s)
                    finished.append(s)
        return finished

    def generate(self, prompts, params=None):
        """The new tokens of every prompt."""
        seqs = [self.add_request(p, params) for p in prompts]
        while self.has_work():
            self.step()
        return [s.output for s in seqs]

    # -- given tokens --------------------------------------------------------------------------------------------------
    def feed(self, entries):
        """Advances sequences by given tokens: entries [(name, tokens, want)], ``want`` the places among these tokens
        whose logits are returned, (wanted, vocab) fp32 in the order of the entries (None if nothing is wanted)."""
        plan, wanted = [], []
        for name, tokens, want in entries:
            self._check_ids(tokens)
            seq = self.fed.get(name)
            if (len(seq.tokens) if seq else 0) + len(tokens) > self.max_len:
                raise ValueError(f"sequence {name!r} exceeds the longest one served ({self.max_len})")
            if seq is None:
                seq = Sequence(name, [])
                if not self.cache.admit(seq):
                    raise OutOfCache("no free state slot")
                self.fed[name] = seq
            seq.tokens.extend(int(t) for t in tokens)
            if tokens:
                plan.append((seq, len(tokens)))
            wanted.append((seq, list(want)))
        order = sorted(plan, key=lambda e: e[1] != 1)                 # decoding sequences first, otherwise as given
        first, at = {}, 0
        for s, n in order:
            first[id(s)] = at
            at += n
        rows = [first[id(s)] + w for s, want in wanted for w in want]
        ascending = sorted(set(rows))
        if not self.model.mixed_batches and any(n == 1 for _, n in order) and any(n > 1 for _, n in order):
            raise ValueError("this model does not mix decoding sequences and prompts in one step")
        logits = self.runner.step(order, ascending) if order else None
        if not rows:
            return None
        where = {r: i for i, r in enumerate(ascending)}
        return logits[torch.tensor([where[r] for r in rows], device=logits.device)]

    def release(self, name):
        """Gives back what a fed sequence holds."""
        self.cache.release(self.fed.pop(name))
