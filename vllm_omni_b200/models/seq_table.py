"""Per-sequence index tensors of one flattened batch, for models whose kernels take a mixed batch
(prompt portions beside single decoded tokens) as a whole."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


@dataclass(frozen=True)
class StateTensor:
    """Part of what a sequence carries beside its pages: the shape of one row of a state pool."""
    shape: tuple[int, ...]
    dtype: torch.dtype | None = None           # None: the activations' type


def layer_caches(cfg, num_blocks: int, block_size: int, num_state_rows: int, dtype, device, kv_heads: int | None = None,
                 fill=torch.zeros) -> list[tuple]:
    """Cache entry of every layer of a decoder configuration: (key pages, value pages, *state pools).  A layer may hold
    no pages (zero heads or channels) or keys only.  ``kv_heads`` overrides the heads (tensor parallel ranks)."""
    out = [tuple(fill(num_blocks, block_size, kv_heads or h, d, dtype=dtype, device=device) for d in (dk, dv))
           for h, dk, dv in cfg.kv_layer_shapes()]
    if num_state_rows and hasattr(cfg, "state_shapes"):
        out = [kv + tuple(torch.zeros(num_state_rows, *s.shape, dtype=s.dtype or dtype, device=device) for s in states)
               for kv, states in zip(out, cfg.state_shapes())]
    return out


def round_up4(n: int) -> int:
    return (n + 3) // 4 * 4


@dataclass
class KeyGroup:
    """Sequences whose keys lie back to back in one buffer (``SeqTable.long_groups``)."""
    key_start: torch.Tensor                    # int32 [S of the batch]: where position 0 of a member is, or (< first key)
                                               # would be if a window did not leave its first positions out
    members: torch.Tensor                      # int32 [2 (members + 1)]: (sequence, first key), closed by (-1, keys)
    n_members: int
    keys: int
    items: torch.Tensor                        # int32 [n_items, 2]: (sequence, first row) of every block of rows
    n_items: int
    rows_per_block: int


@dataclass
class Chunks:
    """Short runs of rows for recurrences that take several tokens at a time (``SeqTable.chunks``)."""
    table: torch.Tensor                        # int32 [n, 4]: (sequence, first row in the portion, rows, 0), a portion's in order
    n: int
    seqs: torch.Tensor                         # int32 [n_seqs, 2]: (sequence, its first chunk), longest portions first
    n_seqs: int


@dataclass
class SeqTable:
    """Sequence s owns rows [q_start[s], q_start[s + 1]) of the batch; context[s] of its tokens came before."""
    q_start: torch.Tensor                      # int32 [S + 1]
    context: torch.Tensor                      # int32 [S]
    block_tables: torch.Tensor                 # int32 [S, W]
    row_seq: torch.Tensor                      # int32 [T]
    decode_list: torch.Tensor                  # int32 [n_decode]: sequences with exactly one row
    n_seqs: int
    n_decode: int
    max_context: int                           # upper bound of context over the decode sequences
    state_in: torch.Tensor | None = None       # int32 [S]: state-pool row a sequence reads
    state_out: torch.Tensor | None = None      # int32 [S]: row it writes (another one), < 0 = none
    lens: list[int] = field(default_factory=list)      # host copy of the row counts; empty when every one is 1
    contexts: list[int] = field(default_factory=list)  # host copy of the contexts (with ``lens``)
    _items: dict = field(default_factory=dict)

    @classmethod
    def build(cls, lens, contexts, tables, states, device) -> "SeqTable":
        """``lens`` / ``contexts`` / ``tables`` (page ids) / ``states`` ((in, out) pairs or None) per sequence.
        Everything crosses to the device in one copy."""
        S, W = len(lens), max(1, max(len(t) for t in tables))
        starts, row_seq = [0], []
        for s, n in enumerate(lens):
            starts.append(starts[-1] + n)
            row_seq.extend([s] * n)
        decode = [s for s, n in enumerate(lens) if n == 1]
        flat, cuts = [], []

        def put(vals):
            cuts.append((len(flat), len(vals)))
            flat.extend(vals)
            flat.extend([0] * (-len(flat) % 4))            # every part starts on 16 bytes
        put(starts)
        put(list(contexts))
        put([b for t in tables for b in list(t) + [0] * (W - len(t))])
        put(row_seq)
        put(decode or [0])
        if states is not None:
            put([s[0] for s in states])
            put([s[1] for s in states])
        buf = torch.tensor(flat, dtype=torch.int32).to(device)
        part = [buf[o:o + n] for o, n in cuts]
        return cls(part[0], part[1], part[2].view(S, W), part[3], part[4], S, len(decode),
                   max((contexts[s] for s in decode), default=0), *(part[5:7] if states is not None else (None, None)),
                   lens=list(lens), contexts=list(contexts))

    def short_rows(self, limit: int):
        """Rows of the sequences with at most ``limit`` rows: int32 on the device, their number, upper bound of the
        keys any of them sees."""
        got = self._items.get(("short", limit))
        if got is None:
            if not self.lens:                              # one row each
                got = (self.q_start[:self.n_seqs], self.n_seqs, self.max_context + 1)
            else:
                rows, keys, at = [], 0, 0
                for n, c in zip(self.lens, self.contexts):
                    if n <= limit:
                        rows.extend(range(at, at + n))
                        keys = max(keys, c + n)
                    at += n
                dev = self.q_start.device
                got = (torch.tensor(rows or [0], dtype=torch.int32).to(dev), len(rows), keys)
            self._items[("short", limit)] = got
        return got

    def _first_key(self, s: int, window: int | None) -> int:
        """First position that a row of sequence s sees, rounded down to the 32 keys a kernel reads at a time."""
        return 0 if window is None else max(0, self.contexts[s] - window + 1) // 32 * 32

    def long_groups(self, limit: int, max_keys: int, rows_per_block: int, window: int | None = None):
        """The sequences with more than ``limit`` rows in groups whose keys (context and new tokens, with a ``window`` only
        those some row sees) fit ``max_keys`` together, at least one sequence each: ``KeyGroup`` list, for kernels that want
        a group's keys back to back."""
        key = ("long", limit, max_keys, rows_per_block, window)
        got = self._items.get(key)
        if got is None:
            got, cur, keys = [], [], 0
            for s, n in enumerate(self.lens):
                if n <= limit:
                    continue
                k = n + self.contexts[s] - self._first_key(s, window)
                if cur and keys + k > max_keys:
                    got.append(self._key_group(cur, rows_per_block, window))
                    cur, keys = [], 0
                cur.append(s)
                keys += k
            if cur:
                got.append(self._key_group(cur, rows_per_block, window))
            self._items[key] = got
        return got

    def _key_group(self, seqs, rows_per_block, window):
        start, firsts, at = [0] * self.n_seqs, [], 0
        for s in seqs:
            lo = self._first_key(s, window)
            start[s] = at - lo
            firsts += [s, at]
            at += self.lens[s] + self.contexts[s] - lo
        items = sorted(((s, o) for s in seqs for o in range(0, self.lens[s], rows_per_block)),
                       key=lambda it: -(self.contexts[it[0]] + it[1]))     # most keys first
        members = firsts + [-1, at]                                        # (sequence, first key) pairs, then the end
        flat = start + [0] * (-len(start) % 4) + members + [0] * (-len(members) % 4) + [v for it in items for v in it]
        buf = torch.tensor(flat, dtype=torch.int32).to(self.q_start.device)
        o1 = round_up4(len(start))
        o2 = o1 + round_up4(len(members))
        return KeyGroup(buf[:len(start)], buf[o1:o1 + len(members)], len(seqs), at, buf[o2:o2 + 2 * len(items)].view(-1, 2), len(items),
                        rows_per_block)

    def time_runs(self, key, pick):
        """Runs of consecutive rows of the sequences with more than one row, for scans over time: ``pick(lens)`` gives the
        run length for portions of ``lens`` rows (asked once per ``key``).  int32 [m, 4] of (sequence, first row in the
        portion, rows, index of the sequence's first run), m, and whether any sequence has several runs."""
        got = self._items.get(("time", key))
        if got is None:
            runs, several = [], False
            step = pick([n for n in self.lens if n > 1])
            for s, n in enumerate(self.lens):
                if n > 1:
                    first = len(runs)
                    runs += [(s, o, min(step, n - o), first) for o in range(0, n, step)]
                    several |= len(runs) - first > 1
            got = (torch.tensor(runs, dtype=torch.int32).to(self.q_start.device), len(runs), several)
            self._items[("time", key)] = got
        return got

    def chunks(self, size: int) -> Chunks:
        """The portions of more than one row, cut into chunks of ``size`` rows."""
        got = self._items.get(("chunks", size))
        if got is None:
            rows, long = [], []
            for s, n in enumerate(self.lens):
                if n > 1:
                    long.append((s, len(rows) // 4))
                    for o in range(0, n, size):
                        rows += (s, o, min(size, n - o), 0)
            long.sort(key=lambda it: -self.lens[it[0]])
            buf = torch.tensor(rows + [v for it in long for v in it], dtype=torch.int32).to(self.q_start.device)
            got = Chunks(buf[:len(rows)].view(-1, 4), len(rows) // 4, buf[len(rows):].view(-1, 2), len(long))
            self._items[("chunks", size)] = got
        return got

    def prefill_items(self, rows_per_block: int):
        """(sequence, first row within it) pairs of every block of ``rows_per_block`` rows of the sequences with
        more than one row, longest context last in, first out: int32 [n, 2] on the device, n."""
        got = self._items.get(rows_per_block)
        if got is None:
            pairs = [(s, o) for s, n in enumerate(self.lens) if n > 1 for o in range(0, n, rows_per_block)]
            pairs.reverse()                    # the blocks with the most keys behind them start first
            got = (torch.tensor(pairs, dtype=torch.int32).to(self.q_start.device), len(pairs))
            self._items[rows_per_block] = got
        return got
