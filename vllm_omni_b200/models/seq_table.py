"""Per-sequence index tensors of one flattened batch, for models whose kernels take a mixed batch
(prompt portions beside single decoded tokens) as a whole."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


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
                   lens=list(lens))

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
