"""Ragged batches: one model step over several requests, each bringing any number of new tokens.

A continuous-batching step is a flat list of tokens: a portion of one request's prompt beside single decoded tokens of
others.  ``RaggedEntry`` names one request's share, ``RaggedPlan`` is what the kernels need, built on the host from the
requests' page lists and moved to the device as ONE pinned block:

    ids [T] | tok_pos [T] | tok_seq [T] | want_rows [W] | block_table [S, max_pages] | tiles [n, 3] per tile size | seq_info [S, 4] | seq_prev [S]

``tok_pos`` is the position of a token in its sequence, ``tok_seq`` its row in this step's block table, ``tiles`` the
attention kernels' work lists (runs of at most ``tile`` consecutive tokens of one sequence; one list per tile size
the model's layers ask for, ``tiles_for(size)``), ``seq_info`` one row per sequence for kernels that walk a sequence's new
tokens in order (first flat token, token count, position of the first token, the request's recurrent-state slot or -1),
``seq_prev`` the token that every sequence ended its last step with (-1: none, or its cache keeps no token history).
Building the plan also
does the step's cache bookkeeping: every request's page list grows by its new tokens (pages come from the pool's free
list first), before anything is launched.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Sequence

import numpy as np
import torch


@dataclass
class RaggedEntry:
    tokens: Sequence[int]
    cache: list                       # the request's per-layer caches (model.create_kv_cache())
    want: Sequence[int] | None = None  # places among `tokens` whose logits are wanted; None = the last one


class RaggedPlan:
    @staticmethod
    def block_ints(tokens: int, wanted: int, seqs: int, max_pages: int, tiles: int) -> int:
        """Number of int32 in a plan's device block (``tiles`` summed over the tile sizes)."""
        return 3 * tokens + wanted + seqs * max_pages + 3 * tiles + 5 * seqs

    def __init__(self, entries: Sequence[RaggedEntry], device, tile, max_pages: int | None = None, into: torch.Tensor | None = None):
        """``max_pages`` fixes the block table's width (at least what the longest request needs) and ``into`` names a
        preallocated int32 device block to upload into: a captured graph reads the same addresses every step."""
        sizes = sorted({int(tile)} if isinstance(tile, int) else {int(t) for t in tile})
        owners = [getattr(e.cache[0], "owner", e.cache[0]) for e in entries]
        counts = [len(e.tokens) for e in entries]
        if min(counts) == 0:
            raise ValueError("a ragged entry needs at least one token")
        if len({id(o) for o in owners}) < len(owners):
            raise ValueError("a request may appear once per step")
        wants = [[n - 1] if e.want is None else list(e.want) for e, n in zip(entries, counts)]
        for n, places in zip(counts, wants):  # checked before anything is appended
            for place in places:
                if not 0 <= place < n:
                    raise ValueError(f"wanted place {place} is outside the entry's {n} tokens")
        tokens = [np.asarray(e.tokens, dtype=np.int64) for e in entries]
        starts = [o.offset for o in owners]
        done = []
        try:
            for o, n in zip(owners, counts):
                o.append_slots(n)
                done.append((o, n))
        except Exception:
            for o, n in done:  # all-or-nothing: give the pages of this step back
                o.rewind(n)
            raise
        T, S = sum(counts), len(entries)
        needed = max(o.num_pages for o in owners)
        if max_pages is not None and max_pages < needed:
            for o, n in done:
                o.rewind(n)
            raise ValueError(f"block table of {max_pages} pages, {needed} needed")
        max_pages = needed if max_pages is None else max_pages
        W = sum(len(w) for w in wants)
        n_tiles = {size: sum(-(-n // size) for n in counts) for size in sizes}
        total = self.block_ints(T, W, S, max_pages, sum(n_tiles.values()))
        host = torch.empty(max(total, 1), dtype=torch.int32, pin_memory=torch.cuda.is_available() and torch.device(device).type == "cuda")
        buf = host.numpy()
        ids, pos, seq = buf[0:T], buf[T : 2 * T], buf[2 * T : 3 * T]
        want = buf[3 * T : 3 * T + W]
        table = buf[3 * T + W : 3 * T + W + S * max_pages].reshape(S, max_pages)
        table[:] = -1
        tile_at, at = {}, 3 * T + W + S * max_pages
        for size in sizes:
            tile_at[size] = (at, n_tiles[size])
            at += 3 * n_tiles[size]
        info = buf[at : at + 4 * S].reshape(S, 4)
        prev = buf[at + 4 * S : at + 5 * S]
        work = [(size, buf[start : start + 3 * n].reshape(n, 3)) for size, (start, n) in tile_at.items()]
        row_of = np.arange(S)
        firsts = np.cumsum([0] + counts[:-1])
        ids[:] = np.concatenate(tokens) if S > 1 else tokens[0]
        seq[:] = np.repeat(row_of, counts) if T > S else row_of
        info[:, 0], info[:, 1], info[:, 2] = firsts, counts, starts
        info[:, 3] = [getattr(o, "state_slot", -1) for o in owners]
        histories = [getattr(o, "tokens", None) for o in owners]
        prev[:] = [h[start - 1] if h is not None and 0 < start <= len(h) else -1 for h, start in zip(histories, starts)]
        for s, o in enumerate(owners):
            table[s, : o.num_pages] = o.page_ids
        if T == S:  # one token per sequence
            pos[:] = starts
            want[:] = [s for s, places in enumerate(wants) for _ in places]
            for _, rows in work:
                rows[:, 0], rows[:, 1], rows[:, 2] = row_of, 1, row_of
        else:
            at_row, w = {size: 0 for size in sizes}, 0
            for s, (t, n, start) in enumerate(zip(firsts.tolist(), counts, starts)):
                pos[t : t + n] = np.arange(start, start + n)
                if wants[s]:
                    want[w : w + len(wants[s])] = np.asarray(wants[s]) + t
                    w += len(wants[s])
                for size, rows in work:
                    offsets = np.arange(0, n, size)
                    part = rows[at_row[size] : at_row[size] + len(offsets)]
                    part[:, 0], part[:, 1], part[:, 2] = t + offsets, np.minimum(size, n - offsets), s
                    at_row[size] += len(offsets)
        self.num_tokens, self.num_seqs, self.num_want, self.max_pages = T, S, W, max_pages
        self.h2d_bytes = total * 4
        if into is None:
            dev = host.to(device, non_blocking=True)
        else:
            if into.numel() != total or into.dtype != torch.int32:
                raise ValueError("the device block does not fit this plan")
            dev = into
            dev.copy_(host[:total], non_blocking=True)
        self.total_ints = total
        self._host = host  # keep the pinned block alive until the copy has run
        self.ids, self.tok_pos, self.tok_seq = dev[0:T], dev[T : 2 * T], dev[2 * T : 3 * T]
        self.want_rows = dev[3 * T : 3 * T + W]
        self.block_table = dev[3 * T + W : 3 * T + W + S * max_pages].view(S, max_pages)
        self._tiles = {size: dev[start : start + 3 * n].view(n, 3) for size, (start, n) in tile_at.items()}
        self.seq_info = dev[at : at + 4 * S].view(S, 4)
        self.seq_prev = dev[at + 4 * S : at + 5 * S]
        self.tiles = self._tiles[sizes[0]]
        self.max_context = max(o.offset for o in owners)  # the longest sequence after this step's append
        self.want_counts = [len(x) for x in wants]
        self.all_wanted = W == T and all(x == list(range(len(x))) for x in wants)  # the wanted rows are the step's rows, in order
        self.starts = starts
        self.max_tokens = max(counts)  # the longest entry of the step
        self.owners = owners
        for o, ran in zip(owners, tokens):  # from here on the step runs: what it consumes cannot be taken back from a recurrent state
            if hasattr(o, "record_tokens"):
                o.record_tokens(ran)
            if hasattr(o, "ran_offset"):
                o.ran_offset = o.offset

    def rope_tables(self, dims: int, base: float, factor: float = 1.0, ramp: tuple | None = None):
        """(cos, sin) fp32 ``[T, dims // 2]`` of this step's token positions, made once per step and rotation."""
        from extensions_b200.tiny_llm_ext_b200 import blocks

        key = (int(dims), float(base), float(factor), ramp)
        tables = self.__dict__.setdefault("_rope_tables", {})
        if key not in tables:
            tables[key] = blocks.rope_table(self.tok_pos, dims=key[0], base=key[1], factor=key[2], ramp=key[3])
        return tables[key]

    def tiles_for(self, size: int) -> torch.Tensor:
        """The work list cut into runs of at most ``size`` tokens (one of the sizes the plan was built for)."""
        return self._tiles[size]
