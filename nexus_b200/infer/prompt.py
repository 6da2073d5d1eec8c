"""How the long segments of a step reach the tcgen05 prompt kernels: blocks of query rows, and the keys that earlier steps left in
the cache pages gathered beside those of the step.  Built on the host once per step, one table per window."""
from __future__ import annotations

from typing import NamedTuple

import torch

QUERY_BLOCK = 256    # query rows of one work item


class Window(NamedTuple):
    """What a layer's rows see: the last ``size`` keys (0: all of them), with ``chunk`` > 0 only those of the row's own chunk of
    positions, and the first ``keep_first`` ones."""
    size: int
    keep_first: int = 0
    chunk: int = 0


def _cuts(pos: int, count: int, chunk: int):
    """(offset, rows) of the query blocks; chunks that fill a block end one."""
    at = 0
    while at < count:
        rows = min(QUERY_BLOCK, count - at)
        if chunk >= QUERY_BLOCK:
            rows = min(rows, chunk - (pos + at) % chunk)
        yield at, rows
        at += rows


def long_segments(segs, window: int, keep_first: int = 0, chunk: int = 0):
    """The work for segments (first row, rows, first position, sequence): (blocks, runs, rows of kv).

    A segment that does not start at position 0 needs keys of earlier steps: if there is one, all keys are gathered from the
    cache (``runs``: first row, rows, first position, sequence), else they are the rows of the step and ``runs`` is empty.
    ``blocks``: first query row, rows, position of the first row, kv row of position 0 and, last, the row that position 0 has
    among the kept first keys; the most keys first."""
    back, blocks, runs, d = window - 1 if window > 0 else 1 << 30, [], [], 0

    def first_key(p):
        return max(0, p - back, p // chunk * chunk if chunk > 0 else 0)
    gather = any(pos > 0 for _, _, pos, _ in segs)
    for row0, count, pos, seq in segs:
        kv0 = kept0 = row0
        if gather:
            base = first_key(pos)
            kept, kept0 = min(keep_first, base), d
            if kept:                          # in front of the keys from `base` on
                runs.append((d, kept, 0, seq))
                d += kept
            kv0 = d - base
            if not kept:
                kept0 = kv0
            runs.append((d, pos + count - base, base, seq))
            d += pos + count - base
        for b, rows in _cuts(pos, count, chunk):
            blocks.append((pos + b - first_key(pos + b) + rows, row0 + b, rows, pos + b, kv0, kept0))
    blocks.sort(key=lambda x: -x[0])
    return [b[1:] for b in blocks], runs, d


def row_slices(blocks, most: int):
    """Blocks (first row, rows, ..; the most keys first) in groups of up to ``most`` consecutive rows, each in the order given: (blocks, first row,
    rows of the group).  A block is never cut."""
    out, group, first, end = [], [], 0, 0
    for i in sorted(range(len(blocks)), key=lambda i: blocks[i][0]):
        row, rows = blocks[i][:2]
        if group and row + rows - first > most:
            out.append((group, first, end - first))
            group = []
        if not group:
            first = row
        group.append(i)
        end = row + rows
    if group:
        out.append((group, first, end - first))
    return [([blocks[i] for i in sorted(g)], row, rows) for g, row, rows in out]


class StepPlan:
    """How the segments of a step that has long ones are split; ``rows``: the rows of the one-token and short segments,
    ``groups`` these segments over the compacted rows; per window the blocks and runs of the long ones (`long_segments`).  ``sliced``:
    windows whose blocks are wanted in groups of consecutive rows too, and the most rows of a group (`row_slices`)."""

    def __init__(self, engine, windows, sliced):
        from ..ops import _mixers as M
        single, short, long_ = engine._groups
        host, n = engine._host_rows[engine.INDEX_ROWS:], single.count + short.count
        segs = [tuple(int(v) for v in host[:, j]) for j in range(n + long_.count)]
        data, at = [], {}

        def put(name, values):
            at[name] = (len(data), len(values))
            data.extend(values)
            data.extend([0] * (-len(data) % 4))        # tables start on 16 bytes
        first, table = 0, [[], [], [], []]
        for row0, count, pos, seq in segs[:n]:
            for t, v in zip(table, (first, count, pos, seq)):
                t.append(v)
            first += count
        put("rows", [r for row0, count, _, _ in segs[:n] for r in range(row0, row0 + count)])
        put("table", [v for t in table for v in t])
        self.kv_rows, self.longest, self.slices = {}, {}, {}
        for w in windows:
            blocks, runs, self.kv_rows[w] = long_segments(segs[n:], *w)
            self.longest[w] = max((r[1] for r in runs), default=0)
            put(("blocks", w), [v for b in blocks for v in b[:4]])
            put(("kept", w), [b[4] for b in blocks])
            put(("runs", w), [v for r in runs for v in r])
            groups = row_slices(blocks, sliced[w]) if w in sliced else []
            self.slices[w] = [(("slice", w, i), row, rows) for i, (_, row, rows) in enumerate(groups)]
            for i, (part, _, _) in enumerate(groups):
                put(("slice", w, i), [v for b in part for v in b[:4]])
        self.gathered = any(self.kv_rows.values())
        dev = torch.tensor(data, dtype=torch.int32).pin_memory().to(engine.dev, non_blocking=True)

        def get(name):
            return dev[at[name][0]: at[name][0] + at[name][1]]
        self.blocks = {w: get(("blocks", w)).view(-1, 4) for w in windows}
        self.kept = {w: get(("kept", w)) for w in windows}
        self.runs = {w: get(("runs", w)).view(-1, 4) for w in windows}
        self.slices = {w: [(get(name).view(-1, 4), row, rows) for name, row, rows in s] for w, s in self.slices.items()}
        self.rows = get("rows").long() if n else None
        if n:
            t = get("table").view(4, n)
            self.groups = [M.Segments(t, 0, single.count, single.max_len, single.total),
                           M.Segments(t, single.count, short.count, short.max_len, short.total)]


def plan(engine, windows, sliced=None) -> None:
    """Called once per step, before the layers; ``windows``: those of the layers that a prompt kernel can take."""
    engine._prompt_plan = None
    if engine.fast and engine._groups[2].count > 0 and windows:
        engine._prompt_plan = StepPlan(engine, sorted(windows), sliced or {})
