"""Online use of a runner: the host decides which tokens of which request run next, the device does the rest.

`OnlineSession` drives a runner built with mode="online".  A request is a row of the token table; the session posts it,
appends tokens to it and closes it through the control words the batching task reads (include/mpk_b200.h, request_ctl).
Admission, page allocation, state slots and the composition of every batch are the batching task's, the same code that
schedules offline generation; a step with more tokens than one batch takes runs as several launches.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Hashable, Iterable, List, Sequence, Tuple

import torch

from . import _native as N


@dataclass
class _Request:
    row: int
    length: int      # tokens supplied so far


class OnlineSession:
    def __init__(self, runner):
        if runner.mpk.mode != "online":
            raise ValueError("OnlineSession needs a runner built with mode='online'")
        self.runner, self.mpk, self.meta = runner, runner.mpk, runner.meta
        rows, self.max_length = self.meta["tokens"].shape
        self._ctl = torch.zeros(rows, dtype=torch.int32)          # host copy of the control words
        self._plen = torch.zeros(rows, dtype=torch.int32)
        self._free: List[int] = list(range(rows))
        self._closing: List[int] = []                             # closed, retired by the next launch
        self._live: Dict[Hashable, _Request] = {}
        self.mpk.reset()

    def _launch(self) -> List[Tuple[int, int, int, int]]:
        """One launch; returns (row, first batch index, tokens, position of the first) of every batch slot with tokens."""
        self.mpk.step(1)
        status = self.mpk.status()
        for row in self._closing:
            self._ctl[row] = N.REQ_FREE
            self._free.append(row)
        self._closing.clear()
        ids = self.meta["request_ids"].tolist()
        qo = self.meta["qo_indptr_buffer"].tolist()
        step = self.meta["step"].tolist()          # of the batch that just ran; advanced by the next launch
        out = [(row, qo[k], qo[k + 1] - qo[k], step[row]) for k, row in enumerate(ids) if row >= 0 and qo[k + 1] > qo[k]]
        assert sum(n for _, _, n, _ in out) == status.active_tokens
        return out

    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]],
             end: Iterable[Hashable] = ()) -> List[torch.Tensor]:
        """Runs the next tokens of each request: entries of (id, tokens, want), `want` indexing into `tokens`.  Returns
        per entry the float32 logits [len(want), vocabulary] (host memory).  Requests in `end` give back pages and slot."""
        todo: Dict[int, Tuple[int, int]] = {}                      # row -> (entry, length before this step)
        ids = [rid for rid, tokens, _ in entries if len(tokens)]
        if len(set(ids)) != len(ids):
            raise ValueError("a request appears twice in one step")
        for rid, tokens, _ in entries:                             # nothing is changed when a step is refused
            have = self._live[rid].length if rid in self._live else 0
            if have + len(tokens) >= self.max_length:
                raise ValueError(f"request {rid!r} outgrows the token table ({self.max_length} positions)")
        if sum(rid not in self._live for rid in ids) > len(self._free):
            raise RuntimeError("no free row in the token table: too many live requests")
        for e, (rid, tokens, _) in enumerate(entries):
            if not len(tokens):
                continue
            req = self._live.get(rid)
            if req is None:
                req = self._live[rid] = _Request(self._free.pop(0), 0)
            todo[req.row] = (e, req.length)
            self.meta["tokens"][req.row, req.length:req.length + len(tokens)] = torch.tensor(
                list(tokens), dtype=torch.int64, device=self.meta["tokens"].device)
            req.length += len(tokens)
            self._plen[req.row] = req.length
            self._ctl[req.row] = N.REQ_HOLD
        rows: List[Dict[int, torch.Tensor]] = [{} for _ in entries]   # per entry: place -> logits
        if todo:
            self.meta["prompt_lengths"].copy_(self._plen)
            self.meta["request_ctl"][0].copy_(self._ctl)
        pending = sum(len(tokens) for _, tokens, _ in entries)
        while pending > 0:
            ran = self._launch()
            if not ran:
                raise RuntimeError("the batch is empty although tokens are waiting: out of pages or state slots")
            picks = []                                             # (entry, place, batch index)
            for row, b0, n, pos in ran:
                pending -= n
                e, before = todo[row]
                first = pos - before
                picks += [(e, w, b0 + w - first) for w in set(entries[e][2]) if first <= w < first + n]
            if picks:
                idx = torch.tensor([b for _, _, b in picks], device=self.runner.logits.device)
                got = self.runner.logits.index_select(0, idx).float().cpu()
                for (e, w, _), row_logits in zip(picks, got):
                    rows[e][w] = row_logits
        for rid in end:
            req = self._live.pop(rid)
            self._ctl[req.row] = N.REQ_CLOSE
            self._closing.append(req.row)
            self.meta["request_ctl"][0].copy_(self._ctl)
        vocab = self.runner.logits.shape[1]
        return [torch.stack([rows[e][w] for w in want]) if len(want) else torch.empty(0, vocab)
                for e, (_, _, want) in enumerate(entries)]
