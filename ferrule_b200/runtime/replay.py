"""Replay of given token streams through the engine's own transactions.

`ReplayEngine.replay` runs one step: the next tokens of any number of requests as one batch (portions of prompts beside
single decoded tokens), lowered, reserved, executed and committed exactly as a scheduled batch is - page manager,
state slots, runner - except that the tokens come from the caller and nothing is sampled.  It returns the logits of the
rows the caller asked for.  A request is admitted at its first entry and holds its pages and slot until it is ended.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Sequence

import numpy as np

from .engine import Engine, Transaction
from .execution import ExecutionBatch, LogitsRequest
from .session import FinishReason, GenerateRequest, SeqStatus, SequenceState


@dataclass
class ReplayEntry:
    request_id: str
    tokens: List[int]
    want: List[int] = field(default_factory=list)        # indices into `tokens` whose logits are returned


class ReplayError(RuntimeError):
    pass


class ReplayEngine(Engine):
    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self._live: Dict[str, SequenceState] = {}
        self._wanted: Dict[str, List[int]] = {}
        self._rows: Dict[str, Dict[int, np.ndarray]] = {}
        if not self.runner.capabilities().supports_full_logits:
            raise ReplayError("this model's runner does not return whole logit rows")

    # ------------------------------------------------------------------ public
    def replay(self, entries: Sequence[ReplayEntry], end: Sequence[str] = ()) -> List[np.ndarray]:
        """One step.  -> a [len(want), vocab] fp32 array per entry, in order; `end` names the requests that are
        finished after it."""
        prefills, decodes = [], []
        seen = set()
        for e in entries:
            if not e.tokens or e.request_id in seen:
                raise ReplayError(f"request {e.request_id!r}: an entry needs tokens, and one entry per step")
            if any(not 0 <= w < len(e.tokens) for w in e.want):
                raise ReplayError(f"request {e.request_id!r}: wanted rows lie outside the entry's tokens")
            seen.add(e.request_id)
            seq = self._live.get(e.request_id) or self._admit(e.request_id, e.tokens)
            for q in (self.scheduler.prefill, self.scheduler.decode_ready):
                if seq in q:
                    q.remove(seq)
            seq.status = SeqStatus.RUNNING
            if len(e.tokens) == 1 and seq.position > 0:
                seq.staged_token = e.tokens[0]
                decodes.append(seq)
            else:
                seq.tokens = seq.tokens[:seq.position] + list(e.tokens)
                seq.prompt_len = len(seq.tokens)
                prefills.append((seq, len(e.tokens)))
            self._wanted[e.request_id] = list(e.want)
        self._rows.clear()
        if entries:
            stalls, self.last_error = self.stats.kv_stalls, None
            self._execute_ordinary(prefills, decodes)
            if self.last_error is not None:
                raise ReplayError(f"the step failed: {self.last_error}") from self.last_error
            if self.stats.kv_stalls != stalls:
                raise ReplayError("the page pool cannot hold the live requests")
        out = []
        for e in entries:
            rows = self._rows.get(e.request_id, {})
            out.append(np.stack([rows[w] for w in e.want]) if e.want else np.zeros((0, self.runner.vocab_size), np.float32))
        for rid in end:
            seq = self._live.pop(rid, None)
            if seq is not None:
                self._finish(seq, FinishReason.MAX_TOKENS)
        self._outbox.clear()
        self._drive_retirements()
        return out

    # ------------------------------------------------------------------ engine hooks
    def _admit(self, request_id: str, tokens: List[int]) -> SequenceState:
        seq = self.submit(GenerateRequest(request_id, list(tokens), max_new_tokens=1 << 30, ignore_eos=True))
        self.scheduler._admit()
        if seq.slot < 0:
            raise ReplayError(f"request {request_id!r}: every sequence slot is taken")
        self._live[request_id] = seq
        return seq

    def _lower(self, txn: Transaction) -> ExecutionBatch:
        batch = super()._lower(txn)
        batch.logits = [LogitsRequest.none()] * batch.rows
        for m in txn.members:
            for w in self._wanted[m.seq.request_id]:
                batch.logits[m.query_start + w] = LogitsRequest.full()
        return batch

    def _publish(self, txn: Transaction) -> None:
        start = {m.seq.request_id: m.query_start for m in txn.members}
        out = txn.output.by_row()
        super()._publish(txn)
        for rid, r0 in start.items():
            self._rows[rid] = {w: np.asarray(out[r0 + w].full_logits, dtype=np.float32) for w in self._wanted[rid]}

    def _apply_output(self, seq: SequenceState, top1) -> None:
        """Nothing is sampled: the next token comes with the next entry."""
