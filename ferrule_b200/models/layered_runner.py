"""Engine runner for layer-list models: the paged runner's transactions, graphs and look-ahead over a model that also
carries recurrent state.

Latent rows, or keys and values, live in the engine's pages; recurrent state and convolution inputs live in the sequence's slot
(`RecurrentStatePool`).  A transaction reads the committed buffer of a slot and writes the next one; publishing makes it
current, rolling back needs nothing.  State cannot be cut at an earlier position, so speculation (rows that may be
rejected) and shared prefixes (forks, prompt-prefix cache) are refused; a retained session keeps its slot, a swapped-out
sequence keeps its slot and copies its pages.
"""
from __future__ import annotations

from typing import Dict, List

import numpy as np
import torch

from ..runtime.arena import SequenceStateCore
from ..runtime.execution import (ExecutionBatch, ExecutionCapabilities, ExecutionOutput, KvLayoutSchema,
                                 KvPlaneDescriptor, LogitsKind, RowOutput)
from ..runtime.runner import EndIntent, EndStatus
from .deepseek import KvPool
from .layered import LayeredCuda, LayeredReference
from .layered_weights import LayeredWeights
from .runner import BatchStaging, DeepSeekRunner
from .state_pool import RecurrentStatePool


class LayeredRunner(DeepSeekRunner):
    supports_prefix_sharing = False

    def __init__(self, weights: LayeredWeights, n_pages: int, page_size: int = 64, max_rows: int = 2048, max_seqs: int = 64,
                 max_seq_len: int = 4096, device=None, use_graphs: bool = True, attn_splits: int = 8, lookahead: bool = True,
                 full_logit_rows: int = 0):
        self.states = RecurrentStatePool(weights.cfg, max_seqs, weights.embed.device, weights.embed.dtype,
                                         buffers=3 if lookahead else 2, max_tokens=max_seq_len)
        self.full_logit_rows = full_logit_rows          # logit rows per head pass of batches that ask for whole rows
        self.seq_state: Dict[int, SequenceStateCore] = {}
        self._binds: Dict[int, List[tuple]] = {}
        super().__init__(weights, n_pages, page_size, max_rows=max_rows, max_seqs=max_seqs, max_seq_len=max_seq_len,
                         device=device, use_graphs=use_graphs, attn_splits=attn_splits, enable_mtp=False,
                         lookahead=lookahead)

    # ------------------------------------------------------------------ parts
    def _make_pool(self, n_pages: int) -> KvPool:
        return KvPool(self.cfg, n_pages, self.page_size, self.device, dtype=self.w.embed.dtype,
                      row_dims=[self.cfg.plane_dim(self.cfg.runs[r]) for r in self.cfg.cache_runs])

    def _prefill_tc_heads(self) -> tuple:
        """Rows per position of the tile tables: one for all grouped-query layers (as many positions as the widest group of
        query heads leaves room for), one for every head count of the latent layers."""
        from ..ops.layered import gqa_tc_group, latent_tc_group
        mixer = lambda i: self.cfg.layers[i].mixer
        grouped = [gqa_tc_group(mixer(i), self.w.embed.dtype, self.page_size)
                   for i in self.cfg.attention_layers + self.cfg.window_layers]
        latent = {latent_tc_group(mixer(i), self.w.embed.dtype, self.page_size) for i in self.cfg.latent_layers}
        return tuple(sorted({max(grouped, default=0), *latent} - {0}))

    def _make_staging(self, rows: int, seqs: int, prefill: bool = False) -> BatchStaging:
        return BatchStaging(rows, seqs, self.max_blocks, self.device,
                            tc_heads=self._prefill_tc_heads() if (prefill and self.is_cuda) else 0, state_slots=True)

    def _make_forward(self, logit_rows: int, attn_splits: int, emulate_bf16: bool):
        if not self.is_cuda:
            return LayeredReference(self.w, self.pool, self.states)
        return LayeredCuda(self.w, self.pool, self.states, max_rows=self.max_rows,
                           max_logit_rows=max(logit_rows, self.full_logit_rows), decode_rows=self.max_seqs,
                           max_seq_len=self.max_seq_len, attn_splits=attn_splits)

    def _stage(self, st: BatchStaging, b: ExecutionBatch, ahead: bool = False):
        out = st.fill(b)
        st.fill_states([(*self.states.bind(s.state_slot, s.context_len == 0, ahead), s.query_len) for s in b.sequences])
        return out

    # ------------------------------------------------------------------ contract
    def capabilities(self) -> ExecutionCapabilities:
        return ExecutionCapabilities(max_batch_rows=self.max_rows, max_sequences=self.max_seqs, max_topk=40,
                                     supports_provisional=False, supports_full_logits=True)

    def kv_schema(self) -> KvLayoutSchema:
        layer = lambda i: self.cfg.runs[self.cfg.cache_runs[i]]
        kinds = {}
        for i in range(self.pool.n_layers):
            key = ("latent_kv" if layer(i) in self.cfg.latent_layers else "kv", self.cfg.plane_dim(layer(i)))
            kinds[key] = kinds.get(key, 0) + 1
        planes = tuple(KvPlaneDescriptor(name, width, n) for (name, width), n in sorted(kinds.items(), reverse=True))
        return KvLayoutSchema(planes or (KvPlaneDescriptor("kv", self.cfg.kv_row_dim, 0),), self.page_size, self.max_seq_len)

    def prepare_batch(self, txn_id: int, batch: ExecutionBatch) -> None:
        for s in batch.sequences:
            if s.cow:
                raise RuntimeError("recurrent state is bound by slot: shared (copy-on-write) pages are not supported")
            if s.state_slot >= self.max_seqs or s.sequence_len > min(self.max_seq_len, self.cfg.max_position):
                raise RuntimeError(f"sequence in slot {s.state_slot} exceeds the runner's pools")
        super().prepare_batch(txn_id, batch)

    def execute(self, txn_id: int):
        binds = []
        for s in self.txns[txn_id].sequences:
            core = self.seq_state.get(s.state_slot)
            if s.context_len == 0:
                # a sequence that starts (again) reads zeros, whatever the slot held
                core = self.seq_state[s.state_slot] = SequenceStateCore()
                self.states.release(s.state_slot)
            if core is None or core.position != s.context_len:
                raise RuntimeError(f"slot {s.state_slot}: state holds {core.position if core else 0} tokens, batch expects "
                                   f"{s.context_len}")
            written = self.states.bind(s.state_slot, s.context_len == 0)[1]
            binds.append((s.state_slot, core.begin_step(), s.query_len, written))
        self._binds[txn_id] = binds
        return super().execute(txn_id)

    def end_transaction(self, txn_id: int, intent: EndIntent) -> EndStatus:
        for slot, binding, rows, written in self._binds.pop(txn_id, ()):
            core = self.seq_state.get(slot)
            if core is not None and intent == EndIntent.PUBLISH:
                core.commit_step(binding, rows)
                self.states.commit(slot, written)
        return super().end_transaction(txn_id, intent)

    def release_slot(self, state_slot: int) -> None:
        super().release_slot(state_slot)
        self.seq_state.pop(state_slot, None)
        self.states.release(state_slot)

    # ------------------------------------------------------------------ whole logit rows
    @staticmethod
    def _wants_full(b: ExecutionBatch) -> bool:
        return any(lr.kind == LogitsKind.FULL for lr in b.logits)

    @staticmethod
    def _row_output(r: int, req, logits: torch.Tensor) -> RowOutput:
        from ..ops import reference as ref
        ids, vals = ref.topk_logits(logits[None], max(req.k, 1))
        return RowOutput(r, ids[0].tolist(), vals[0].tolist(), logits.numpy() if req.kind == LogitsKind.FULL else None)

    def _execute_cuda(self, b: ExecutionBatch, start_layer: int = 0, h0=None) -> ExecutionOutput:
        if not self._wants_full(b):
            return super()._execute_cuda(b, start_layer, h0)
        ahead, self._ahead = self._ahead, None
        if ahead is not None:
            ahead[2].synchronize()
        st = self.staging
        T, _, lrows = self._stage(st, b)
        self.stats.h2d_bytes += st.upload()
        rows: List[RowOutput] = []

        def consume(first: int, logits: torch.Tensor) -> None:
            host = logits.cpu()
            self.stats.d2h_bytes += host.numel() * 4
            rows.extend(self._row_output(r, b.logits[r], host[i]) for i, r in enumerate(lrows[first:first + host.shape[0]]))

        db = st.device_batch(T, len(lrows))
        db.decode_only = db.n_seqs == T          # one row per sequence: earlier cache rows predate this step
        self.fwd.forward_rows(db, consume)
        self._last_hidden = None
        torch.cuda.current_stream().synchronize()
        self.stats.kernel_launches += self.fwd.launches
        self.stats.eager_steps += 1
        return ExecutionOutput(rows)

    def _execute_reference(self, b: ExecutionBatch, start_layer: int = 0, h0=None) -> ExecutionOutput:
        st = self.staging
        T, _, lrows = self._stage(st, b)
        db = st.device_batch(T, len(lrows))
        with torch.no_grad():
            x = self.fwd.hidden_states(db)
            logits = self.fwd.logits_from_hidden(x, db)
        self._last_hidden = x
        self.stats.eager_steps += 1
        return ExecutionOutput([self._row_output(r, b.logits[r], logits[i]) for i, r in enumerate(lrows)])

    def observability(self) -> Dict[str, object]:
        d = super().observability()
        d["model"] = self.cfg.name
        d["state_pool_bytes"] = self.states.nbytes
        return d
