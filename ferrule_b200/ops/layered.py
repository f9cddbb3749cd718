"""Launchers of the layer-list model kernels (csrc/layered_ops.cu, stream_ops.cu, delta_rule.cu, selective_scan.cu,
gqa_*.cu, head_prep.cu, pre_norm.cu, head_scan.cu).

Activations are bf16, or fp32 for models that run in full 32 bits: the launcher follows the tensors' dtype.
"""
from __future__ import annotations

import ctypes as C
import functools
from typing import Optional

import torch

from . import _lib
from ._lib import (AttnArgs, ConvArgs, DeltaArgs, GqaArgs, HeadPrepArgs, HeadScanArgs, LatentPrepArgs, LayerTailArgs, PoolArgs,
                   PreNormArgs, SandwichArgs, ScanArgs, StreamArgs, check, get_lib, ptr, status_tensor, stream_ptr)


def _fp32(t: torch.Tensor) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32)
    return 1 if t.dtype == torch.float32 else 0


def embed_norm(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, norm_w: torch.Tensor, h: torch.Tensor, dim: int,
               eps: float) -> None:
    """x = table[ids] (fp32), h = RMSNorm(x) * norm_w (one number, or a vector over `dim`)."""
    assert x.dtype == torch.float32 and table.dtype == h.dtype and norm_w.dtype == torch.float32
    check(get_lib(True).fb_embed_norm(ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0], x.data_ptr(),
                                      x.stride(0), norm_w.data_ptr(), 0 if norm_w.numel() == 1 else 1, h.data_ptr(),
                                      h.stride(0), ids.shape[0], dim, table.shape[1], eps, _fp32(h),
                                      status_tensor(x.device).data_ptr(), stream_ptr()), "fb_embed_norm")


def gated_residual_norm(x: torch.Tensor, norm_w: torch.Tensor, h: torch.Tensor, dim: int, eps: float, *,
                        mix: Optional[torch.Tensor] = None, gate1: Optional[torch.Tensor] = None,
                        bias1: Optional[torch.Tensor] = None, ffn: Optional[torch.Tensor] = None, topk: int = 0,
                        gate2: Optional[torch.Tensor] = None, bias2: Optional[torch.Tensor] = None) -> None:
    """x += sigmoid(gate1 + bias1) * mix + sigmoid(gate2 + bias2) * sum(ffn rows of the token); h = RMSNorm(x) * norm_w.
    ffn: [rows, slots, width], of which the first `topk` slots are summed."""
    a = LayerTailArgs()
    a.x, a.ldx, a.rows, a.dim, a.dim_pad, a.eps, a.fp32 = x.data_ptr(), x.stride(0), x.shape[0], dim, h.shape[1], eps, _fp32(h)
    a.norm_w, a.norm_stride = norm_w.data_ptr(), 0 if norm_w.numel() == 1 else 1
    a.h, a.ldh = h.data_ptr(), h.stride(0)
    if mix is not None:
        assert mix.dtype == h.dtype
        a.mix, a.ldm = mix.data_ptr(), mix.stride(0)
    if gate1 is not None:
        a.gate1, a.ldg1, a.bias1 = gate1.data_ptr(), gate1.stride(0), bias1.data_ptr()
    if ffn is not None:
        assert ffn.dtype == h.dtype and ffn.dim() == 3 and ffn.is_contiguous() and topk <= ffn.shape[1]
        a.ffn, a.ldf, a.slots, a.topk = ffn.data_ptr(), ffn.stride(1), ffn.shape[1], topk
    if gate2 is not None:
        a.gate2, a.ldg2, a.bias2 = gate2.data_ptr(), gate2.stride(0), bias2.data_ptr()
    check(get_lib(True).fb_gated_residual_norm(C.byref(a), stream_ptr()), "fb_gated_residual_norm")


def latent_append(src: torch.Tensor, rank: int, norm_w: torch.Tensor, eps: float, write_slot: torch.Tensor,
                  pool_layer: torch.Tensor) -> None:
    """pool row of every token <- RMSNorm(src[:, :rank]) * norm_w, padded with zeros to the pool's row width."""
    rows, row_dim = src.shape[0], pool_layer.shape[-1]
    assert pool_layer.is_contiguous() and pool_layer.dtype == src.dtype and norm_w.numel() == row_dim
    check(get_lib(True).fb_latent_append(src.data_ptr(), src.stride(0), rank, row_dim, norm_w.data_ptr(), eps,
                                         write_slot.data_ptr(), pool_layer.data_ptr(), pool_layer.numel() // row_dim, rows,
                                         _fp32(src), status_tensor(src.device).data_ptr(), stream_ptr()),
          "fb_latent_append")


def softcap_(logits: torch.Tensor, cap: float) -> torch.Tensor:
    """logits <- cap * tanh(logits / cap) (fp32)."""
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    check(get_lib(True).fb_softcap(logits.data_ptr(), logits.stride(0), logits.shape[0], logits.shape[1], cap,
                                   stream_ptr()), "fb_softcap")
    return logits


def state_rotate(state_in: torch.Tensor, state_out: torch.Tensor, buffers: int) -> None:
    """The next step reads what this one wrote: state_in <- state_out <- the slot's next buffer."""
    check(get_lib(True).fb_state_rotate(state_in.data_ptr(), state_out.data_ptr(), state_in.numel(), buffers,
                                        stream_ptr()), "fb_state_rotate")


def latent_attention(q: torch.Tensor, kv_layer: torch.Tensor, block_table: torch.Tensor, row_seq: torch.Tensor,
                     row_pos: torch.Tensor, page_size: int, scale: float, out: torch.Tensor,
                     gate: Optional[torch.Tensor] = None, window: int = 0) -> torch.Tensor:
    """Causal attention over a latent cache in 32-bit arithmetic: q / out [rows, heads, row_dim].  window > 0: the last
    `window` tokens of a row only."""
    rows, heads, D = q.shape
    assert q.stride(1) == D and out.stride(1) == D and kv_layer.shape[-1] == D and kv_layer.dtype == q.dtype
    a = AttnArgs()
    a.q, a.kv, a.out = q.data_ptr(), kv_layer.data_ptr(), out.data_ptr()
    a.block_table, a.row_seq, a.row_pos = block_table.data_ptr(), row_seq.data_ptr(), row_pos.data_ptr()
    a.status = status_tensor(q.device).data_ptr()
    a.ldq, a.ldo, a.pool_rows = q.stride(0), out.stride(0), kv_layer.numel() // D
    a.rows, a.heads, a.kv_lora = rows, heads, D
    a.num_seqs, a.max_blocks, a.page_size = block_table.shape[0], block_table.shape[1], page_size
    a.softmax_scale, a.window = scale, window
    if gate is not None:
        a.gate, a.ldg = gate.data_ptr(), gate.stride(0)
    check(get_lib(True).fb_latent_attention(C.byref(a), _fp32(q), stream_ptr()), "fb_latent_attention")
    return out


def latent_prep(proj: torch.Tensor, off, mixer, img, rotation, positions: torch.Tensor, write_slot: torch.Tensor,
                pool_layer: torch.Tensor, eps: float) -> None:
    """Latent layers with a query latent or a rotated part: the query latent (block `dq` of the projection) is normalised in
    place, the cache row of every token is [RMSNorm(latent) | turned key part | zeros].  rotation = (cos, sin) fp32
    [positions, rot_dim / 2]."""
    a = LatentPrepArgs()
    item, DL = proj.element_size(), pool_layer.shape[-1]
    assert pool_layer.is_contiguous() and pool_layer.dtype == proj.dtype and DL == mixer.row_dim and write_slot.dtype == torch.int64
    if mixer.q_rank:
        a.cq, a.rank_q, a.q_w = proj.data_ptr() + off["dq"] * item, mixer.q_rank, img.dq_norm.data_ptr()
    a.ckv, a.ldp = proj.data_ptr() + off["dkv"] * item, proj.stride(0)
    a.rank, a.rot, a.row_dim, a.rot_off, a.rows = mixer.kv_rank, mixer.rot_dim, DL, mixer.rot_offset, proj.shape[0]
    a.kv_w, a.fp32, a.eps = img.kv_norm.data_ptr(), _fp32(proj), eps
    if mixer.rot_dim:
        a.cos_t, a.sin_t, a.max_pos = rotation[0].data_ptr(), rotation[1].data_ptr(), rotation[0].shape[0]
        a.positions = positions.data_ptr()
    a.write_slot, a.pool, a.pool_rows = write_slot.data_ptr(), pool_layer.data_ptr(), pool_layer.numel() // DL
    a.status = status_tensor(proj.device).data_ptr()
    check(get_lib(True).fb_latent_prep(C.byref(a), stream_ptr()), "fb_latent_prep")


def latent_turn(src: torch.Tensor, mixer, rotation, positions: torch.Tensor, q: torch.Tensor) -> None:
    """Rotated query parts (src [rows, heads * rot_dim]) into their columns of the query rows q [rows, heads, row_dim]."""
    rows, heads, DL = q.shape
    assert src.dtype == q.dtype and q.stride(1) == DL and src.stride(1) == 1
    check(get_lib(True).fb_latent_turn(src.data_ptr(), src.stride(0), heads, mixer.rot_dim, rotation[0].data_ptr(),
                                       rotation[1].data_ptr(), rotation[0].shape[0], positions.data_ptr(), q.data_ptr(),
                                       q.stride(0), DL, mixer.rot_offset, rows, _fp32(q), status_tensor(q.device).data_ptr(),
                                       stream_ptr()), "fb_latent_turn")


class DeltaScratch:
    """Intermediate rows of the prefill form of the delta rule, for mixers up to the given sizes."""

    def __init__(self, rows: int, mixers, device):
        f32 = dict(dtype=torch.float32, device=device)
        big = lambda f: max(f(m) for m in mixers)
        self.rows = rows
        self.qn = torch.empty(rows * big(lambda m: m.kv_heads * m.dim), **f32)
        self.kn = torch.empty_like(self.qn)
        self.decay = torch.empty(rows * big(lambda m: m.heads if m.head_decay else m.heads * m.dim), **f32)
        self.v = torch.empty(rows * big(lambda m: m.heads * m.vdim), **f32)
        self.o = torch.empty_like(self.v)
        self.beta = torch.empty(rows * big(lambda m: m.heads), **f32)
        self.qk = torch.empty(rows * big(lambda m: m.kv_heads), **f32)


def delta_decode_supported(mixer) -> bool:
    return mixer.vdim <= 128 and mixer.vdim % 4 == 0 and mixer.dim <= 128


def delta_rule(proj: torch.Tensor, off, ag: Optional[torch.Tensor], img, mixer, eps: float, state: torch.Tensor,
               tail: torch.Tensor, seq_start: torch.Tensor, state_in: torch.Tensor, state_out: torch.Tensor, n_seqs: int,
               out: torch.Tensor, *, row_seq: Optional[torch.Tensor] = None, scratch: Optional[DeltaScratch] = None,
               decode: bool = False, long_seqs: int = 0) -> torch.Tensor:
    """Convolutions, recurrence and gated output norm of a delta mixer over the rows of a packed batch.
    proj: rows of the layer's input projection, `off` its block offsets; ag: fp32 rows of the second low-rank halves (None:
    decay and gate pre-activations are blocks `a` and `g` of the projection, one decay per head);
    decode: one row per sequence, a single launch; long_seqs: sequences with more than one row, when known."""
    assert (ag is None) == mixer.head_decay and (ag is None or ag.dtype == torch.float32)
    assert state.dtype == torch.float32 and state.is_contiguous() and tail.is_contiguous()
    assert tail.dtype == proj.dtype == out.dtype
    a = DeltaArgs()
    a.proj, a.ldp = proj.data_ptr(), proj.stride(0)
    a.off_q, a.off_k, a.off_v, a.off_b = off["q"], off["k"], off["v"], off["b"]
    a.ag, a.ldag, a.off_gate, a.fp32 = ptr(ag), ag.stride(0) if ag is not None else 0, img.off_gate, _fp32(proj)
    a.off_a, a.off_g = (off["a"], off["g"]) if ag is None else (-1, -1)
    a.gate_silu, a.long_seqs = 1 if mixer.gate == "silu" else 0, long_seqs
    a.conv, a.a_neg, a.dt_bias, a.norm_w = (img.conv.data_ptr(), img.a_neg.data_ptr(), img.dt_bias.data_ptr(),
                                            img.o_norm.data_ptr())
    a.state, a.tail, a.n_states = state.data_ptr(), tail.data_ptr(), state.shape[0]
    a.row_seq, a.seq_start = ptr(row_seq), seq_start.data_ptr()
    a.state_in, a.state_out = state_in.data_ptr(), state_out.data_ptr()
    a.rows, a.n_seqs = proj.shape[0], n_seqs
    a.heads, a.kv_heads, a.dim, a.vdim, a.taps = mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim, mixer.taps
    a.out, a.ldo, a.eps = out.data_ptr(), out.stride(0), eps
    a.status = status_tensor(proj.device).data_ptr()
    if decode:
        assert n_seqs == proj.shape[0]
        check(get_lib(True).fb_delta_decode(C.byref(a), stream_ptr()), "fb_delta_decode")
        return out
    assert scratch is not None and scratch.rows >= proj.shape[0]
    a.qn, a.kn, a.v, a.decay = (scratch.qn.data_ptr(), scratch.kn.data_ptr(), scratch.v.data_ptr(),
                                scratch.decay.data_ptr())
    a.beta, a.qk, a.o = scratch.beta.data_ptr(), scratch.qk.data_ptr(), scratch.o.data_ptr()
    check(get_lib(True).fb_delta_prefill(C.byref(a), stream_ptr()), "fb_delta_prefill")
    _lib.LAUNCHES[0] += 2                    # prepare, scan, output
    return out


# ------------------------------------------------------------------ output-norm blocks
def _canon(a: StreamArgs, conv, tail, state_in, state_out, h) -> None:
    a.conv, a.taps = conv.data_ptr(), conv.shape[0]
    a.tail, a.n_states = tail.data_ptr(), tail.shape[0]
    a.state_in, a.state_out = state_in.data_ptr(), state_out.data_ptr()
    a.h, a.ldh = h.data_ptr(), h.stride(0)
    assert tail.is_contiguous() and tail.dtype == torch.float32 and conv.is_contiguous()


def _stream(x: torch.Tensor, dim: int, like: torch.Tensor, act: Optional[torch.Tensor], canon) -> StreamArgs:
    assert x.dtype == torch.float32 and (act is None or act.dtype == like.dtype)
    a = StreamArgs()
    a.x, a.ldx, a.rows, a.dim, a.dim_pad, a.fp32 = x.data_ptr(), x.stride(0), x.shape[0], dim, x.shape[1], _fp32(like)
    a.status = status_tensor(x.device).data_ptr()
    if act is not None:
        a.act, a.lda = act.data_ptr(), act.stride(0)
    if canon is not None:
        _canon(a, *canon)
    return a


def embed_stream(ids: torch.Tensor, table: torch.Tensor, x: torch.Tensor, dim: int, *,
                 positions: Optional[torch.Tensor] = None, pos_table: Optional[torch.Tensor] = None, canon=None) -> None:
    """x = table[ids] (+ pos_table[positions]).  canon = (filters [taps, width], state plane, state_in, state_out, h): one
    row per sequence, h = x + conv(x) with the convolution's state."""
    a = _stream(x, dim, table, None, canon)
    a.ids, a.table, a.ldt, a.vocab = ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0]
    if pos_table is not None:
        assert pos_table.dtype == table.dtype and pos_table.stride(0) == table.stride(0)
        a.positions, a.pos_table, a.max_pos = positions.data_ptr(), pos_table.data_ptr(), pos_table.shape[0]
    check(get_lib(True).fb_stream_step(C.byref(a), stream_ptr()), "fb_stream_step")


def add_normed(x: torch.Tensor, y: torch.Tensor, norm: torch.Tensor, dim: int, eps: float, *,
               act: Optional[torch.Tensor] = None, canon=None, rms: bool = False) -> None:
    """x += norm(y); norm: [2, width] weight and bias of a layer norm (rms: [1, width], an RMS norm).  act: the new rows as
    activations; canon as in `embed_stream`."""
    a = _stream(x, dim, y, act, canon)
    a.y, a.ldy, a.eps, a.rms = y.data_ptr(), y.stride(0), eps, 1 if rms else 0
    a.norm_w, a.norm_b = norm[0].data_ptr(), None if rms else norm[1].data_ptr()
    check(get_lib(True).fb_stream_step(C.byref(a), stream_ptr()), "fb_stream_step")


def norm_rows(x: torch.Tensor, rows: torch.Tensor, norm: torch.Tensor, out: torch.Tensor, dim: int, eps: float,
              rms: bool = False) -> torch.Tensor:
    """out[i] = norm(x[rows[i]]) (see `add_normed`)."""
    assert x.dtype == torch.float32 and rows.dtype == torch.int32 and out.shape[0] == rows.shape[0]
    check(get_lib(True).fb_norm_rows(x.data_ptr(), x.stride(0), x.shape[0], rows.data_ptr(), rows.shape[0], norm[0].data_ptr(),
                                     None if rms else norm[1].data_ptr(), 1 if rms else 0, out.data_ptr(), out.stride(0), dim,
                                     x.shape[1], eps, _fp32(out), status_tensor(x.device).data_ptr(), stream_ptr()),
          "fb_norm_rows")
    return out


def sandwich_step(x: torch.Tensor, *, dim: int, eps: float, groups: int, y: Optional[torch.Tensor] = None,
                  bias: Optional[torch.Tensor] = None, out_norm: Optional[torch.Tensor] = None,
                  ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None, fresh: bool = False,
                  in_norm: Optional[torch.Tensor] = None, act: Optional[torch.Tensor] = None) -> None:
    """x (zeros when `fresh`) += norm(y + bias) * out_norm + table[ids]; act = norm(x) * in_norm.  Every norm divides each of
    `groups` equal parts of a row by its own root mean square."""
    a = SandwichArgs()
    assert x.dtype == torch.float32 and dim % groups == 0 and (act is None) == (in_norm is None)
    like = next(t for t in (y, table, act) if t is not None)
    a.x, a.ldx, a.rows, a.dim, a.dim_pad, a.groups, a.eps, a.fp32 = (x.data_ptr(), x.stride(0), x.shape[0], dim, x.shape[1],
                                                                     groups, eps, _fp32(like))
    if y is not None:
        a.y, a.ldy, a.out_w, a.y_bias = y.data_ptr(), y.stride(0), out_norm.data_ptr(), ptr(bias)
    if ids is not None:
        assert table.dtype == like.dtype
        a.ids, a.table, a.ldt, a.vocab = ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0]
    if act is not None:
        assert act.dtype == like.dtype
        a.in_w, a.act, a.lda = in_norm.data_ptr(), act.data_ptr(), act.stride(0)
    a.fresh, a.status = int(fresh), status_tensor(x.device).data_ptr()
    check(get_lib(True).fb_sandwich_step(C.byref(a), stream_ptr()), "fb_sandwich_step")


def sandwich_rows(x: torch.Tensor, rows: torch.Tensor, norm: torch.Tensor, out: torch.Tensor, dim: int, eps: float,
                  groups: int) -> torch.Tensor:
    """out[i] = norm(x[rows[i]]) (see `sandwich_step`)."""
    assert x.dtype == torch.float32 and rows.dtype == torch.int32 and out.shape[0] == rows.shape[0] and dim % groups == 0
    check(get_lib(True).fb_sandwich_rows(x.data_ptr(), x.stride(0), x.shape[0], rows.data_ptr(), rows.shape[0],
                                         norm.data_ptr(), out.data_ptr(), out.stride(0), dim, x.shape[1], groups, eps,
                                         _fp32(out), status_tensor(x.device).data_ptr(), stream_ptr()), "fb_sandwich_rows")
    return out


def pre_norm_step(x: Optional[torch.Tensor], x_out: torch.Tensor, *, dim: int, eps: float, like: torch.Tensor,
                  ids: Optional[torch.Tensor] = None, table: Optional[torch.Tensor] = None, scale: float = 1.0,
                  y: Optional[torch.Tensor] = None, ffn: Optional[torch.Tensor] = None, topk: int = 0,
                  shared: Optional[torch.Tensor] = None, shared_gate: Optional[torch.Tensor] = None,
                  norm: Optional[torch.Tensor] = None, act: Optional[torch.Tensor] = None, shift: Optional[torch.Tensor] = None,
                  plane: Optional[torch.Tensor] = None, seqs=None) -> None:
    """x_out = (x, or table[ids] * scale) + y + the first `topk` of a token's ffn rows [rows, slots, width] + sigmoid(shared_gate)
    shared; act = RMSNorm(x_out) * norm, with `shift` moved towards the previous token's row.  plane: the shift's state;
    seqs = (row_seq, seq_start, state_in, state_out, n_seqs).  `like` has the activations' dtype."""
    a = PreNormArgs()
    assert x_out.dtype == torch.float32 and (x is None or (x.dtype == torch.float32 and x.stride(0) == x_out.stride(0)))
    assert all(t is None or t.dtype == like.dtype for t in (table, y, ffn, shared, act))
    a.x, a.x_out, a.ldx = ptr(x), x_out.data_ptr(), x_out.stride(0)
    if ids is not None:
        a.ids, a.table, a.ldt, a.vocab, a.scale = ids.data_ptr(), table.data_ptr(), table.stride(0), table.shape[0], scale
    if y is not None:
        a.y, a.ldy = y.data_ptr(), y.stride(0)
    if ffn is not None:
        assert ffn.dim() == 3 and ffn.is_contiguous() and topk <= ffn.shape[1]
        a.ffn, a.ldf, a.slots, a.topk = ffn.data_ptr(), ffn.stride(1), ffn.shape[1], topk
    if shared is not None:
        assert shared_gate.dtype == torch.float32
        a.shared, a.lds, a.shared_gate, a.ldsg = shared.data_ptr(), shared.stride(0), shared_gate.data_ptr(), shared_gate.stride(0)
    if act is not None:
        a.norm_w, a.act, a.lda = norm.data_ptr(), act.data_ptr(), act.stride(0)
    if shift is not None:
        assert plane.dtype == torch.float32 and plane.is_contiguous() and plane.shape[1] == x_out.shape[1]
        a.shift, a.plane, a.n_states = shift.data_ptr(), plane.data_ptr(), plane.shape[0]
        a.row_seq, a.seq_start, a.state_in, a.state_out = (t.data_ptr() for t in seqs[:4])
        a.n_seqs = seqs[4]
    a.rows, a.dim, a.dim_pad, a.fp32, a.eps = x_out.shape[0], dim, x_out.shape[1], _fp32(like), eps
    a.status = status_tensor(x_out.device).data_ptr()
    check(get_lib(True).fb_pre_norm_step(C.byref(a), stream_ptr()), "fb_pre_norm_step")


def group_norm_rows(x: torch.Tensor, norm: torch.Tensor, out: torch.Tensor, dim: int, groups: int, eps: float) -> torch.Tensor:
    """out = x with each of `groups` equal parts of a row divided by its root mean square, times norm (in place allowed)."""
    assert x.dtype == out.dtype and x.shape == out.shape
    check(get_lib(True).fb_group_norm_rows(x.data_ptr(), x.stride(0), norm.data_ptr(), out.data_ptr(), out.stride(0), x.shape[0],
                                           dim, x.shape[1], groups, eps, _fp32(x), stream_ptr()), "fb_group_norm_rows")
    return out


def head_scan(xbc: torch.Tensor, proj: torch.Tensor, off, mixer, img, states: torch.Tensor, seq_start: torch.Tensor,
              state_in: torch.Tensor, state_out: torch.Tensor, n_seqs: int, out: torch.Tensor, long_seqs: int = 0,
              by_token: bool = False) -> torch.Tensor:
    """(scan + D x) * silu(z) of a head-decay scan over packed rows: xbc the convolved x | B | C, z and dt blocks of the
    projection; long_seqs: sequences with more than one row, when known; by_token: prompts not in chunks."""
    assert states.dtype == torch.float32 and states.is_contiguous() and xbc.dtype == proj.dtype == out.dtype
    a = HeadScanArgs()
    item = proj.element_size()
    a.xbc, a.ldx, a.off_b, a.off_c = xbc.data_ptr(), xbc.stride(0), img.off_b, img.off_c
    a.dt, a.z, a.ldp = proj.data_ptr() + off["dt"] * item, proj.data_ptr() + off["z"] * item, proj.stride(0)
    a.dt_bias, a.a_neg, a.d_skip = img.dt_bias.data_ptr(), img.a_neg.data_ptr(), img.d_skip.data_ptr()
    a.states, a.n_states = states.data_ptr(), states.shape[0]
    a.seq_start, a.state_in, a.state_out = seq_start.data_ptr(), state_in.data_ptr(), state_out.data_ptr()
    a.out, a.ldo, a.rows, a.n_seqs, a.fp32 = out.data_ptr(), out.stride(0), xbc.shape[0], n_seqs, _fp32(xbc)
    a.long_seqs, a.by_token = long_seqs, int(by_token)
    a.heads, a.vdim, a.state, a.groups = mixer.heads, mixer.vdim, mixer.state, mixer.groups
    a.status = status_tensor(xbc.device).data_ptr()
    check(get_lib(True).fb_head_scan(C.byref(a), stream_ptr()), "fb_head_scan")
    return out


def short_conv(x: torch.Tensor, w: torch.Tensor, tail: torch.Tensor, out: torch.Tensor, row_seq: torch.Tensor,
               seq_start: torch.Tensor, state_in: torch.Tensor, state_out: torch.Tensor, n_seqs: int, *,
               bias: Optional[torch.Tensor] = None, residual: bool = False, silu: bool = False) -> torch.Tensor:
    """Causal convolution of packed rows with one filter per channel: x [rows, channels], w fp32 [taps, channels].
    residual: out = x + conv(x); silu: out = silu(conv(x) + bias)."""
    assert tail.dtype == x.dtype and tail.is_contiguous() and tail.shape[-1] == w.shape[1] and w.is_contiguous()
    a = ConvArgs()
    a.x, a.ldx, a.w, a.bias, a.tail = x.data_ptr(), x.stride(0), w.data_ptr(), ptr(bias), tail.data_ptr()
    a.out, a.ldo = out.data_ptr(), out.stride(0)
    a.row_seq, a.seq_start, a.state_in, a.state_out = (row_seq.data_ptr(), seq_start.data_ptr(), state_in.data_ptr(),
                                                       state_out.data_ptr())
    a.rows, a.channels, a.taps, a.n_states, a.n_seqs = x.shape[0], w.shape[1], w.shape[0], tail.shape[0], n_seqs
    a.x_fp32, a.out_fp32, a.residual, a.silu = _fp32(x), _fp32(out), int(residual), int(silu)
    a.status = status_tensor(x.device).data_ptr()
    check(get_lib(True).fb_short_conv(C.byref(a), stream_ptr()), "fb_short_conv")
    return out


def selective_scan(x: torch.Tensor, z: torch.Tensor, bc: torch.Tensor, off_b: int, off_c: int, dt: torch.Tensor, img,
                   states: torch.Tensor, seq_start: torch.Tensor, state_in: torch.Tensor, state_out: torch.Tensor,
                   n_seqs: int, out: torch.Tensor) -> torch.Tensor:
    """(scan + D x) * silu(z) over packed rows; x, z, out [rows, inner], bc rows with B at off_b and C at off_c, dt fp32
    [rows, inner] without bias; img: a_log2, dt_bias, d_skip."""
    assert dt.dtype == torch.float32 and states.dtype == torch.float32 and states.is_contiguous()
    assert x.dtype == z.dtype == bc.dtype == out.dtype
    a = ScanArgs()
    a.x, a.ldx, a.z, a.ldz, a.bc, a.ldbc = x.data_ptr(), x.stride(0), z.data_ptr(), z.stride(0), bc.data_ptr(), bc.stride(0)
    a.off_b, a.off_c, a.dt, a.lddt = off_b, off_c, dt.data_ptr(), dt.stride(0)
    a.dt_bias, a.a_log2, a.d_skip = img.dt_bias.data_ptr(), img.a_log2.data_ptr(), img.d_skip.data_ptr()
    a.states, a.n_states, a.state, a.inner = states.data_ptr(), states.shape[0], states.shape[1], states.shape[2]
    a.seq_start, a.state_in, a.state_out = seq_start.data_ptr(), state_in.data_ptr(), state_out.data_ptr()
    a.out, a.ldo, a.rows, a.n_seqs, a.fp32 = out.data_ptr(), out.stride(0), x.shape[0], n_seqs, _fp32(x)
    a.status = status_tensor(x.device).data_ptr()
    check(get_lib(True).fb_selective_scan(C.byref(a), stream_ptr()), "fb_selective_scan")
    return out


# ------------------------------------------------------------------ grouped-query attention in chunks and windows
def _gqa(q: torch.Tensor, mixer, pool: torch.Tensor, slopes: Optional[torch.Tensor] = None,
         gate: Optional[torch.Tensor] = None, diff_lambda: float = 0.0, eps: float = 0.0, mean=None,
         talk: Optional[torch.Tensor] = None) -> GqaArgs:
    a = GqaArgs()
    assert q.dtype == pool.dtype and pool.is_contiguous()
    a.q, a.ldq, a.rows, a.fp32 = q.data_ptr(), q.stride(0), q.shape[0], _fp32(q)
    a.pool, a.pool_ld, a.pool_rows = pool.data_ptr(), pool.shape[-1], pool.numel() // pool.shape[-1]
    a.heads, a.kv_heads, a.dim, a.vdim, a.dim_pad, a.vdim_pad = (mixer.heads, mixer.kv_heads, mixer.dim, mixer.vdim,
                                                                 mixer.dim_pad, mixer.vdim_pad)
    a.chunk, a.window, a.keep_first = mixer.chunk, mixer.window, mixer.keep_first
    a.maps, a.key_width, a.v_offset = mixer.maps, mixer.key_width, mixer.v_offset
    a.key_stride = 0 if mixer.shared_keys else mixer.key_width
    a.slopes, a.eps, a.diff_lambda = ptr(slopes), eps, diff_lambda
    a.diff_scale = 1.0 - mixer.diff if mixer.maps == 2 else 1.0
    a.value_width, a.value_stride = mixer.value_width, 0 if mixer.shared_values else mixer.vdim_pad
    a.softcap, a.score_bound, a.talk = mixer.softcap, mixer.score_bound, ptr(talk)
    if mean is not None:
        rows, a.slot_div, slots = mean
        assert rows.dtype == q.dtype and rows.is_contiguous() and rows.shape[2] == pool.shape[-1]
        a.pooled, a.pooled_rows, a.pooled_stride, a.pool_tokens = rows.data_ptr(), rows.shape[0] * rows.shape[1], rows.shape[1], mixer.pool
        a.slot_of = slots.data_ptr()
    if gate is not None:
        assert gate.dtype == q.dtype
        a.gate, a.ldg = gate.data_ptr(), gate.stride(0)
    a.status = status_tensor(q.device).data_ptr()
    return a


def _scaled(a: GqaArgs, mixer) -> GqaArgs:
    """Scale of the products q . k: queries that `head_prep` wrote carry theirs."""
    a.scale = 1.0 if mixer.scaled_queries else mixer.scale
    return a


def _pool_args(mixer, pool: torch.Tensor, mean, positions, row_seq, block_table, page_size: int) -> PoolArgs:
    rows, div, slots = mean
    a = PoolArgs()
    assert rows.dtype == pool.dtype and rows.is_contiguous() and pool.is_contiguous() and rows.shape[2] == pool.shape[-1]
    a.pool, a.pool_ld, a.pool_rows = pool.data_ptr(), pool.shape[-1], pool.numel() // pool.shape[-1]
    a.pooled, a.pooled_rows, a.pooled_stride, a.slot_div = rows.data_ptr(), rows.shape[0] * rows.shape[1], rows.shape[1], div
    a.positions, a.row_seq, a.block_table, a.slot_of = (positions.data_ptr(), row_seq.data_ptr(), block_table.data_ptr(),
                                                        slots.data_ptr())
    a.rows, a.width, a.num_seqs, a.max_blocks = positions.shape[0], mixer.row_dim, block_table.shape[0], block_table.shape[1]
    a.page_size, a.pool_tokens, a.fp32 = page_size, mixer.pool, _fp32(pool)
    a.status = status_tensor(pool.device).data_ptr()
    return a


def pool_blocks(mixer, pool: torch.Tensor, mean, positions: torch.Tensor, row_seq: torch.Tensor, block_table: torch.Tensor,
                page_size: int) -> None:
    """Mean cache rows of the blocks that end with rows of this batch, whose cache rows are written.  mean = (rows [slots,
    blocks, row width], divisor, slot numbers): sequence s owns rows[slots[s] // divisor]."""
    a = _pool_args(mixer, pool, mean, positions, row_seq, block_table, page_size)
    check(get_lib(True).fb_pool_blocks(C.byref(a), stream_ptr()), "fb_pool_blocks")


def head_prep(proj: torch.Tensor, off, mixer, img, write_slot: torch.Tensor, pool: torch.Tensor, eps: float,
              q_out: torch.Tensor, rotation=None, positions: Optional[torch.Tensor] = None, blocks=None) -> None:
    """Between the projection and window attention: biases, rotation, query and key norm per head, factors and mixing of the
    queries across heads (into q_out, which may be the projection's own queries), cache append of keys and values.  blocks
    (one row per sequence) = the further arguments of `pool_blocks`."""
    assert proj.dtype == pool.dtype == q_out.dtype and pool.is_contiguous() and write_slot.dtype == torch.int64
    a = HeadPrepArgs()
    item = proj.element_size()
    at = lambda name: proj.data_ptr() + off[name] * item
    a.q, a.k, a.v, a.ldp = at("q"), at("k"), None if mixer.tied_values else at("v"), proj.stride(0)
    a.q_bias, a.k_bias, a.q_norm, a.k_norm = ptr(img.q_bias), ptr(img.k_bias), ptr(img.q_norm), ptr(img.k_norm)
    if mixer.rot_dims:
        a.cos_t, a.sin_t, a.max_pos, a.half = (rotation[0].data_ptr(), rotation[1].data_ptr(), rotation[0].shape[0],
                                               mixer.rot_dims // 2)
        a.positions = positions.data_ptr()
    if blocks is not None:
        pool_args = _pool_args(mixer, pool, *blocks)
        a.blocks = C.pointer(pool_args)
    a.q_mix, a.mix, a.q_out, a.ldqo = img.q_mix.data_ptr(), int(mixer.mix_heads), q_out.data_ptr(), q_out.stride(0)
    a.write_slot, a.pool, a.pool_ld, a.pool_rows = (write_slot.data_ptr(), pool.data_ptr(), pool.shape[-1],
                                                    pool.numel() // pool.shape[-1])
    a.rows, a.heads, a.kv_heads, a.maps, a.dim, a.dim_pad, a.vdim_pad = (proj.shape[0], mixer.heads, mixer.kv_heads, mixer.maps,
                                                                         mixer.dim, mixer.dim_pad, mixer.vdim_pad)
    a.fp32, a.eps, a.status = _fp32(proj), eps, status_tensor(proj.device).data_ptr()
    check(get_lib(True).fb_head_prep(C.byref(a), stream_ptr()), "fb_head_prep")


def gqa_prep(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, mixer, img, rotation, positions: torch.Tensor,
             write_slot: torch.Tensor, pool: torch.Tensor, eps: float, first_pool: Optional[torch.Tensor] = None,
             first_off: int = 0) -> None:
    """Query rows are normalised and rotated in place; keys and values go into the pool rows of their tokens.
    rotation = (cos, sin) fp32 [positions, rot_dims / 2]; first_pool: the pool of the layer whose values are mixed in, at
    column first_off."""
    a = _scaled(_gqa(q, mixer, pool), mixer)
    assert k.stride(0) == v.stride(0)
    a.k, a.v, a.ldkv = k.data_ptr(), v.data_ptr(), k.stride(0)
    a.q_norm, a.k_norm = img.q_norm.data_ptr(), img.k_norm.data_ptr()
    a.cos_t, a.sin_t, a.max_pos = rotation[0].data_ptr(), rotation[1].data_ptr(), rotation[0].shape[0]
    a.positions, a.write_slot, a.eps = positions.data_ptr(), write_slot.data_ptr(), eps
    a.rot_dims = mixer.rot_dims
    if first_pool is not None:
        assert first_pool.shape == pool.shape
        a.first_pool, a.first_off, a.v_mix = first_pool.data_ptr(), first_off, img.v_mix
    check(get_lib(True).fb_gqa_prep(C.byref(a), stream_ptr()), "fb_gqa_prep")


def _gqa_rows(a: GqaArgs, block_table, row_seq, row_pos, page_size: int, out: torch.Tensor) -> None:
    if row_seq is not None:
        a.row_seq, a.row_pos = row_seq.data_ptr(), row_pos.data_ptr()
    a.block_table, a.num_seqs, a.max_blocks, a.page_size = (block_table.data_ptr(), block_table.shape[0],
                                                            block_table.shape[1], page_size)
    a.out, a.ldo = out.data_ptr(), out.stride(0)


def gqa_attention(q: torch.Tensor, mixer, pool: torch.Tensor, block_table: torch.Tensor, row_seq: torch.Tensor,
                  row_pos: torch.Tensor, page_size: int, out: torch.Tensor, **form) -> torch.Tensor:
    """32-bit arithmetic: out [rows, heads * value_width].  form: slopes, gate, diff_lambda, eps, mean of a window mixer."""
    a = _scaled(_gqa(q, mixer, pool, **form), mixer)
    _gqa_rows(a, block_table, row_seq, row_pos, page_size, out)
    check(get_lib(True).fb_gqa_attention(C.byref(a), stream_ptr()), "fb_gqa_attention")
    return out


def value_mix(o: torch.Tensor, talk: torch.Tensor, mixer, out: torch.Tensor) -> torch.Tensor:
    """Outputs of every head on the values of every kv head (o [rows, heads * value_width]) -> those of mixed softmax weights."""
    assert o.dtype == out.dtype and talk.dtype == torch.float32 and talk.is_contiguous() and mixer.shared_values
    check(get_lib(True).fb_value_mix(o.data_ptr(), o.stride(0), talk.data_ptr(), out.data_ptr(), out.stride(0), o.shape[0],
                                     mixer.heads, mixer.kv_heads, mixer.vdim_pad, _fp32(o), stream_ptr()), "fb_value_mix")
    return out


def gqa_tc_group(mixer, dtype, page_size: int) -> int:
    """Query rows per key / value head when the bf16 prompt kernel serves the mixer, else 0."""
    per = mixer.heads // mixer.kv_heads * mixer.maps
    ok = (dtype == torch.bfloat16 and (mixer.vdim_pad <= 256 or mixer.shared_values) and per <= 128
          and (mixer.shared_keys or mixer.key_width <= 256) and (mixer.scaled_queries or mixer.scale > 0)
          and page_size >= 8 and page_size & (page_size - 1) == 0)
    return per if ok else 0


def latent_tc_group(mixer, dtype, page_size: int) -> int:
    """Query rows per position when the bf16 prompt kernel serves the latent mixer, else 0."""
    from .kernels import prefill_tc_supported
    ok = dtype == torch.bfloat16 and prefill_tc_supported(mixer.heads, mixer.value_dim, mixer.row_dim - mixer.value_dim, page_size)
    return mixer.heads if ok else 0


@functools.lru_cache(maxsize=None)
def gqa_decode_supported(mixer, dtype, page_size: int) -> bool:
    """Whether the bf16 kernels for few rows serve the mixer."""
    if dtype != torch.bfloat16:
        return False
    if mixer.shared_keys or mixer.shared_values:
        return bool(get_lib(True).fb_gqa_decode_wide_ok(mixer.key_width, mixer.kv_heads, mixer.vdim_pad, mixer.shared_values,
                                                        mixer.heads, not mixer.shared_keys))
    if mixer.pool or mixer.softcap:
        return False
    return max(mixer.key_width, mixer.vdim_pad) <= 256


def gqa_decode_splits(rows: int, mixer, max_keys: int) -> int:
    """CTAs per row: about two per SM over the batch (one where it takes all kv heads, or wide ones), each with at least 128
    (64) keys of the longest row."""
    most, visible = 8, mixer.chunk or mixer.window + mixer.keep_first
    if mixer.pool:
        visible += max(max_keys - mixer.window, 0) // mixer.pool
    if mixer.shared_keys or mixer.shared_values:
        ctas, fill, least = rows * ((mixer.heads + 15) // 16), 148, 64
        if mixer.shared_values:
            most = 8 // ((mixer.heads + 15) // 16)         # a row's head blocks belong to its cluster
    else:
        ctas = rows * mixer.kv_heads * ((mixer.heads // mixer.kv_heads * mixer.maps + 15) // 16)
        fill, least = 296 if max(mixer.key_width, mixer.vdim_pad) <= 128 else 148, 128
    splits = 1
    while splits * 2 <= most and ctas * splits * 2 <= fill and min(visible, max_keys) >= splits * 2 * least:
        splits *= 2
    return splits


def gqa_decode(q: torch.Tensor, mixer, pool: torch.Tensor, block_table: torch.Tensor, row_seq: torch.Tensor,
               row_pos: torch.Tensor, page_size: int, out: torch.Tensor, splits: int = 1, decode_only: bool = False, **form
               ) -> torch.Tensor:
    """Few query rows, bf16.  decode_only: one row per sequence, every key below its position predates the running step."""
    a = _scaled(_gqa(q, mixer, pool, **form), mixer)
    _gqa_rows(a, block_table, row_seq, row_pos, page_size, out)
    name = "fb_gqa_decode_wide" if mixer.shared_keys or mixer.shared_values else "fb_gqa_decode"
    check(getattr(get_lib(True), name)(C.byref(a), splits, 1 if decode_only else 0, stream_ptr()), name)
    return out


def gqa_prefill_tc(q: torch.Tensor, mixer, pool: torch.Tensor, block_table: torch.Tensor, tiles: torch.Tensor, n_tiles: int,
                   tile_positions: int, page_size: int, out: torch.Tensor, **form) -> torch.Tensor:
    """Prompt rows on tcgen05, bf16: tiles as `kernels.prefill_tiles` makes them; rows no tile covers are left alone."""
    a = _scaled(_gqa(q, mixer, pool, **form), mixer)
    _gqa_rows(a, block_table, None, None, page_size, out)
    assert tiles.dtype == torch.int32 and tiles.shape[1] == 4 and tiles.is_contiguous() and n_tiles <= tiles.shape[0]
    check(get_lib(True).fb_gqa_prefill_tc(C.byref(a), tiles.data_ptr(), n_tiles, tile_positions, stream_ptr()),
          "fb_gqa_prefill_tc")
    return out
