"""Forward pass of layer-list models over a packed ragged batch (paged pool + recurrent-state pool).

Parallel gated blocks:

    x = embed[token]                                             (residual stream, fp32)
    per layer:  h = RMSNorm(x) * g
                x += sigmoid(rg1 h + b1) * mixer(h) + sigmoid(rg2 h + b2) * ff(h)
    logits = softcap(head . RMSNorm(x) * g_final)

Output-norm blocks:

    x = embed[token] + pos[position]
    per layer:  x += norm1(mixer(x + conv(x)))                   (conv: short causal convolution, one filter per channel)
                x += norm2(ff(x))
    logits = head . norm_final(x)

Sandwich blocks (every norm an RMS norm in groups):

    x = embed[token]
    per run:    x += embed[token]                                (first layer of every later pass of a loop)
                x += norm1b(mixer(norm1(x)))
                x += norm2b(ff(norm2(x)))
    logits = head . norm_final(x)

Pre-norm blocks:

    x = embed[token] * embed_scale
    per layer:  x += mixer(shift(norm1(x)))                      (shift: h + (h of the previous token - h) * s)
                x += ff(norm2(x))
    logits = head . norm_final(x)

A layer that runs several times has a cache plane and a state per run.

* `LayeredReference` - plain PyTorch; the execution path of a CPU runner.
* `LayeredCuda`      - the sm_100a kernel pipeline, allocation-free over a preallocated workspace, so a decode step can be
  captured in a CUDA graph.  With fp32 weights the same pipeline runs in full 32 bits.

Kernels of a latent layer: input projection (one GEMM for q, latent, gates) -> latent append -> W_uk absorption ->
attention over the latent pool (head gate in its epilogue) -> W_uv -> W_o; with a query latent the append also normalises it
and W_uq follows, with rotated parts their queries join behind the absorption.  Of an attention layer: input projection (q, k,
v) -> norms, rotation, value mixing and cache append in one launch -> attention -> W_o.  Of a window layer: input projection
(q, k, v, gate) -> norms, mixing of the queries across heads and cache append in one launch -> attention (distance bias,
difference of the two maps, soft cap, gate inside) -> W_o; with pooled blocks their mean rows are written in front of the
attention (in decode steps by the append), and outputs whose softmax weights are mixed across heads are mixed behind the prompt
attention (in decode steps inside).  Of a delta layer: input projection -> second low-rank halves -> delta rule -> W_o.  Of a selective-scan layer: input projection -> convolution -> W_x -> W_dt
-> scan (step sizes, skip and output gate inside) -> W_o.  Of a head-decay scan: input projection -> convolution -> scan (step
sizes, skip and output gate inside) -> group norm -> W_o.

In a parallel gated block the feed-forward branch reads the same h and runs on a second stream beside the mixer: router
(+ row reservation) -> grouped SwiGLU GEMM -> grouped scatter GEMM.  One kernel joins both branches: gated residual
additions, expert reduction, next layer's norm.  In an output-norm block one kernel after each sublayer normalises its
output, adds it to the stream and leaves the rows the next GEMM reads; in decode steps it also applies the next mixer's
input convolution, whose earlier inputs are in the state pool then.  In a sandwich block the same kernel takes the norm of the
sublayer's output, the addition, the embedding of a new pass and the next sublayer's input norm.  In a pre-norm block it adds
the output (a token's expert rows and its gated shared expert), takes the next norm and the token shift; when rows have their
predecessors in the same batch it writes the stream to a second buffer.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch
import torch.nn.functional as F

from ..ops import reference as ref
from .config import SCORE_SOFTMAX
from .deepseek import DeviceBatch, KvPool, _pow2_at_least
from .layered_config import (OUTPUT_NORM, PARALLEL_GATED, PRE_NORM, SANDWICH_NORM, AttentionMixer, DeltaMixer, LatentMixer,
                             Mamba2Mixer, MambaMixer, MoeSpec, WindowMixer, pad_to)
from .layered_weights import LayerImage, LayeredWeights, MixerImage
from .state_pool import RecurrentStatePool


def rotation_frequencies(base: float, dims: int) -> torch.Tensor:
    """Angle per position of every rotated pair of a head (double)."""
    return base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))


# ======================================================================================
# reference forward (PyTorch)
# ======================================================================================
class LayeredReference:
    def __init__(self, weights: LayeredWeights, pool: KvPool, states: RecurrentStatePool):
        self.w, self.cfg, self.pool, self.states = weights, weights.cfg, pool, states
        self.cache_index = {r: i for i, r in enumerate(self.cfg.cache_runs)}
        self.prof = self.tap = None

    def _norm(self, x: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
        W = self.cfg.width
        inv = torch.rsqrt(x[:, :W].pow(2).mean(-1, keepdim=True) + self.cfg.norm_eps)
        return x * inv * g

    def _latent(self, layer: int, mx: MixerImage, m: LatentMixer, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        T, DL, R, eps = proj.shape[0], m.row_dim, m.rot_dim, self.cfg.norm_eps
        o = mx.off
        dp, vp = pad_to(m.dim, 8), pad_to(m.vdim, 8)
        q_src, q_off = proj, o
        if m.q_rank:
            cq = proj[:, o["dq"]:o["dq"] + m.q_rank]
            cq = cq * torch.rsqrt(cq.pow(2).mean(-1, keepdim=True) + eps) * mx.dq_norm[:m.q_rank]
            q_src, q_off = cq @ mx.w_uq[:, :m.q_rank].float().T, mx.off_uq
        q = q_src[:, q_off["q"]:q_off["q"] + m.heads * dp].view(T, m.heads, dp)
        c = proj[:, o["dkv"]:o["dkv"] + m.kv_rank]
        c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * mx.kv_norm[:m.kv_rank]
        pool = self.pool.layer(self.cache_index[layer]).view(-1, DL)
        row = torch.zeros(T, DL)
        row[:, :m.kv_rank] = c
        q_lat = torch.einsum("thk,hnk->thn", q, mx.w_uk_t.float())
        if R:
            a = b.positions[:T].double()[:, None] * rotation_frequencies(m.rot_base, R)
            cs, sn = torch.cos(a).float()[:, None], torch.sin(a).float()[:, None]

            def turn(t):
                u, w = t[..., 0::2], t[..., 1::2]
                return torch.stack([u * cs - w * sn, w * cs + u * sn], -1).flatten(-2)

            at = slice(m.rot_offset, m.rot_offset + R)
            row[:, at] = turn(proj[:, None, o["dkv"] + m.kv_rank:o["dkv"] + m.kv_rank + R])[:, 0]
            q_lat[:, :, at] = turn(q_src[:, q_off["qr"]:q_off["qr"] + m.heads * R].view(T, m.heads, R))
        slots = b.write_slot[:T]
        ok = slots >= 0
        pool[slots[ok]] = row[ok].to(pool.dtype)
        if m.window:
            lat = torch.zeros(T, m.heads, DL)
            for r in range(T):
                p, seq, ps = int(b.row_pos[r]), int(b.row_seq[r]), self.pool.page_size
                t = torch.arange(max(p - m.window + 1, 0), p + 1)
                if t.numel():
                    kv = pool[b.block_table[seq, t // ps].long() * ps + t % ps].float()
                    lat[r] = torch.softmax(q_lat[r] @ kv.T * m.scale, -1) @ kv
        else:
            lat = ref.mla_paged_attention(q_lat, pool, b.block_table, b.row_seq[:T], b.row_pos[:T], self.pool.page_size, DL,
                                          m.scale)
        v = torch.einsum("thn,hvn->thv", lat, mx.w_uv.float())
        gate = torch.sigmoid(proj[:, o["g"]:o["g"] + m.heads])
        return (v * gate[:, :, None]).reshape(T, m.heads * vp) @ mx.w_o.float().T

    def _delta(self, layer: int, mx: MixerImage, m, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        T, o = proj.shape[0], mx.off
        H, KV, D, V = m.heads, m.kv_heads, m.dim, m.vdim
        nk, nv, keep = KV * D, H * V, m.taps - 1
        nd = H if m.head_decay else H * D
        if m.low_rank:
            ag = proj[:, o["a1"]:o["a1"] + mx.w_ag.shape[1]] @ mx.w_ag.float().T
            pre, gate = ag[:, :nd], ag[:, mx.off_gate:mx.off_gate + nv]
        else:
            pre, gate = proj[:, o["a"]:o["a"] + nd], proj[:, o["g"]:o["g"] + nv]
        gate = torch.sigmoid(gate) if m.gate == "sigmoid" else F.silu(gate)
        raw = torch.cat([proj[:, o["q"]:o["q"] + nk], proj[:, o["k"]:o["k"] + nk], proj[:, o["v"]:o["v"] + nv]], 1)
        decay = torch.exp(mx.a_neg[:, None] * F.softplus(pre + mx.dt_bias).view(T, H, nd // H))
        beta = torch.sigmoid(proj[:, o["b"]:o["b"] + H])
        state, tail = self.states.state[layer], self.states.tail[layer]
        out = torch.zeros(T, mx.w_o.shape[1])
        for s in range(b.n_seqs):
            r0, r1 = int(b.seq_start[s]), int(b.seq_start[s + 1])
            sin, sout = int(b.state_in[s]), int(b.state_out[s])
            old = tail[sin, :keep].float() if (sin >= 0 and keep) else torch.zeros(keep, m.channels)
            S = state[sin].clone() if sin >= 0 else torch.zeros(H, D, V)
            x = torch.cat([old, raw[r0:r1]], 0)
            n = r1 - r0
            y = sum(x[j:j + n] * mx.conv[j] for j in range(m.taps))
            y = F.silu(y)
            q, k, v = y[:, :nk].view(n, KV, D), y[:, nk:2 * nk].view(n, KV, D), y[:, 2 * nk:].view(n, H, V)
            unit = lambda t: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
            q = (unit(q) * D ** -0.5).repeat_interleave(H // KV, 1)
            k = unit(k).repeat_interleave(H // KV, 1)
            for i in range(n):
                S = S * decay[r0 + i][:, :, None]
                u = beta[r0 + i][:, None] * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
                S = S + k[i][:, :, None] * u[:, None, :]
                oi = torch.einsum("hdv,hd->hv", S, q[i])
                oi = oi * torch.rsqrt(oi.pow(2).mean(-1, keepdim=True) + self.cfg.norm_eps) * mx.o_norm
                out[r0 + i, :nv] = (oi * gate[r0 + i].view(H, V)).reshape(-1)
            if sout >= 0:
                state[sout] = S
                if keep:
                    tail[sout, :keep] = x[-keep:].to(tail.dtype)
        return out @ mx.w_o.float().T

    @staticmethod
    def _expert(s: MoeSpec, limit: float, x: torch.Tensor, w13: torch.Tensor, w2: torch.Tensor) -> torch.Tensor:
        g, u = (x @ w13.float().T).chunk(2, -1)
        if limit:
            g, u = g.clamp(max=limit), u.clamp(-limit, limit)
        return (g * torch.sigmoid(s.alpha * g) * (u + s.shift)) @ w2.float().T

    def _moe(self, lw: LayerImage, h: torch.Tensor) -> torch.Tensor:
        s = lw.spec.mlp
        z = h @ lw.router_w.float().T
        logits = z[:, :s.experts] if lw.router_b is None else z[:, :s.experts] + lw.router_b
        idx, wts = ref.route(logits, s.top, SCORE_SOFTMAX, n_groups=s.groups, topk_groups=s.keep, normalize=s.renormalize,
                             group_top=1)
        out = torch.zeros_like(h)
        for e in range(s.experts):
            hit = idx == e
            rows = hit.any(-1).nonzero().flatten()
            if rows.numel() == 0:
                continue
            out[rows] += self._expert(s, s.limit, h[rows], lw.e_w13[e], lw.e_w2[e]) * (wts * hit)[rows].sum(-1, keepdim=True)
        if s.shared_ff:
            out += torch.sigmoid(z[:, s.experts:]) * self._expert(s, s.shared_limit, h, lw.s_w13, lw.s_w2)
        return out

    def _conv(self, x: torch.Tensor, w: torch.Tensor, tail: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        """Causal convolution of packed rows x [T, channels] with w [taps, channels]; inputs before a sequence's first
        row come from its state, which is brought up to date."""
        keep, out = w.shape[0] - 1, torch.empty_like(x)
        for s in range(b.n_seqs):
            r0, r1 = int(b.seq_start[s]), int(b.seq_start[s + 1])
            sin, sout = int(b.state_in[s]), int(b.state_out[s])
            old = tail[sin, :keep].float() if (sin >= 0 and keep) else torch.zeros(keep, x.shape[1])
            xs = torch.cat([old, x[r0:r1]], 0)
            out[r0:r1] = sum(xs[j:j + r1 - r0] * w[j] for j in range(keep + 1))
            if sout >= 0 and keep:
                tail[sout, :keep] = xs[-keep:].to(tail.dtype)
        return out

    def _attention(self, layer: int, mx: MixerImage, m: AttentionMixer, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        T, o, eps = proj.shape[0], mx.off, self.cfg.norm_eps
        H, G, D, V, dp, vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_pad, m.vdim_pad
        part = lambda name, heads, pad, d: proj[:, o[name]:o[name] + heads * pad].view(T, heads, pad)[:, :, :d]
        rms = lambda t, dims: t * torch.rsqrt(t.pow(2).mean(dims, keepdim=True) + eps)
        q = rms(part("q", H, dp, D), (1, 2)) * mx.q_norm.view(H, dp)[:, :D]
        k = rms(part("k", G, dp, D), (1, 2)) * mx.k_norm.view(G, dp)[:, :D]
        v = rms(part("v", G, vp, V), (2,))
        half = m.rot_dims // 2
        a = b.positions[:T].double()[:, None] * rotation_frequencies(m.rot_base, m.rot_dims)
        c, sn = torch.cos(a).float()[:, None], torch.sin(a).float()[:, None]

        def turn(t):
            u, w = t[:, :, :half], t[:, :, half:2 * half]
            return torch.cat([u * c - w * sn, w * c + u * sn, t[:, :, 2 * half:]], -1)

        slots = b.write_slot[:T]
        ok = slots >= 0
        rows = self.pool.layer(self.cache_index[layer]).view(-1, self.cfg.kv_row_dim)
        first = self.cfg.first_value_layer
        if m.v_mix and layer != first:
            fm = self.cfg.layers[first].mixer
            fv = self.pool.layer(self.cache_index[first]).view(-1, self.cfg.kv_row_dim)[slots.clamp(min=0)]
            fv = fv[:, fm.v_offset:fm.v_offset + G * vp].view(T, G, vp)[:, :, :V].float()
            v = (1 - mx.v_mix) * v + mx.v_mix * fv
        row = torch.zeros(T, rows.shape[1])
        row[:, :m.v_offset].view(T, G, dp)[:, :, :D] = turn(k)
        row[:, m.v_offset:m.v_offset + G * vp].view(T, G, vp)[:, :, :V] = v
        rows[slots[ok]] = row[ok].to(rows.dtype)
        q, out, ps = turn(q), torch.zeros(T, H, vp), self.pool.page_size
        for r in range(T):
            p, seq = int(b.row_pos[r]), int(b.row_seq[r])
            t = torch.arange(max(p, 0) // m.chunk * m.chunk, p + 1)
            if t.numel() == 0:
                continue
            kv = rows[b.block_table[seq, t // ps].long() * ps + t % ps].float()
            k = kv[:, :m.v_offset].view(-1, G, dp)[:, :, :D]
            v = kv[:, m.v_offset:m.v_offset + G * vp].view(-1, G, vp)
            w = torch.softmax(torch.einsum("ghd,tgd->ght", q[r].view(G, H // G, D), k) * m.scale, -1)
            out[r] = torch.einsum("ght,tgv->ghv", w, v).reshape(H, vp)
        return out.view(T, H * vp) @ mx.w_o.float().T

    def _window(self, run: int, mx: MixerImage, m: WindowMixer, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        T, o, eps = proj.shape[0], mx.off, self.cfg.norm_eps
        H, G, M, D, V, dp, vp = m.heads, m.kv_heads, m.maps, m.dim, m.vdim, m.dim_pad, m.vdim_pad
        part = lambda name, heads, pad: proj[:, o[name]:o[name] + heads * pad]
        rms = lambda t, n: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) / n + eps)
        q, k = part("q", H * M, dp), part("k", G * M, dp)
        if mx.q_bias is not None:
            q, k = q + mx.q_bias, k + mx.k_bias
        v = k if m.tied_values else part("v", G, vp)
        q, k = q.reshape(T, H, M, dp), k.reshape(T, G * M, dp)
        if m.rot_dims:
            half = m.rot_dims // 2
            a = b.positions[:T].double()[:, None] * rotation_frequencies(m.rot_base, m.rot_dims)
            cs, sn = torch.cos(a).float(), torch.sin(a).float()

            def turn(t):
                u, w = t[..., :half], t[..., half:2 * half]
                c_, s_ = (x.view(T, *[1] * (t.dim() - 2), half) for x in (cs, sn))
                return torch.cat([u * c_ - w * s_, w * c_ + u * s_, t[..., 2 * half:]], -1)

            q, k = turn(q), turn(k)
        q, k = rms(q, D), rms(k, D)
        if m.norm_weights:
            q, k = q * mx.q_norm, k * mx.k_norm
        rows = self.pool.layer(self.cache_index[run])
        rows = rows.view(-1, rows.shape[-1])
        row = torch.zeros(T, rows.shape[1])
        row[:, :m.v_offset] = k.view(T, -1)
        row[:, m.v_offset:m.v_offset + G * vp] = v
        slots = b.write_slot[:T]
        ok = slots >= 0
        rows[slots[ok]] = row[ok].to(rows.dtype)
        out, ps = torch.zeros(T, H, vp), self.pool.page_size
        at = lambda seq, t: rows[b.block_table[seq, t // ps].long() * ps + t % ps].float()
        pooled = None
        if m.pool:
            for r in range(T):
                p, seq = int(b.row_pos[r]), int(b.row_seq[r])
                if (p + 1) % m.pool == 0 and p >= 0:
                    self.states.pooled[run][int(b.state_out[seq]) // self.states.buffers, p // m.pool] = (
                        at(seq, torch.arange(p + 1 - m.pool, p + 1)).mean(0).to(rows.dtype))
        for r in range(T):
            p, seq = int(b.row_pos[r]), int(b.row_seq[r])
            first = max(p - m.window + 1, 0)
            t = torch.cat([torch.arange(min(m.keep_first, first)), torch.arange(first, p + 1)])
            if t.numel() == 0:
                continue
            kv = at(seq, t)
            if m.pool:
                blocks = max(p - m.window + 1, 0) // m.pool
                pooled = self.states.pooled[run][int(b.state_out[seq]) // self.states.buffers, :blocks]
                kv = torch.cat([pooled.float(), kv])
            k = kv[:, :m.v_offset].view(-1, G, M, dp).repeat_interleave(H // G, 1)
            v = kv[:, m.v_offset:m.v_offset + G * vp].view(-1, G, vp).repeat_interleave(H // G, 1)
            s = torch.einsum("hmd,thmd->hmt", q[r], k)
            s = torch.einsum("hg,gmt->hmt", mx.q_mix, s) if m.mix_heads else s * mx.q_mix[:, None, None]
            if m.distance_bias:
                s = s - (mx.slopes[:, None] * (p - t))[:, None]
            if m.softcap:
                s = m.softcap * torch.tanh(s / m.softcap)
            s = torch.softmax(s, -1)
            if m.mix_weights:
                s = torch.einsum("hg,gmt->hmt", mx.talk, s)
            a = torch.einsum("hmt,thv->hmv", s, v)
            out[r] = a[:, 0] if M == 1 else rms(a[:, 0] - mx.diff_lambda * a[:, 1], V) * (1 - m.diff)
        if m.gate:
            out = out * torch.sigmoid(part("g", H, vp).reshape(T, H, vp))
        y = out.view(T, H * vp) @ mx.w_o.float().T
        return y if mx.o_bias is None else y + mx.o_bias

    def _mamba(self, layer: int, mx: MixerImage, m: MambaMixer, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        o, Ip, N = mx.off, m.inner_pad, m.state
        x = F.silu(self._conv(proj[:, o["x"]:o["x"] + Ip], mx.conv, self.states.tail[layer], b) + mx.conv_b)
        low = x @ mx.w_x.float().T
        dt = F.softplus(low[:, :mx.w_dt.shape[1]] @ mx.w_dt.float().T + mx.dt_bias)
        B, C = low[:, mx.off_b:mx.off_b + N], low[:, mx.off_c:mx.off_c + N]
        state, y = self.states.state[layer], torch.empty_like(x)
        for s in range(b.n_seqs):
            sin, sout = int(b.state_in[s]), int(b.state_out[s])
            S = state[sin].clone() if sin >= 0 else torch.zeros(N, Ip)
            for r in range(int(b.seq_start[s]), int(b.seq_start[s + 1])):
                S = torch.exp2(dt[r] * mx.a_log2) * S + B[r][:, None] * (dt[r] * x[r])
                y[r] = C[r] @ S + mx.d_skip * x[r]
            if sout >= 0:
                state[sout] = S
        return (y * F.silu(proj[:, o["z"]:o["z"] + Ip])) @ mx.w_o.float().T

    def _mamba2(self, layer: int, mx: MixerImage, m: Mamba2Mixer, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        o, H, V, N, G, I, T = mx.off, m.heads, m.vdim, m.state, m.groups, m.inner, proj.shape[0]
        xbc = F.silu(self._conv(proj[:, :m.channels], mx.conv, self.states.tail[layer], b) + mx.conv_b)
        x = xbc[:, :I].view(T, H, V)
        B, C = (xbc[:, at:at + G * N].view(T, G, N).repeat_interleave(H // G, 1) for at in (mx.off_b, mx.off_c))
        dt = F.softplus(proj[:, o["dt"]:o["dt"] + H] + mx.dt_bias)
        decay = torch.exp(mx.a_neg * dt)
        state, y = self.states.state[layer], torch.zeros(T, m.inner_pad)
        for s in range(b.n_seqs):
            sin, sout = int(b.state_in[s]), int(b.state_out[s])
            S = state[sin].clone() if sin >= 0 else torch.zeros(H, N, V)
            for r in range(int(b.seq_start[s]), int(b.seq_start[s + 1])):
                S = decay[r][:, None, None] * S + B[r][:, :, None] * (dt[r][:, None] * x[r])[:, None]
                y[r, :I] = (torch.einsum("hn,hnv->hv", C[r], S) + mx.d_skip[:, None] * x[r]).flatten()
            if sout >= 0:
                state[sout] = S
        y = (y * F.silu(proj[:, o["z"]:o["z"] + m.inner_pad]))[:, :I].view(T, m.norm_groups, -1)
        y = (y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + self.cfg.norm_eps)).view(T, I) * mx.o_norm[:I]
        return y @ mx.w_o[:, :I].float().T

    def _mixer(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        m = lw.spec.mixer
        fn = {LatentMixer: self._latent, AttentionMixer: self._attention, WindowMixer: self._window,
              DeltaMixer: self._delta, MambaMixer: self._mamba, Mamba2Mixer: self._mamba2}[type(m)]
        return fn(layer, lw.mixer, m, proj, b)

    def _gated_layer(self, i: int, lw: LayerImage, x: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        Wp, mx = self.cfg.width_pad, lw.mixer
        h = self._norm(x, lw.norm)
        proj = h @ mx.w_in.float().T
        y = self._mixer(i, lw, proj, b)
        y = y * torch.sigmoid(proj[:, mx.off["rg1"]:mx.off["rg1"] + Wp] + lw.rg1_b)
        if lw.spec.mlp is not None:
            y = y + self._moe(lw, h) * torch.sigmoid(proj[:, mx.off["rg2"]:mx.off["rg2"] + Wp] + lw.rg2_b)
        return x + y

    def _layer_norm(self, x: torch.Tensor, wb: torch.Tensor) -> torch.Tensor:
        W, out = self.cfg.width, torch.zeros_like(x)
        out[:, :W] = F.layer_norm(x[:, :W], (W,), wb[0, :W], wb[1, :W], self.cfg.norm_eps)
        return out

    def _output_norm_layer(self, i: int, lw: LayerImage, x: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        h = x + self._conv(x, lw.canon, self.states.canon[i], b) if lw.canon is not None else x
        x = x + self._layer_norm(self._mixer(i, lw, h @ lw.mixer.w_in.float().T, b), lw.norm1)
        if lw.spec.mlp is not None:
            x = x + self._layer_norm(F.gelu(x @ lw.w_up.float().T) @ lw.w_down.float().T, lw.norm2)
        return x

    def _group_norm(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        W, out = self.cfg.width, torch.zeros_like(x)
        parts = x[:, :W].unflatten(1, (self.cfg.norm_groups, -1))
        out[:, :W] = (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + self.cfg.norm_eps)).flatten(1) * w[:W]
        return out

    def _sandwich_layer(self, i: int, lw: LayerImage, x: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        norm = self._group_norm
        x = x + norm(self._mixer(i, lw, norm(x, lw.norm1) @ lw.mixer.w_in.float().T, b), lw.norm1b)
        if lw.spec.mlp is not None:
            g, u = (norm(x, lw.norm2) @ lw.w_up.float().T).chunk(2, -1)
            x = x + norm((F.gelu(g, approximate="tanh") * u) @ lw.w_down.float().T, lw.norm2b)
        return x

    def _shift(self, h: torch.Tensor, s: torch.Tensor, plane: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        """Rows moved towards their sequence's previous row, which the state plane holds for the first one."""
        before = torch.zeros_like(h)
        for q in range(b.n_seqs):
            r0, r1 = int(b.seq_start[q]), int(b.seq_start[q + 1])
            sin, sout = int(b.state_in[q]), int(b.state_out[q])
            if sin >= 0:
                before[r0] = plane[sin]
            before[r0 + 1:r1] = h[r0:r1 - 1]
            if sout >= 0:
                plane[sout] = h[r1 - 1]
        return h + (before - h) * s

    def _pre_norm_layer(self, i: int, lw: LayerImage, x: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        mx = lw.mixer
        h = self._norm(x, lw.norm1)
        if lw.shift is not None:
            h = self._shift(h, lw.shift, self.states.shift[i], b)
        proj = h @ mx.w_in.float().T
        x = x + self._mixer(i, lw, proj if mx.b_in is None else proj + mx.b_in, b)
        if isinstance(lw.spec.mlp, MoeSpec):
            x = x + self._moe(lw, self._norm(x, lw.norm2))
        elif lw.spec.mlp is not None:
            u = self._norm(x, lw.norm2) @ lw.w_up.float().T
            y = F.gelu(u if lw.up_b is None else u + lw.up_b) @ lw.w_down.float().T
            x = x + (y if lw.down_b is None else y + lw.down_b)
        return x

    def hidden_states(self, b: DeviceBatch, allreduce=None, start_layer: int = 0, h0=None) -> torch.Tensor:
        """Residual stream after the last layer [rows, width_pad]."""
        x = embedded = self.w.embed[b.token_ids[:b.n_rows].long()].float()
        if self.cfg.embed_scale != 1.0:
            x = x * self.cfg.embed_scale
        if self.w.pos is not None:
            x = x + self.w.pos[b.positions[:b.n_rows].long()].float()
        layer = {PARALLEL_GATED: self._gated_layer, OUTPUT_NORM: self._output_norm_layer,
                 SANDWICH_NORM: self._sandwich_layer, PRE_NORM: self._pre_norm_layer}[self.cfg.block]
        for i, l in enumerate(self.cfg.runs):
            if self.prof is not None:
                self.prof.mark(i, "layer")
            if i in self.cfg.pass_starts:
                x = x + embedded
            x = layer(i, self.w.layers[l], x, b)
            if self.tap is not None:
                self.tap.write(i, "layer_out", x)
        return x

    def logits_from_hidden(self, x: torch.Tensor, b: DeviceBatch) -> torch.Tensor:
        norm = {PARALLEL_GATED: self._norm, OUTPUT_NORM: self._layer_norm, SANDWICH_NORM: self._group_norm,
                PRE_NORM: self._norm}[self.cfg.block]
        logits = norm(x[b.logit_rows[:b.n_logit].long()], self.w.final_norm) @ self.w.lm_head.float().T
        cap = self.cfg.logit_softcap
        return cap * torch.tanh(logits / cap) if cap else logits


# ======================================================================================
# CUDA forward (sm_100a kernels)
# ======================================================================================
class LayeredWorkspace:
    """Preallocated activations for up to `max_rows` packed rows."""

    def __init__(self, w: LayeredWeights, max_rows: int, max_logit_rows: int, device):
        from ..ops import layered as KL
        from ..ops.kernels import ArgmaxScratch, MoePlan, static_plan
        cfg = w.cfg
        dt = w.embed.dtype
        act = dict(dtype=dt, device=device)
        f32 = dict(dtype=torch.float32, device=device)
        i32 = dict(dtype=torch.int32, device=device)
        R, Wp = max_rows, cfg.width_pad
        self.max_rows, self.max_logit_rows = R, max_logit_rows
        self.x = torch.zeros(R, Wp, **f32)
        if cfg.token_shift:
            self.x_next = torch.zeros(R, Wp, **f32)
        self.h = torch.zeros(R, Wp, **act)
        self.proj = torch.zeros(R * max(l.mixer.w_in.shape[0] for l in w.layers), **act)
        self.mix_in = torch.zeros(R * max(l.mixer.w_o.shape[1] for l in w.layers), **act)
        self.mix = torch.zeros(R, Wp, **act)
        latent, delta, mamba = ([cfg.layers[i].mixer for i in ids] for ids in (cfg.latent_layers, cfg.delta_layers,
                                                                               cfg.mamba_layers))
        if latent:
            n = max(m.heads * m.row_dim for m in latent)
            self.q_lat = torch.zeros(R * n, **act)
            self.o_lat = torch.zeros(R * n, **act)
            self.uq = torch.zeros(R * max((l.mixer.w_uq.shape[0] for l in w.layers if l.mixer.w_uq is not None), default=0), **act)
        if delta:
            low = [l.mixer.w_ag for l in w.layers if l.mixer.w_ag is not None]
            self.ag = torch.zeros(R * max((t.shape[0] for t in low), default=0), **f32)
            self.delta = KL.DeltaScratch(R, delta, device)
        if mamba:
            n = max(m.inner_pad for m in mamba)
            self.conv_x = torch.zeros(R * n, **act)
            self.dt = torch.zeros(R * n, **f32)
            self.low = torch.zeros(R * max(l.mixer.w_x.shape[0] for l in w.layers if l.mixer.w_x is not None), **act)
        head_scan = [cfg.layers[i].mixer for i in cfg.mamba2_layers]
        if head_scan:
            self.conv_x = torch.zeros(R * max([m.channels for m in head_scan] + [m.inner_pad for m in mamba]), **act)
        window = [cfg.layers[i].mixer for i in cfg.window_layers]
        if window:
            # (queries that are neither mixed nor split into maps stay in the projection's rows)
            self.q_rows = torch.zeros(R * max((m.heads * m.maps * m.key_width for m in window if m.shared_keys or m.maps > 1),
                                              default=0), **act)
            self.o_all = torch.zeros(R * max((m.heads * m.value_width for m in window if m.shared_values), default=0), **act)
        if any(l.w_up is not None for l in w.layers):
            self.ff = torch.zeros(R * max(l.w_down.shape[1] for l in w.layers if l.w_up is not None), **act)
            if cfg.block == OUTPUT_NORM:
                self.act = torch.zeros(R, Wp, **act)
        moes = [(i, l.mlp) for i, l in enumerate(cfg.layers) if isinstance(l.mlp, MoeSpec)]
        self.plans: Dict[tuple, MoePlan] = {}
        self.static_plans: Dict[tuple, MoePlan] = {}
        self.static_rows = (16, 32, 64)
        if moes:
            kmax, emax = max(s.top for _, s in moes), max(s.experts for _, s in moes)
            self.router_logits = torch.zeros(R * (emax + 1), **f32)
            sff = [l.s_w2.shape[1] for l in w.layers if l.s_w2 is not None]
            if sff:
                self.shared_mid = torch.zeros(R * max(sff), **act)
                self.shared_out = torch.zeros(R, Wp, **act)
                self.shared_gate = torch.zeros(R, 1, **f32)
            self.topk_idx = torch.zeros(R * kmax, **i32)
            self.topk_w = torch.zeros(R * kmax, **f32)
            xrows = max(R * kmax, emax * self.static_rows[-1])
            self.xg = torch.zeros(xrows, Wp, **act)
            self.hmid = torch.zeros(xrows * max(l.e_w2.shape[2] for l in w.layers if l.e_w2 is not None), **act)
            self.route_out = torch.zeros(R * kmax, Wp, **act)
            self.route_cnt = torch.zeros(cfg.n_layers, emax, **i32)
            for E, k in sorted({(s.experts, s.top) for _, s in moes}):
                for ntok in (16, 32, 64, 128):
                    self.plans[E, k, ntok] = MoePlan.allocate(R * k, E, ntok, device)
                self.plans[E, k, 256] = None                        # tile table of the scatter GEMM, built on first use
            base: Dict[tuple, MoePlan] = {}
            for i, s in moes:
                for nt in self.static_rows:
                    p = static_plan(nt, s.experts, self.route_cnt[i][:s.experts], base.get((s.experts, nt)))
                    base.setdefault((s.experts, nt), p)
                    self.static_plans[i, nt] = p
        L = max_logit_rows
        self.hn_last = torch.zeros(L, Wp, **act)
        self.logits = torch.zeros(L, pad_to(cfg.vocab_size, 4), **f32)[:, :cfg.vocab_size]     # 16-byte aligned rows
        self.out_buf = torch.zeros(2 * L, **i32)          # greedy result: [ids | fp32 value bits]
        self.next_id = self.out_buf[:L]
        self.next_val = self.out_buf[L:].view(torch.float32)
        self.argmax_scratch = ArgmaxScratch.allocate(max(L, 1), device)


class LayeredCuda:
    def __init__(self, weights: LayeredWeights, pool: KvPool, states: RecurrentStatePool, max_rows: int = 4096,
                 max_logit_rows: int = 256, decode_rows: int = 64, max_seq_len: int = 4096, attn_splits: int = 8):
        from ..ops import kernels as K
        from ..ops import layered as KL
        from ..ops import movers as M
        self.K, self.KL, self.M = K, KL, M
        self.w, self.cfg, self.pool, self.states = weights, weights.cfg, pool, states
        self.device = weights.embed.device
        self.fp32 = weights.embed.dtype == torch.float32
        self.decode_rows = decode_rows
        self.attn_splits = attn_splits
        self.max_seq_len = max_seq_len
        self.ws = LayeredWorkspace(weights, max_rows, max_logit_rows, self.device)
        self.cache_index = {r: i for i, r in enumerate(self.cfg.cache_runs)}
        self.gqa_table = max((KL.gqa_tc_group(self.cfg.layers[i].mixer, weights.embed.dtype, pool.page_size)
                              for i in self.cfg.attention_layers + self.cfg.window_layers), default=0)
        # cosines and sines of every rotation in use, computed in double
        self.rotation: Dict[tuple, tuple] = {}
        for l in self.cfg.layers:
            base, dims = self._rotation_key(l.mixer)
            if dims and (base, dims) not in self.rotation:
                a = (torch.arange(min(max_seq_len, self.cfg.max_position), dtype=torch.float64)[:, None]
                     * rotation_frequencies(base, dims))
                self.rotation[base, dims] = tuple(f(a).float().to(self.device) for f in (torch.cos, torch.sin))
        self.static_moe = not self.fp32 and self.cfg.width_pad <= 8192
        self.side_stream = torch.cuda.Stream(device=self.device)      # the feed-forward runs beside the mixer
        self.launches = 0
        self.last_hidden = None
        self.prof = self.tap = None
        for l in self.cfg.layers:
            m, f = l.mixer, l.mlp
            if isinstance(m, DeltaMixer) and m.dim > 256:
                raise ValueError("delta mixers wider than 256 key channels per head are not supported")
            if isinstance(m, MambaMixer) and m.state > 128:
                raise ValueError("selective scans with more than 128 states per channel are not supported")
            if isinstance(m, Mamba2Mixer) and (m.state > 256 or m.vdim > 1024):
                raise ValueError("head-decay scans with more than 256 states or 1024 columns per head are not supported")
            if isinstance(m, (AttentionMixer, WindowMixer)) and max(m.dim, m.vdim) > 512:
                raise ValueError("attention heads wider than 512 are not supported")
            if isinstance(f, MoeSpec) and (f.experts > 256 or f.top > 32 or f.groups > 32):
                raise ValueError("the router takes at most 256 experts, top 32, 32 groups")

    @staticmethod
    def _rotation_key(m) -> tuple:
        dims = m.rot_dim if isinstance(m, LatentMixer) else getattr(m, "rot_dims", 0)
        return (m.rot_base, dims) if dims else (0.0, 0)

    @staticmethod
    def _view(buf: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
        return buf[:rows * cols].view(rows, cols)

    # -- mixers ---------------------------------------------------------------------------
    def _latent(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        K, KL, ws, cfg = self.K, self.KL, self.ws, self.cfg
        mx, m = lw.mixer, lw.spec.mixer
        DL, dp, vp = m.row_dim, pad_to(m.dim, 8), pad_to(m.vdim, 8)
        pool = self.pool.layer(self.cache_index[layer])
        rotation = self.rotation.get(self._rotation_key(m))
        q_src, q_off = proj, mx.off
        if m.q_rank or m.rot_dim:
            KL.latent_prep(proj, mx.off, m, mx, rotation, b.positions[:T], b.write_slot[:T], pool, cfg.norm_eps)
        else:
            KL.latent_append(proj[:, mx.off["dkv"]:], m.kv_rank, mx.kv_norm, cfg.norm_eps, b.write_slot[:T], pool)
        if m.q_rank:
            q_src, q_off = self._view(ws.uq, T, mx.w_uq.shape[0]), mx.off_uq
            K.gemm(proj[:, mx.off["dq"]:mx.off["dq"] + mx.w_uq.shape[1]], mx.w_uq, out=q_src)
        q = q_src[:, q_off["q"]:q_off["q"] + m.heads * dp]
        q_lat = self._view(ws.q_lat, T, m.heads * DL)
        K.gemm(q, mx.w_uk_t, out=q_lat, x_group_koff=dp, out_group_coff=DL, k=dp)
        q3 = q_lat.view(T, m.heads, DL)
        if m.rot_dim:
            KL.latent_turn(q_src[:, q_off["qr"]:q_off["qr"] + m.heads * m.rot_dim], m, rotation, b.positions[:T], q3)
        gate = proj[:, mx.off["g"]:]
        # the tensor-core attention kernels take values up to 512 features
        mma = not self.fp32 and m.value_dim <= 512
        D = m.value_dim if mma else DL
        o_lat = self._view(ws.o_lat, T, m.heads * D)
        o3 = o_lat.view(T, m.heads, D)
        if not mma:
            KL.latent_attention(q3, pool, b.block_table, b.row_seq[:T], b.row_pos[:T], self.pool.page_size, m.scale, o3,
                                gate=gate, window=m.window)
        else:
            ranges, rope = [(0, T)], DL - D
            tiles = b.tc_tables.get(KL.latent_tc_group(m, q3.dtype, self.pool.page_size)) if b.n_tc_tiles else None
            if tiles:
                # sequences with many rows: 128-row tiles on tcgen05; the other rows keep the row-tile kernel
                K.mla_prefill_tc(q3, pool, b.block_table, *tiles, self.pool.page_size, D, rope, m.scale, o3, gate=gate,
                                 window=m.window)
                ranges = b.rest_ranges
            span = min(self.max_seq_len, m.window + 64) if m.window else self.max_seq_len
            split_tokens = max(64, pad_to((span + self.attn_splits - 1) // self.attn_splits, 64))
            for r0, r1 in ranges:
                split = self.attn_splits > 1 and r1 - r0 <= 4 * self.decode_rows
                K.mla_attention(q3[r0:r1], pool, b.block_table, b.row_seq[r0:r1], b.row_pos[r0:r1], self.pool.page_size, D,
                                rope, m.scale, o3[r0:r1], splits=self.attn_splits if split else 1,
                                split_tokens=split_tokens if split else (1 << 29), decode_only=b.decode_only,
                                gate=gate[r0:r1], window=m.window)
        out = self._view(ws.mix_in, T, m.heads * vp)
        K.gemm(o_lat, mx.w_uv, out=out, x_group_koff=D, out_group_coff=vp, k=D)
        return out

    def _delta(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        K, KL, ws = self.K, self.KL, self.ws
        mx, m = lw.mixer, lw.spec.mixer
        ag = None
        if m.low_rank:
            ag = self._view(ws.ag, T, mx.w_ag.shape[0])
            a0 = mx.off["a1"]
            K.gemm(proj[:, a0:a0 + mx.w_ag.shape[1]], mx.w_ag, out=ag)
        out = self._view(ws.mix_in, T, mx.w_o.shape[1])
        decode = b.n_seqs == T and KL.delta_decode_supported(m)
        KL.delta_rule(proj, mx.off, ag, mx, m, self.cfg.norm_eps, self.states.state[layer], self.states.tail[layer],
                      b.seq_start, b.state_in, b.state_out, b.n_seqs, out, row_seq=b.row_seq[:T], scratch=ws.delta,
                      decode=decode, long_seqs=b.long_seqs)
        return out

    def _attention(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        KL, cfg = self.KL, self.cfg
        mx, m = lw.mixer, lw.spec.mixer
        pool = self.pool.layer(self.cache_index[layer])
        q = proj[:, mx.off["q"]:mx.off["q"] + m.heads * m.dim_pad]
        first = cfg.first_value_layer if m.v_mix else layer
        mixed = {} if first == layer else dict(first_pool=self.pool.layer(self.cache_index[first]),
                                               first_off=cfg.layers[first].mixer.v_offset)
        KL.gqa_prep(q, proj[:, mx.off["k"]:], proj[:, mx.off["v"]:], m, mx, self.rotation[m.rot_base, m.rot_dims],
                    b.positions[:T], b.write_slot[:T], pool, cfg.norm_eps, **mixed)
        return self._attend(q, m, pool, b, T)

    def _attend(self, q: torch.Tensor, m, pool: torch.Tensor, b: DeviceBatch, T: int, gate: Optional[torch.Tensor] = None,
                talk: Optional[torch.Tensor] = None, **form) -> torch.Tensor:
        """Attention of query rows over a layer's pool: prompt tiles on tcgen05, the other rows in the decode kernels.  With
        `talk` the rows of both get mixed softmax weights."""
        KL = self.KL
        out = self._view(self.ws.mix_in, T, m.heads * m.vdim_pad)
        page = self.pool.page_size
        ranges = [(0, T)]
        few = KL.gqa_decode_supported(m, q.dtype, page)
        o = out if talk is None else self._view(self.ws.o_all, T, m.heads * m.value_width)
        if b.n_tc_tiles and KL.gqa_tc_group(m, q.dtype, page):
            KL.gqa_prefill_tc(q, m, pool, b.block_table, *b.tc_tables[self.gqa_table], 128 // self.gqa_table, page, o, gate=gate,
                              **form)
            ranges = b.rest_ranges
        at = lambda r0, r1, o: (q[r0:r1], m, pool, b.block_table, b.row_seq[r0:r1], b.row_pos[r0:r1], page, o[r0:r1])
        rows = lambda r0, r1: dict(gate=None if gate is None else gate[r0:r1], **form)
        if not few:
            for r0, r1 in ranges:
                KL.gqa_attention(*at(r0, r1, o), **rows(r0, r1))
        if talk is not None and (not few or ranges != [(0, T)]):
            KL.value_mix(o, talk, m, out)
        if few:
            mixed = {} if talk is None else dict(talk=talk)
            for r0, r1 in ranges:
                KL.gqa_decode(*at(r0, r1, out), splits=KL.gqa_decode_splits(r1 - r0, m, self.max_seq_len),
                              decode_only=b.decode_only, **rows(r0, r1), **mixed)
        return out

    def _window(self, run: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        KL, mx, m = self.KL, lw.mixer, lw.spec.mixer
        pool = self.pool.layer(self.cache_index[run])
        form: dict = {}
        blocks = None
        if m.pool:
            form["mean"] = (self.states.pooled[run], self.states.buffers, b.state_out)
            blocks = (form["mean"], b.positions[:T], b.row_seq[:T], b.block_table, self.pool.page_size)
        if m.shared_keys or m.maps > 1:
            q = self._view(self.ws.q_rows, T, m.heads * m.maps * m.key_width)
        else:
            q = proj[:, mx.off["q"]:mx.off["q"] + m.heads * m.dim_pad]
        single = b.n_seqs == T
        KL.head_prep(proj, mx.off, m, mx, b.write_slot[:T], pool, self.cfg.norm_eps, q, self.rotation.get(self._rotation_key(m)),
                     b.positions[:T], blocks if single else None)
        if blocks is not None and not single:
            KL.pool_blocks(m, pool, *blocks)
        gate = proj[:, mx.off["g"]:] if m.gate else None
        return self._attend(q, m, pool, b, T, slopes=mx.slopes, gate=gate, talk=mx.talk, diff_lambda=mx.diff_lambda,
                            eps=self.cfg.norm_eps, **form)

    def _mamba(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        K, KL, ws = self.K, self.KL, self.ws
        mx, m = lw.mixer, lw.spec.mixer
        Ip = m.inner_pad
        seqs = (b.seq_start, b.state_in, b.state_out, b.n_seqs)
        x = self._view(ws.conv_x, T, Ip)
        KL.short_conv(proj[:, mx.off["x"]:mx.off["x"] + Ip], mx.conv, self.states.tail[layer], x, b.row_seq[:T], *seqs,
                      bias=mx.conv_b, silu=True)
        low = self._view(ws.low, T, mx.w_x.shape[0])
        # few output columns: row tiles small enough to fill the GPU
        K.gemm(x, mx.w_x, out=low, ntok=64 if (T >= 512 and not self.fp32) else None)
        dt = self._view(ws.dt, T, Ip)
        K.gemm(low[:, :mx.w_dt.shape[1]], mx.w_dt, out=dt)
        out = self._view(ws.mix_in, T, Ip)
        return KL.selective_scan(x, proj[:, mx.off["z"]:mx.off["z"] + Ip], low, mx.off_b, mx.off_c, dt, mx,
                                 self.states.state[layer], *seqs, out)

    def _mamba2(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        KL, ws = self.KL, self.ws
        mx, m = lw.mixer, lw.spec.mixer
        seqs = (b.seq_start, b.state_in, b.state_out, b.n_seqs)
        xbc = self._view(ws.conv_x, T, m.channels)
        KL.short_conv(proj[:, :m.channels], mx.conv, self.states.tail[layer], xbc, b.row_seq[:T], *seqs, bias=mx.conv_b, silu=True)
        out = self._view(ws.mix_in, T, m.inner_pad)
        KL.head_scan(xbc, proj, mx.off, m, mx, self.states.state[layer], *seqs, out, long_seqs=b.long_seqs)
        return KL.group_norm_rows(out, mx.o_norm, out, m.inner, m.norm_groups, self.cfg.norm_eps)

    def _mixer(self, layer: int, lw: LayerImage, proj: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        fn = {LatentMixer: self._latent, AttentionMixer: self._attention, WindowMixer: self._window,
              DeltaMixer: self._delta, MambaMixer: self._mamba, Mamba2Mixer: self._mamba2}[type(lw.spec.mixer)]
        return fn(layer, lw, proj, b, T)

    # -- feed-forward ------------------------------------------------------------------------
    def _shared_expert(self, lw: LayerImage, h: torch.Tensor, T: int) -> torch.Tensor:
        K, ws, s = self.K, self.ws, lw.spec.mlp
        mid = self._view(ws.shared_mid, T, lw.s_w2.shape[1])
        K.gemm(h, lw.s_w13, out=mid, epilogue=K.EPI_SWIGLU, act_limit=s.shared_limit, act_alpha=s.alpha, act_shift=s.shift)
        return K.gemm(mid, lw.s_w2, out=ws.shared_out[:T])

    def _moe(self, layer: int, lw: LayerImage, h: torch.Tensor, T: int, gate: Optional[list] = None) -> torch.Tensor:
        """Routed experts -> [T, top, width_pad] weighted expert rows.  With a shared expert the pre-activation of its gate is
        put into `gate`: fp32 [T, 1]."""
        K, ws, s = self.K, self.ws, lw.spec.mlp
        k, E, Wp = s.top, s.experts, self.cfg.width_pad
        fp = lw.e_w2.shape[2]
        idx, wts = self._view(ws.topk_idx, T, k), self._view(ws.topk_w, T, k)
        route_out = ws.route_out[:T * k]
        static = next((nt for nt in ws.static_rows if T <= nt), 0) if self.static_moe else 0
        if static:
            plan = ws.static_plans[layer, static]
            extra = ws.shared_gate[:T] if s.shared_ff else None
            K.router_append(h, lw.router_w, k, SCORE_SOFTMAX, plan, 0, E, idx, wts, ws.xg, n_groups=s.groups,
                            topk_groups=s.keep, group_top=1, dst_slots=k, normalize=s.renormalize, logit_bias=lw.router_b,
                            extra=extra)
            if extra is not None:
                gate.append(extra)
            rows = plan.cap_rows
            scatter_plan = plan
        else:
            products = self._view(ws.router_logits, T, lw.router_w.shape[0])
            K.gemm(h, lw.router_w, out=products, ntok=32 if (T >= 1024 and not self.fp32) else None)
            if s.shared_ff:
                gate.append(products[:, E:])
            K.router_topk(products[:, :E], k, SCORE_SOFTMAX, n_groups=s.groups, topk_groups=s.keep, group_top=1, out_idx=idx,
                          out_w=wts, normalize=s.renormalize, logit_bias=lw.router_b)
            ntok = _pow2_at_least(2 * T * k / E, 16, 128)
            plan = ws.plans[E, k, ntok]
            K.moe_plan(idx, wts, plan, 0, E, dst_slots=k)
            rows = T * k
            if self.fp32:       # a row copy: two bf16 elements per fp32 element
                K.gather_rows(h.view(torch.bfloat16), plan, ws.xg.view(torch.bfloat16), cap_rows=rows)
            else:
                K.gather_rows(h, plan, ws.xg, cap_rows=rows)
            scatter_plan = plan
            if not self.fp32 and ntok == 128 and rows >= 160 * E:
                # prefill-sized expert loads: the scatter GEMM keeps one accumulator and takes 256-row tiles
                scatter_plan = ws.plans[E, k, 256] = K.moe_retile(plan, 256, ws.plans[E, k, 256])
        hmid = self._view(ws.hmid, rows, fp)
        K.gemm(ws.xg[:rows], lw.e_w13, out=hmid, epilogue=K.EPI_SWIGLU, plan=plan, act_limit=s.limit, act_alpha=s.alpha,
               act_shift=s.shift)
        K.gemm(hmid, lw.e_w2, out=route_out, epilogue=K.EPI_SCATTER, plan=scatter_plan, scatter_rows=T * k)
        return route_out.view(T, k, Wp)

    # -- blocks ----------------------------------------------------------------------------
    def _mix(self, i: int, lw: LayerImage, h: torch.Tensor, b: DeviceBatch, T: int) -> torch.Tensor:
        """Input projection, mixer and output projection (into `ws.mix`); returns the projected rows."""
        K, ws, mx, prof = self.K, self.ws, lw.mixer, self.prof
        if prof is not None:
            prof.mark(i, "proj")
        proj = self._view(ws.proj, T, mx.w_in.shape[0])
        K.gemm(h, mx.w_in, out=proj, bias=mx.b_in)
        if prof is not None:
            prof.mark(i, "mixer")
        a = self._mixer(i, lw, proj, b, T)
        if prof is not None:
            prof.mark(i, "mixer.out")
        K.gemm(a, mx.w_o, out=ws.mix[:T])
        return proj

    def _tapped(self, i: int, x: torch.Tensor) -> None:
        if self.tap is not None and self.tap.wants(i, "layer_out"):
            self.tap.write(i, "layer_out", x)

    def _gated_blocks(self, b: DeviceBatch, T: int, x: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        KL, ws, cfg = self.KL, self.ws, self.cfg
        layers = self.w.layers
        if self.static_moe and T <= ws.static_rows[-1] and ws.static_plans:
            self.M.fill_(ws.route_cnt, 0)
        KL.embed_norm(b.token_ids[:T], self.w.embed, x, layers[0].norm, h, cfg.width, cfg.norm_eps)
        for i, lw in enumerate(layers):
            mx = lw.mixer
            ffn = None
            if lw.spec.mlp is not None:
                main = torch.cuda.current_stream()
                self.side_stream.wait_stream(main)
                with torch.cuda.stream(self.side_stream):
                    ffn = self._moe(i, lw, h, T)
            proj = self._mix(i, lw, h, b, T)
            if ffn is not None:
                torch.cuda.current_stream().wait_stream(self.side_stream)
            if self.prof is not None:
                self.prof.mark(i, "tail")
            nxt = layers[i + 1].norm if i + 1 < len(layers) else self.w.final_norm
            KL.gated_residual_norm(
                x, nxt, h, cfg.width, cfg.norm_eps, mix=ws.mix[:T], gate1=proj[:, mx.off["rg1"]:], bias1=lw.rg1_b,
                ffn=ffn, topk=lw.spec.mlp.top if ffn is not None else 0,
                gate2=proj[:, mx.off["rg2"]:] if ffn is not None else None, bias2=lw.rg2_b)
            self._tapped(i, x)
        return x

    def _output_norm_blocks(self, b: DeviceBatch, T: int, x: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        K, KL, ws, cfg = self.K, self.KL, self.ws, self.cfg
        layers, eps = self.w.layers, cfg.norm_eps
        single = b.n_seqs == T          # one row per sequence: a row's earlier convolution inputs are all in the state
        seqs = (b.seq_start, b.state_in, b.state_out, b.n_seqs)

        def fused(i):
            """Input convolution of layer i inside the kernel that completes its stream rows."""
            if i >= len(layers) or not single or layers[i].canon is None:
                return None
            return layers[i].canon, self.states.canon[i], b.state_in, b.state_out, h

        KL.embed_stream(b.token_ids[:T], self.w.embed, x, cfg.width, positions=b.positions[:T], pos_table=self.w.pos,
                        canon=fused(0))
        for i, lw in enumerate(layers):
            if lw.canon is not None and not single:
                KL.short_conv(x, lw.canon, self.states.canon[i], h, b.row_seq[:T], *seqs, residual=True)
            self._mix(i, lw, h, b, T)
            if self.prof is not None:
                self.prof.mark(i, "tail")
            if lw.spec.mlp is None:
                KL.add_normed(x, ws.mix[:T], lw.norm1, cfg.width, eps, canon=fused(i + 1))
            else:
                act, ff = ws.act[:T], self._view(ws.ff, T, lw.w_up.shape[0])
                KL.add_normed(x, ws.mix[:T], lw.norm1, cfg.width, eps, act=act)
                K.gemm(act, lw.w_up, out=ff, epilogue=K.EPI_GELU)
                K.gemm(ff, lw.w_down, out=ws.mix[:T])
                KL.add_normed(x, ws.mix[:T], lw.norm2, cfg.width, eps, canon=fused(i + 1))
            self._tapped(i, x)
        return x

    def _sandwich_blocks(self, b: DeviceBatch, T: int, x: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        K, KL, ws, cfg = self.K, self.KL, self.ws, self.cfg
        runs, starts = cfg.runs, set(cfg.pass_starts)
        grouped = dict(dim=cfg.width, eps=cfg.norm_eps, groups=cfg.norm_groups)
        embedding = dict(ids=b.token_ids[:T], table=self.w.embed)
        layer = lambda r: self.w.layers[runs[r]]

        def close(r: int, norm: torch.Tensor, bias=None) -> None:
            """End of run r: its last output norm and residual addition, then what the next run starts with."""
            nxt = layer(r + 1).norm1 if r + 1 < len(runs) else None
            again = embedding if r + 1 in starts else {}
            y = ws.mix[:T]
            if again and self.tap is not None and self.tap.wants(r, "layer_out"):
                # the tapped stream is the layer's own: the embedding joins it in a launch of its own
                KL.sandwich_step(x, out_norm=norm, y=y, bias=bias, **grouped)
                self._tapped(r, x)
                KL.sandwich_step(x, in_norm=nxt, act=h, **again, **grouped)
                return
            KL.sandwich_step(x, out_norm=norm, y=y, bias=bias, in_norm=nxt, act=h if nxt is not None else None, **again, **grouped)
            self._tapped(r, x)

        KL.sandwich_step(x, in_norm=layer(0).norm1, act=h, fresh=True, **embedding, **grouped)
        for r in range(len(runs)):
            lw = layer(r)
            self._mix(r, lw, h, b, T)
            if self.prof is not None:
                self.prof.mark(r, "tail")
            if lw.spec.mlp is None:
                close(r, lw.norm1b, lw.mixer.o_bias)
                continue
            ff = self._view(ws.ff, T, lw.w_down.shape[1])
            KL.sandwich_step(x, out_norm=lw.norm1b, y=ws.mix[:T], bias=lw.mixer.o_bias, in_norm=lw.norm2, act=h, **grouped)
            K.gemm(h, lw.w_up, out=ff, epilogue=K.EPI_GEGLU)
            K.gemm(ff, lw.w_down, out=ws.mix[:T])
            close(r, lw.norm2b)
        return x

    def _pre_norm_blocks(self, b: DeviceBatch, T: int, x: torch.Tensor, h: torch.Tensor) -> torch.Tensor:
        """Returns the buffer that holds the final stream."""
        K, KL, ws, cfg = self.K, self.KL, self.ws, self.cfg
        layers = self.w.layers
        row = dict(dim=cfg.width, eps=cfg.norm_eps, like=h)
        seqs = (b.row_seq[:T], b.seq_start, b.state_in, b.state_out, b.n_seqs)
        swap = cfg.token_shift and b.n_seqs != T         # a shift that sees rows of this batch leaves the old stream alone
        if self.static_moe and T <= ws.static_rows[-1] and ws.static_plans:
            self.M.fill_(ws.route_cnt, 0)

        def entry(i: int) -> dict:
            """What layer i's mixer reads."""
            if i >= len(layers):
                return {}
            lw = layers[i]
            shift = {} if lw.shift is None else dict(shift=lw.shift, plane=self.states.shift[i], seqs=seqs)
            return dict(norm=lw.norm1, act=h, **shift)

        KL.pre_norm_step(None, x, ids=b.token_ids[:T], table=self.w.embed, scale=cfg.embed_scale, **entry(0), **row)
        other = ws.x_next[:T] if swap else x
        for i, lw in enumerate(layers):
            self._mix(i, lw, h, b, T)
            if self.prof is not None:
                self.prof.mark(i, "tail")
            left = dict(y=ws.mix[:T])
            if lw.spec.mlp is not None:
                KL.pre_norm_step(x, x, norm=lw.norm2, act=h, **left, **row)
                if isinstance(lw.spec.mlp, MoeSpec):
                    left = self._routed(i, lw, h, T)
                else:
                    ff = self._view(ws.ff, T, lw.w_up.shape[0])
                    K.gemm(h, lw.w_up, out=ff, epilogue=K.EPI_GELU, bias=lw.up_b)
                    K.gemm(ff, lw.w_down, out=ws.mix[:T], bias=lw.down_b)
            KL.pre_norm_step(x, other, **left, **entry(i + 1), **row)
            x, other = other, x
            self._tapped(i, x)
        return x

    def _routed(self, i: int, lw: LayerImage, h: torch.Tensor, T: int) -> dict:
        """Expert rows of a layer, with the shared expert computed beside them."""
        s, gate = lw.spec.mlp, []
        if not s.shared_ff:
            return dict(ffn=self._moe(i, lw, h, T), topk=s.top)
        main = torch.cuda.current_stream()
        self.side_stream.wait_stream(main)
        with torch.cuda.stream(self.side_stream):
            shared = self._shared_expert(lw, h, T)
        ffn = self._moe(i, lw, h, T, gate)
        main.wait_stream(self.side_stream)
        return dict(ffn=ffn, topk=s.top, shared=shared, shared_gate=gate[0])

    # -- whole model ---------------------------------------------------------------------
    def hidden_states(self, b: DeviceBatch, T: int) -> torch.Tensor:
        """Runs the layers.  Returns the rows the head starts from: normalised ones
        (`ws.h`) behind parallel gated blocks, the stream itself behind the other forms."""
        ws = self.ws
        x, h = ws.x[:T], ws.h[:T]
        gated = self.cfg.block == PARALLEL_GATED
        x = {PARALLEL_GATED: self._gated_blocks, OUTPUT_NORM: self._output_norm_blocks, SANDWICH_NORM: self._sandwich_blocks,
             PRE_NORM: self._pre_norm_blocks}[self.cfg.block](b, T, x, h)
        if self.prof is not None:
            self.prof.mark(len(self.cfg.runs), None)
        return h if gated else x

    def head(self, h: torch.Tensor, logit_rows: torch.Tensor, L: int):
        """Logits and greedy tokens of `L` rows -> (next_id, next_val, logits), views of the workspace."""
        K, ws = self.K, self.ws
        hn = ws.hn_last[:L]
        if self.cfg.block == PRE_NORM:
            self.KL.norm_rows(h, logit_rows[:L], self.w.final_norm[None], hn, self.cfg.width, self.cfg.norm_eps, rms=True)
        elif self.cfg.block == OUTPUT_NORM:
            self.KL.norm_rows(h, logit_rows[:L], self.w.final_norm, hn, self.cfg.width, self.cfg.norm_eps)
        elif self.cfg.block == SANDWICH_NORM:
            self.KL.sandwich_rows(h, logit_rows[:L], self.w.final_norm, hn, self.cfg.width, self.cfg.norm_eps,
                                  self.cfg.norm_groups)
        else:
            self.M.gather_rows(h, logit_rows[:L], hn)
        logits = ws.logits[:L]
        K.gemm(hn, self.w.lm_head, out=logits)
        if self.cfg.logit_softcap:
            self.KL.softcap_(logits, self.cfg.logit_softcap)
        K.argmax_chunked(logits, ws.argmax_scratch, ws.next_id[:L], ws.next_val[:L])
        return ws.next_id[:L], ws.next_val[:L], logits

    def forward(self, b: DeviceBatch, want_logits: bool = False, start_layer: int = 0, h0=None):
        """Runs the batch; returns (next_id [n_logit] int32, next_val, logits or None)."""
        T = b.token_ids.shape[0]
        assert T <= self.ws.max_rows and b.n_logit <= self.ws.max_logit_rows and start_layer == 0 and h0 is None
        from ..ops import _lib
        start = _lib.LAUNCHES[0]
        h = self.hidden_states(b, T)
        self.last_hidden = h
        out = (None, None, None)
        if b.n_logit:
            ids, vals, logits = self.head(h, b.logit_rows, b.n_logit)
            out = (ids, vals, logits if want_logits else None)
        self.launches = _lib.LAUNCHES[0] - start
        return out

    def forward_rows(self, b: DeviceBatch, consume) -> None:
        """Runs the batch and hands the logits of the wanted rows to `consume(first, logits)`, in pieces of at most
        `max_logit_rows` rows."""
        T = b.token_ids.shape[0]
        assert T <= self.ws.max_rows
        from ..ops import _lib
        start = _lib.LAUNCHES[0]
        h = self.hidden_states(b, T)
        self.last_hidden = h
        for lo in range(0, b.n_logit, self.ws.max_logit_rows):
            n = min(self.ws.max_logit_rows, b.n_logit - lo)
            consume(lo, self.head(h, b.logit_rows[lo:], n)[2])
        self.launches = _lib.LAUNCHES[0] - start
