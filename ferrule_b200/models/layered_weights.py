"""Weight image of a layer-list model, packed once at load time into what the kernels read.

Every linear that reads the mixer's input is one row block of a single matrix `w_in`, so a layer starts with one GEMM;
blocks begin at multiples of 8 columns of its output:

  latent layer     q (heads x dim, each head padded to 8) | rotated q (heads x rot_dim) | dkv | head gates; queries with a
                   latent of their own: dq | dkv | head gates, and q | rotated q are row blocks of `w_uq`
  attention layer  q | k | v, each head padded to 8
  window layer     q | k | v (unless the keys are the values) | output gate, each head padded to 8
  delta layer      q | k | v | decay low rank | gate low rank | beta      (full projections: decay | gate | beta)
  mamba layer      x | z
  mamba2 layer     x | B | C | z | dt

(`b_in`: biases of the projection, added by the GEMM) followed, in parallel gated blocks, by residual gate 1 | residual gate 2.

The second halves of the delta layer's two low-rank projections are one block-diagonal matrix `w_ag` (fp32 output:
decay pre-activations and output-gate pre-activations).  Keys and values of a latent layer are absorbed: `w_uk_t` maps a
query head to the latent space, `w_uv` maps the attention output (a latent row per head) to the head's value.  Widths
are padded with zeros to multiples of 8 (latents to multiples of 64), so every size takes the same kernels.

Constants that enter norms, gates and recurrences are fp32 tensors; everything else has the model's dtype.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional

import torch

from .layered_config import (PARALLEL_GATED, PRE_NORM, SANDWICH_NORM, AttentionMixer, DeltaMixer, DenseSpec, LatentMixer,
                             LayeredConfig, LayerSpec, Mamba2Mixer, MambaMixer, MoeSpec, WindowMixer, pad_to)

GetTensor = Callable[[str], torch.Tensor]


def _pad(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zero-pad at the end of every dimension."""
    if tuple(t.shape) == tuple(shape):
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


@dataclass
class MixerImage:
    w_in: torch.Tensor                       # [sum of blocks, width_pad]
    off: Dict[str, int]                      # block name -> first output column
    w_o: torch.Tensor                        # [width_pad, inputs]
    b_in: Optional[torch.Tensor] = None      # fp32, one per row of w_in
    # latent attention
    w_uk_t: Optional[torch.Tensor] = None    # [heads, row_dim, dim_pad]
    w_uv: Optional[torch.Tensor] = None      # [heads, vdim_pad, row_dim]
    kv_norm: Optional[torch.Tensor] = None   # fp32 [row_dim]
    w_uq: Optional[torch.Tensor] = None      # [heads * dim_pad | heads * rot_dim, q_rank padded to 8]
    off_uq: Dict[str, int] = field(default_factory=dict)     # its blocks: q, qr
    dq_norm: Optional[torch.Tensor] = None   # fp32 [q_rank padded to 8]
    # delta rule
    w_ag: Optional[torch.Tensor] = None      # [heads * dim | heads * vdim, low ranks]
    off_gate: int = 0
    conv: Optional[torch.Tensor] = None      # fp32 [taps, channels]
    a_neg: Optional[torch.Tensor] = None     # fp32 [heads] = -exp(A_log)
    dt_bias: Optional[torch.Tensor] = None   # fp32 [heads * dim] (one decay per head: [heads]); mamba: [inner_pad]
    o_norm: Optional[torch.Tensor] = None    # fp32 [vdim]
    # attention
    q_norm: Optional[torch.Tensor] = None    # fp32 [heads * dim_pad]
    k_norm: Optional[torch.Tensor] = None    # fp32 [kv_heads * dim_pad]
    v_mix: float = 0.0                       # share of the first mixing layer's values
    # window attention (q_norm, k_norm: [dim_pad], shared by the heads)
    q_bias: Optional[torch.Tensor] = None    # fp32 [heads * maps * dim_pad]
    k_bias: Optional[torch.Tensor] = None    # fp32 [kv_heads * maps * dim_pad]
    o_bias: Optional[torch.Tensor] = None    # fp32 [width_pad]
    q_mix: Optional[torch.Tensor] = None     # fp32 [heads, heads]: factor of head g's raw scores in head h's; not mixed: [heads]
    slopes: Optional[torch.Tensor] = None    # fp32 [heads]: taken off a score per token of distance
    diff_lambda: float = 0.0                 # weight of the second map's output
    talk: Optional[torch.Tensor] = None      # fp32 [heads, heads]: share of head g's softmax weights in head h's
    # mamba (also conv, dt_bias)
    w_x: Optional[torch.Tensor] = None       # [dt | B | C rows, inner_pad], blocks at off_b / off_c
    off_b: int = 0
    off_c: int = 0
    w_dt: Optional[torch.Tensor] = None      # [inner_pad, dt_rank padded to 8]
    conv_b: Optional[torch.Tensor] = None    # fp32 [inner_pad]
    a_log2: Optional[torch.Tensor] = None    # fp32 [state, inner_pad] = -exp(A_log) * log2(e)
    d_skip: Optional[torch.Tensor] = None    # fp32 [inner_pad] (mamba2: [heads])
    # mamba2: conv [taps, channels], conv_b [channels], dt_bias, a_neg [heads], o_norm [inner_pad]


@dataclass
class LayerImage:
    spec: LayerSpec
    mixer: MixerImage
    # parallel gated block
    norm: Optional[torch.Tensor] = None      # fp32 [1]: one number for all coordinates
    rg1_b: Optional[torch.Tensor] = None     # fp32 [width_pad]
    rg2_b: Optional[torch.Tensor] = None
    router_w: Optional[torch.Tensor] = None  # [experts, width_pad]
    e_w13: Optional[torch.Tensor] = None     # [experts, 2 * ff_pad, width_pad]
    e_w2: Optional[torch.Tensor] = None      # [experts, width_pad, ff_pad]
    # output-norm block: norm weights and biases of the mixer's and the feed-forward's output, input convolution
    norm1: Optional[torch.Tensor] = None     # fp32 [2, width_pad]
    norm2: Optional[torch.Tensor] = None     # fp32 [2, width_pad]
    canon: Optional[torch.Tensor] = None     # fp32 [taps, width_pad]
    # sandwich block: norm weights of the sublayers' inputs (norm1, norm2 [width_pad]) and outputs
    norm1b: Optional[torch.Tensor] = None    # fp32 [width_pad]
    norm2b: Optional[torch.Tensor] = None    # fp32 [width_pad]
    w_up: Optional[torch.Tensor] = None      # [ff_pad, width_pad]; gated: [gate ff_pad | up ff_pad, width_pad]
    w_down: Optional[torch.Tensor] = None    # [width_pad, ff_pad]
    up_b: Optional[torch.Tensor] = None      # fp32 [ff_pad]
    down_b: Optional[torch.Tensor] = None    # fp32 [width_pad]
    # pre-norm block: norm1, norm2 [width_pad]; share of the previous token in the mixer's input
    shift: Optional[torch.Tensor] = None     # fp32 [width_pad]
    # experts, also: router_w has one row more with a shared expert (its gate)
    router_b: Optional[torch.Tensor] = None  # fp32 [experts]
    s_w13: Optional[torch.Tensor] = None     # shared expert [2 * ff_pad, width_pad]
    s_w2: Optional[torch.Tensor] = None      # [width_pad, ff_pad]


@dataclass
class LayeredWeights:
    cfg: LayeredConfig
    embed: torch.Tensor                      # [vocab, width_pad]
    layers: List[LayerImage]
    final_norm: torch.Tensor                 # fp32 [1], output-norm blocks: [2, width_pad], sandwich and pre-norm blocks: [width_pad]
    lm_head: torch.Tensor                    # [vocab, width_pad]
    pos: Optional[torch.Tensor] = None       # [max_position, width_pad] learned position vectors
    mtp: list = field(default_factory=list)  # the architecture has no proposal stages
    weight_format: str = "bf16"

    def nbytes(self) -> int:
        total = sum(t.numel() * t.element_size() for t in (self.embed, self.final_norm, self.lm_head)
                    + (() if self.pos is None else (self.pos,)))
        for l in {id(l): l for l in self.layers}.values():       # (layers may share an image)
            for holder in (l, l.mixer):
                total += sum(t.numel() * t.element_size() for t in vars(holder).values() if isinstance(t, torch.Tensor))
        return total


class _Blocks:
    """Stacks row blocks, each starting at a multiple of 8."""

    def __init__(self, cols: int):
        self.cols, self.rows, self.off, self.parts, self.biases = cols, 0, {}, [], {}

    def add(self, name: str, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> None:
        n = pad_to(w.shape[0], 8)
        self.off[name] = self.rows
        self.parts.append(_pad(w, n, self.cols))
        if bias is not None:
            self.biases[self.rows] = bias
        self.rows += n

    def matrix(self) -> torch.Tensor:
        return torch.cat(self.parts, 0).contiguous()

    def bias(self) -> Optional[torch.Tensor]:
        if not self.biases:
            return None
        out = torch.zeros(self.rows, dtype=torch.float32, device=self.parts[0].device)
        for at, b in self.biases.items():
            out[at:at + b.shape[0]] = b.float()
        return out


def _pack_latent(m: LatentMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp, DL = cfg.width_pad, m.row_dim
    dp, vp = pad_to(m.dim, 8), pad_to(m.vdim, 8)
    w_q = get(p + ("uq" if m.q_rank else "q")).view(m.heads, m.dim + m.rot_dim, -1)
    src = _Blocks(pad_to(m.q_rank, 8)) if m.q_rank else b
    src.add("q", _pad(w_q[:, :m.dim], m.heads, dp, src.cols).reshape(m.heads * dp, src.cols))
    if m.rot_dim:
        src.add("qr", _pad(w_q[:, m.dim:], m.heads, m.rot_dim, src.cols).reshape(m.heads * m.rot_dim, src.cols))
    if m.q_rank:
        b.add("dq", get(p + "dq"))
    b.add("dkv", get(p + "dkv"))
    b.add("g", get(p + "g"))
    uk = get(p + "uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2)
    uv = get(p + "uv").view(m.heads, m.vdim, m.kv_rank)
    o = _pad(get(p + "o").view(cfg.width, m.heads, m.vdim), Wp, m.heads, vp)
    img = MixerImage(None, b.off, o.reshape(Wp, m.heads * vp).contiguous(),
                     w_uk_t=_pad(uk, m.heads, DL, dp).contiguous(), w_uv=_pad(uv, m.heads, vp, DL).contiguous(),
                     kv_norm=_pad(get(p + "dkv.norm").float(), DL).contiguous())
    if m.q_rank:
        img.w_uq, img.off_uq = src.matrix(), src.off
        img.dq_norm = _pad(get(p + "dq.norm").float(), src.cols).contiguous()
    return img


def _pack_attention(m: AttentionMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp, dp, vp = cfg.width_pad, m.dim_pad, m.vdim_pad
    for name, heads, d, pad in (("q", m.heads, m.dim, dp), ("k", m.kv_heads, m.dim, dp), ("v", m.kv_heads, m.vdim, vp)):
        b.add(name, _pad(get(p + name).view(heads, d, cfg.width), heads, pad, Wp).reshape(heads * pad, Wp))
    o = _pad(get(p + "o").view(cfg.width, m.heads, m.vdim), Wp, m.heads, vp)
    norm = lambda name, heads: _pad(get(p + name).float().view(heads, m.dim), heads, dp).reshape(-1).contiguous()
    return MixerImage(None, b.off, o.reshape(Wp, m.heads * vp).contiguous(), q_norm=norm("q.norm", m.heads),
                      k_norm=norm("k.norm", m.kv_heads), v_mix=float(get(p + "vmix").float()) if m.v_mix else 0.0)


def _pack_window(m: WindowMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp, dp, vp = cfg.width_pad, m.dim_pad, m.vdim_pad
    nq, nk = m.heads * m.maps, m.kv_heads * m.maps
    blocks = [("q", nq, m.dim, dp), ("k", nk, m.dim, dp)]
    if not m.tied_values:
        blocks.append(("v", m.kv_heads, m.vdim, vp))
    if m.gate:
        blocks.append(("g", m.heads, m.vdim, vp))
    bias = lambda name, heads, d, pad: _pad(get(p + name + ".b").float().view(heads, d), heads, pad).reshape(-1).contiguous()
    in_gemm = "v" in m.biases          # the projection adds them all
    for name, heads, d, pad in blocks:
        b.add(name, _pad(get(p + name).view(heads, d, cfg.width), heads, pad, Wp).reshape(heads * pad, Wp),
              bias(name, heads, d, pad) if in_gemm and name in m.biases else None)
    o = _pad(get(p + "o").view(cfg.width, m.heads, m.vdim), Wp, m.heads, vp)
    norm = lambda name: _pad(get(p + name).float(), dp).contiguous() if m.norm_weights else None
    f64 = lambda name: get(p + name).double()
    img = MixerImage(None, b.off, o.reshape(Wp, m.heads * vp).contiguous(), q_norm=norm("q.norm"), k_norm=norm("k.norm"))
    if not in_gemm and "q" in m.biases:
        img.q_bias, img.k_bias = bias("q", nq, m.dim, dp), bias("k", nk, m.dim, dp)
    if m.mix_weights:
        img.talk = get(p + "talk").float().contiguous()
    if "o" in m.biases:
        img.o_bias = _pad(get(p + "o.b").float(), Wp).contiguous()
    # score_h = sum_g T[h, g] (scale temp_g q_g . k - slope_g distance): everything but q and k is constant
    scale = torch.full((m.heads,), m.scale, dtype=torch.float64, device=o.device)
    if m.head_temps:
        scale = scale * f64("temp")
    mix = f64("talk") if m.mix_heads else None
    img.q_mix = (scale if mix is None else mix * scale).float().contiguous()
    if m.distance_bias:
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / m.heads) for h in range(m.heads)], dtype=torch.float64, device=o.device)
        img.slopes = (slopes if mix is None else mix @ slopes).float().contiguous()
    if m.maps == 2:
        dot = lambda a, c: math.exp(float((f64(a) * f64(c)).sum()))
        img.diff_lambda = dot("lq1", "lk1") - dot("lq2", "lk2") + m.diff
    return img


def _pack_mamba(m: MambaMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Ip, LOG2E = m.inner_pad, 1.4426950408889634
    w_in = get(p + "in")
    b.add("x", w_in[:m.inner])
    b.add("z", w_in[m.inner:])
    low, w_x = _Blocks(Ip), get(p + "x")
    low.add("dt", w_x[:m.dt_rank])
    low.add("B", w_x[m.dt_rank:m.dt_rank + m.state])
    low.add("C", w_x[m.dt_rank + m.state:])
    vec = lambda name: _pad(get(p + name).float(), Ip).contiguous()
    a = -torch.exp(get(p + "A_log").double()) * LOG2E
    return MixerImage(None, b.off, _pad(get(p + "o"), cfg.width_pad, Ip).contiguous(), w_x=low.matrix(), off_b=low.off["B"],
                      off_c=low.off["C"], w_dt=_pad(get(p + "dt"), Ip, pad_to(m.dt_rank, 8)).contiguous(),
                      conv=_pad(get(p + "conv").float().t(), m.taps, Ip).contiguous(), conv_b=vec("conv.b"),
                      dt_bias=vec("dt.b"), d_skip=vec("D"), a_log2=_pad(a.float().t(), m.state, Ip).contiguous())


def _pack_mamba2(m: Mamba2Mixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    bc = m.groups * m.state
    z, x, B, C, dt = get(p + "in").split([m.inner, m.inner, bc, bc, m.heads])
    for name, w in (("x", x), ("B", B), ("C", C), ("z", z), ("dt", dt)):
        b.add(name, w)
    assert b.off["z"] == m.channels

    def channels(t):        # x | B | C, padded as the projection's blocks
        return torch.cat([_pad(c, pad_to(c.shape[0], 8), *c.shape[1:]) for c in t.float().split([m.inner, bc, bc])])

    vec = lambda name: get(p + name).float().contiguous()
    return MixerImage(None, b.off, _pad(get(p + "o"), cfg.width_pad, m.inner_pad).contiguous(), off_b=b.off["B"],
                      off_c=b.off["C"], conv=channels(get(p + "conv").view(-1, m.taps)).t().contiguous(),
                      conv_b=channels(get(p + "conv.b")).contiguous(), dt_bias=vec("dt_bias"), d_skip=vec("D"),
                      a_neg=-torch.exp(get(p + "A_log").double()).float(), o_norm=_pad(vec("norm"), m.inner_pad).contiguous())


def _pack_delta(m: DeltaMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp = cfg.width_pad
    nk, nv, nd = m.kv_heads * m.dim, m.heads * m.vdim, m.heads * m.dim
    for name in ("q", "k", "v") + (("a1", "g1", "b") if m.low_rank else ("a", "g", "b")):
        b.add(name, get(p + name))
    ag, nd8 = None, 0
    if m.low_rank:
        ra, rg, nd8 = pad_to(m.decay_rank, 8), pad_to(m.gate_rank, 8), pad_to(nd, 8)
        a2, g2 = get(p + "a2"), get(p + "g2")
        ag = torch.zeros(nd8 + nv, ra + rg, dtype=a2.dtype, device=a2.device)
        ag[:nd, :m.decay_rank] = a2
        ag[nd8:, ra:ra + m.gate_rank] = g2
    conv = torch.cat([get(p + n + ".conv").view(-1, m.taps) for n in ("q", "k", "v")], 0).float().t().contiguous()
    assert conv.shape[1] == m.channels and nk + nk + nv == m.channels
    return MixerImage(None, b.off, _pad(get(p + "o"), Wp, pad_to(nv, 8)).contiguous(), w_ag=ag, off_gate=nd8, conv=conv,
                      a_neg=-torch.exp(get(p + "A_log").float()), dt_bias=get(p + "dt_bias").float().contiguous(),
                      o_norm=get(p + "norm").float().contiguous())


_PACK = {LatentMixer: _pack_latent, AttentionMixer: _pack_attention, WindowMixer: _pack_window, DeltaMixer: _pack_delta,
         MambaMixer: _pack_mamba, Mamba2Mixer: _pack_mamba2}


def _pack_dense(s: DenseSpec, p: str, get: GetTensor, cfg: LayeredConfig, img: LayerImage) -> None:
    Wp, fp = cfg.width_pad, pad_to(s.ff, 8)
    up = _pad(get(p + "up"), fp, Wp)
    img.w_up = (torch.cat([_pad(get(p + "gate"), fp, Wp), up]) if s.gated else up).contiguous()
    img.w_down = _pad(get(p + "down"), Wp, fp).contiguous()
    if s.biases:
        img.up_b, img.down_b = _pad(get(p + "up.b").float(), fp).contiguous(), _pad(get(p + "down.b").float(), Wp).contiguous()


def _pack_moe(s: MoeSpec, p: str, get: GetTensor, cfg: LayeredConfig, img: LayerImage) -> None:
    Wp, fp = cfg.width_pad, pad_to(s.ff, 8)
    router = [get(p + "router")] + ([get(p + "shared.sg")] if s.shared_ff else [])
    img.router_w = _pad(torch.cat(router), s.experts + len(router) - 1, Wp).contiguous()
    if s.router_bias:
        img.router_b = get(p + "router.b").float().contiguous()
    if s.shared_ff:
        sp, q = pad_to(s.shared_ff, 8), p + "shared."
        img.s_w13 = torch.cat([_pad(get(q + "gate"), sp, Wp), _pad(get(q + "up"), sp, Wp)]).contiguous()
        img.s_w2 = _pad(get(q + "down"), Wp, sp).contiguous()
    like = img.router_w
    img.e_w13 = torch.zeros(s.experts, 2 * fp, Wp, dtype=like.dtype, device=like.device)
    img.e_w2 = torch.zeros(s.experts, Wp, fp, dtype=like.dtype, device=like.device)
    for e in range(s.experts):
        q = f"{p}e{e}."
        img.e_w13[e, :s.ff, :cfg.width] = get(q + "gate")
        img.e_w13[e, fp:fp + s.ff, :cfg.width] = get(q + "up")
        img.e_w2[e, :cfg.width, :s.ff] = get(q + "down")


def pack_weights(cfg: LayeredConfig, get: GetTensor) -> LayeredWeights:
    """`get(name)` returns a checkpoint tensor in the dtype and on the device the model runs with."""
    Wp = cfg.width_pad
    gated, sandwich, pre = (cfg.block == k for k in (PARALLEL_GATED, SANDWICH_NORM, PRE_NORM))
    vec = lambda name: _pad(get(name).float(), Wp).contiguous()
    norm = lambda name: vec(name) if sandwich or pre else torch.stack([vec(n) for n in (name, name + ".b")]).contiguous()
    layers: List[LayerImage] = []
    owners: Dict[int, LayerImage] = {}
    for i, spec in enumerate(cfg.layers):
        if cfg.owner(i) in owners:
            layers.append(owners[cfg.owner(i)])
            continue
        p = f"l{cfg.owner(i)}."
        b = _Blocks(Wp)
        mx = _PACK[type(spec.mixer)](spec.mixer, p + "mix.", get, cfg, b)
        img = owners[cfg.owner(i)] = LayerImage(spec, mx)
        if gated:
            img.norm = get(p + "norm1").float().reshape(1).contiguous()
            img.rg1_b = _pad(get(p + "rg1.b").float(), Wp).contiguous()
            b.add("rg1", get(p + "rg1"))
        else:
            img.norm1 = norm(p + "norm1")
        if sandwich:
            img.norm1b = norm(p + "norm1b")
        if cfg.token_shift:
            img.shift = vec(p + "shift")
        if cfg.canon_taps:
            img.canon = _pad(get(p + "canon1").float().view(cfg.width, cfg.canon_taps).t(), cfg.canon_taps, Wp).contiguous()
        if spec.mlp is not None:
            if gated:
                b.add("rg2", get(p + "rg2"))
                img.rg2_b = _pad(get(p + "rg2.b").float(), Wp).contiguous()
            else:
                img.norm2 = norm(p + "norm2")
            if sandwich:
                img.norm2b = norm(p + "norm2b")
            (_pack_moe if isinstance(spec.mlp, MoeSpec) else _pack_dense)(spec.mlp, p + "mlp.", get, cfg, img)
        mx.w_in, mx.b_in = b.matrix(), b.bias()
        layers.append(img)
    final = get("final.norm").float().reshape(1).contiguous() if gated else norm("final.norm")
    pos = _pad(get("pos"), cfg.max_position, Wp).contiguous() if cfg.learned_positions else None
    return LayeredWeights(cfg, _pad(get("embed"), cfg.vocab_size, Wp).contiguous(), layers, final,
                          _pad(get("head"), cfg.vocab_size, Wp).contiguous(), pos=pos)


class RandomTensors:
    """Random checkpoint tensors by name, each from its own seed (independent of the order they are asked for).
    Linears are N(0, std) with std = gain / sqrt(inputs); the other parameters get values a trained model could have:
    decays between a few and a few thousand tokens, gates around one half to one."""

    def __init__(self, cfg: LayeredConfig, seed: int = 0, device="cpu", dtype=torch.bfloat16, gain: float = 1.0,
                 embed_std: float = 1.0):
        self.cfg, self.seed, self.device, self.dtype, self.gain = cfg, seed, torch.device(device), dtype, gain
        self.embed_std = embed_std
        self.shapes = cfg.tensor_shapes()
        self.index = {n: i for i, n in enumerate(self.shapes)}

    def names(self):
        return list(self.shapes)

    def __call__(self, name: str) -> torch.Tensor:
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 1000003 + self.index[name])

        def normal(mean, std):
            t = torch.empty(shape, dtype=torch.float32, device=self.device)
            return t.normal_(0.0, 1.0, generator=g).mul_(std).add_(mean)

        if name == "embed":
            t = normal(0.0, self.embed_std)
        elif name == "pos":
            t = normal(0.0, 0.5 * self.embed_std)
        elif name.endswith("A_log"):
            t = normal(-0.5, 1.0)
        elif name.endswith(("dt_bias", ".dt.b")):
            t = normal(-2.5, 1.0)
        elif name.endswith(".conv"):
            t = normal(0.0, 0.4)
            t[..., -1] += 0.7
        elif name.endswith("canon1"):
            t = normal(0.0, 0.3)
        elif name.endswith(("norm1.b", "norm2.b", "final.norm.b", ".conv.b", ".q.b", ".k.b", ".v.b", ".o.b", ".up.b", ".down.b",
                            ".router.b")):
            t = normal(0.0, 0.2)
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = normal(0.0, 0.1)
        elif name.endswith(".talk"):
            t = normal(0.0, 0.3) + torch.eye(shape[0], device=self.device)
        elif name.endswith(".shift"):
            t = normal(0.4, 0.3)
        elif name.endswith(".temp"):
            t = normal(1.0, 0.3)
        elif name.endswith((".vmix", ".D")):
            t = normal(0.5, 0.2)
        elif name.endswith(("rg1.b", "rg2.b")):
            t = normal(0.7, 0.5)
        elif "norm" in name:
            t = normal(1.0, 0.1)
        else:
            t = normal(0.0, self.gain / shape[-1] ** 0.5)
        return t.to(torch.bfloat16).to(self.dtype)


def random_weights(cfg: LayeredConfig, device="cpu", dtype=torch.bfloat16, seed: int = 0, gain: float = 1.0
                   ) -> LayeredWeights:
    return pack_weights(cfg, RandomTensors(cfg, seed, device, dtype, gain))
