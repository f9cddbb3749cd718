"""Weight image of a layer-list model, packed once at load time into what the kernels read.

Every linear that reads the layer's normalised input is one row block of a single matrix `w_in`, so a layer starts with
one GEMM; blocks begin at multiples of 8 columns of its output:

  latent layer  q (heads x dim, each head padded to 8) | dkv | head gates | residual gate 1 | residual gate 2
  delta layer   q | k | v | decay low rank | gate low rank | beta | residual gate 1 | residual gate 2

The second halves of the delta layer's two low-rank projections are one block-diagonal matrix `w_ag` (fp32 output:
decay pre-activations and output-gate pre-activations).  Keys and values of a latent layer are absorbed: `w_uk_t` maps a
query head to the latent space, `w_uv` maps the attention output (a latent row per head) to the head's value.  Widths
are padded with zeros to multiples of 8 (latents to multiples of 64), so every size takes the same kernels.

Constants that enter norms, gates and recurrences are fp32 tensors; everything else has the model's dtype.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional

import torch

from .layered_config import DeltaMixer, LatentMixer, LayeredConfig, LayerSpec, MoeSpec, pad_to

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
    # latent attention
    w_uk_t: Optional[torch.Tensor] = None    # [heads, row_dim, dim_pad]
    w_uv: Optional[torch.Tensor] = None      # [heads, vdim_pad, row_dim]
    kv_norm: Optional[torch.Tensor] = None   # fp32 [row_dim]
    # delta rule
    w_ag: Optional[torch.Tensor] = None      # [heads * dim | heads * vdim, low ranks]
    off_gate: int = 0
    conv: Optional[torch.Tensor] = None      # fp32 [taps, channels]
    a_neg: Optional[torch.Tensor] = None     # fp32 [heads] = -exp(A_log)
    dt_bias: Optional[torch.Tensor] = None   # fp32 [heads * dim]
    o_norm: Optional[torch.Tensor] = None    # fp32 [vdim]


@dataclass
class LayerImage:
    spec: LayerSpec
    norm: torch.Tensor                       # fp32 [1]: one number for all coordinates
    mixer: MixerImage
    rg1_b: torch.Tensor                      # fp32 [width_pad]
    rg2_b: Optional[torch.Tensor] = None
    router_w: Optional[torch.Tensor] = None  # [experts, width_pad]
    e_w13: Optional[torch.Tensor] = None     # [experts, 2 * ff_pad, width_pad]
    e_w2: Optional[torch.Tensor] = None      # [experts, width_pad, ff_pad]


@dataclass
class LayeredWeights:
    cfg: LayeredConfig
    embed: torch.Tensor                      # [vocab, width_pad]
    layers: List[LayerImage]
    final_norm: torch.Tensor                 # fp32 [1]
    lm_head: torch.Tensor                    # [vocab, width_pad]
    mtp: list = field(default_factory=list)  # the architecture has no proposal stages
    weight_format: str = "bf16"

    def nbytes(self) -> int:
        total = sum(t.numel() * t.element_size() for t in (self.embed, self.final_norm, self.lm_head))
        for l in self.layers:
            for holder in (l, l.mixer):
                total += sum(t.numel() * t.element_size() for t in vars(holder).values() if isinstance(t, torch.Tensor))
        return total


class _Blocks:
    """Stacks row blocks, each starting at a multiple of 8."""

    def __init__(self, cols: int):
        self.cols, self.rows, self.off, self.parts = cols, 0, {}, []

    def add(self, name: str, w: torch.Tensor) -> None:
        n = pad_to(w.shape[0], 8)
        self.off[name] = self.rows
        self.parts.append(_pad(w, n, self.cols))
        self.rows += n

    def matrix(self) -> torch.Tensor:
        return torch.cat(self.parts, 0).contiguous()


def _pack_latent(m: LatentMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp, DL = cfg.width_pad, cfg.kv_row_dim
    dp, vp = pad_to(m.dim, 8), pad_to(m.vdim, 8)
    q = _pad(get(p + "q").view(m.heads, m.dim, cfg.width), m.heads, dp, Wp)
    b.add("q", q.reshape(m.heads * dp, Wp))
    b.add("dkv", get(p + "dkv"))
    b.add("g", get(p + "g"))
    uk = get(p + "uk").view(m.heads, m.dim, m.kv_rank).transpose(1, 2)
    uv = get(p + "uv").view(m.heads, m.vdim, m.kv_rank)
    o = _pad(get(p + "o").view(cfg.width, m.heads, m.vdim), Wp, m.heads, vp)
    return MixerImage(None, b.off, o.reshape(Wp, m.heads * vp).contiguous(),
                      w_uk_t=_pad(uk, m.heads, DL, dp).contiguous(), w_uv=_pad(uv, m.heads, vp, DL).contiguous(),
                      kv_norm=_pad(get(p + "dkv.norm").float(), DL).contiguous())


def _pack_delta(m: DeltaMixer, p: str, get: GetTensor, cfg: LayeredConfig, b: _Blocks) -> MixerImage:
    Wp = cfg.width_pad
    nk, nv, nd = m.kv_heads * m.dim, m.heads * m.vdim, m.heads * m.dim
    for name in ("q", "k", "v", "a1", "g1", "b"):
        b.add(name, get(p + name))
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


def _pack_moe(s: MoeSpec, p: str, get: GetTensor, cfg: LayeredConfig, img: LayerImage) -> None:
    Wp, fp = cfg.width_pad, pad_to(s.ff, 8)
    img.router_w = _pad(get(p + "router"), s.experts, Wp).contiguous()
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
    layers: List[LayerImage] = []
    for i, spec in enumerate(cfg.layers):
        p = f"l{i}."
        b = _Blocks(Wp)
        pack = _pack_latent if isinstance(spec.mixer, LatentMixer) else _pack_delta
        mx = pack(spec.mixer, p + "mix.", get, cfg, b)
        img = LayerImage(spec, get(p + "norm1").float().reshape(1).contiguous(), mx,
                         _pad(get(p + "rg1.b").float(), Wp).contiguous())
        b.add("rg1", get(p + "rg1"))
        if spec.mlp is not None:
            b.add("rg2", get(p + "rg2"))
            img.rg2_b = _pad(get(p + "rg2.b").float(), Wp).contiguous()
            _pack_moe(spec.mlp, p + "mlp.", get, cfg, img)
        mx.w_in = b.matrix()
        layers.append(img)
    return LayeredWeights(cfg, _pad(get("embed"), cfg.vocab_size, Wp).contiguous(), layers,
                          get("final.norm").float().reshape(1).contiguous(),
                          _pad(get("head"), cfg.vocab_size, Wp).contiguous())


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
        elif name.endswith("A_log"):
            t = normal(-0.5, 1.0)
        elif name.endswith("dt_bias"):
            t = normal(-2.5, 1.0)
        elif name.endswith(".conv"):
            t = normal(0.0, 0.4)
            t[..., -1] += 0.7
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
