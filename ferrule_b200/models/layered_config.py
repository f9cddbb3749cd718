"""Layer-list models: every layer names its own mixer and feed-forward, with its own sizes.

`LayeredConfig` is a sequence of `LayerSpec`s over one residual width.  A layer is parallel: one RMS norm feeds the
mixer and the feed-forward, both results are gated element by element and added to a 32-bit residual stream.  Mixers:

  LatentMixer   latent attention without positions: keys and values are linear images of one normalised latent row per
                token (the only thing cached), causal softmax, one output gate per head
  DeltaMixer    gated delta rule: short causal convolutions, unit-norm queries and keys, one decay per key channel,
                a [dim, vdim] state per head, gated per-head output norm

Feed-forward: routed experts (softmax scores, group-limited top-k) or none.

`from_layer_list` reads the `config.json` of the Gitozen architecture, whose checkpoints are stored this way.
"""
from __future__ import annotations

import json
from dataclasses import asdict, dataclass, replace
from pathlib import Path
from typing import Dict, Optional, Tuple, Union


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float

    kind = "latent_attention"

    @property
    def row_dim(self) -> int:
        """Latent features per cache row, padded to what the attention kernels take."""
        return pad_to(self.kv_rank, 64)


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int = 16           # inner width of the two low-rank projections (a checkpoint's tensors say which)
    gate_rank: int = 16

    kind = "channel_delta"

    @property
    def channels(self) -> int:
        """Convolved channels: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1


Mixer = Union[LatentMixer, DeltaMixer]


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    mlp: Optional[MoeSpec]


@dataclass(frozen=True)
class LayeredConfig:
    vocab_size: int
    width: int
    layers: Tuple[LayerSpec, ...]
    norm_eps: float = 1e-6
    logit_softcap: float = 0.0          # 0: none
    name: str = "gitozen"
    eos_token_id: int = -1              # the architecture names no special tokens
    bos_token_id: int = -1
    max_position: int = 1 << 20         # no positional encoding: the cache is the only limit

    n_mtp_layers = 0
    attn_sink = False

    @property
    def n_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def width_pad(self) -> int:
        """Row width of activation buffers and weight rows (padding columns are zero)."""
        return pad_to(self.width, 8)

    @property
    def latent_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, LatentMixer))

    @property
    def delta_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, DeltaMixer))

    @property
    def kv_row_dim(self) -> int:
        """Row width of the latent pool: the widest latent of any layer."""
        return max((self.layers[i].mixer.row_dim for i in self.latent_layers), default=64)

    @property
    def n_heads(self) -> int:
        return max(l.mixer.heads for l in self.layers)

    @property
    def n_routed_experts(self) -> int:
        return max((l.mlp.experts for l in self.layers if l.mlp), default=0)

    @property
    def topk(self) -> int:
        return max((l.mlp.top for l in self.layers if l.mlp), default=0)

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Checkpoint tensor name -> shape, in storage order."""
        W = self.width
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, W)}
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            x = p + "mix."
            out[p + "norm1"] = ()
            if isinstance(m, LatentMixer):
                out.update({x + "q": (m.heads * m.dim, W), x + "dkv": (m.kv_rank, W), x + "dkv.norm": (m.kv_rank,),
                            x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (m.heads * m.vdim, m.kv_rank),
                            x + "g": (m.heads, W), x + "o": (W, m.heads * m.vdim)})
            else:
                nk, nv = m.kv_heads * m.dim, m.heads * m.vdim
                out.update({x + "q": (nk, W), x + "q.conv": (nk, m.taps), x + "k": (nk, W), x + "k.conv": (nk, m.taps),
                            x + "v": (nv, W), x + "v.conv": (nv, m.taps), x + "b": (m.heads, W), x + "A_log": (m.heads,),
                            x + "norm": (m.vdim,), x + "a1": (m.decay_rank, W), x + "a2": (m.heads * m.dim, m.decay_rank),
                            x + "dt_bias": (m.heads * m.dim,), x + "g1": (m.gate_rank, W), x + "g2": (nv, m.gate_rank),
                            x + "o": (W, nv)})
            if l.mlp:
                for e in range(l.mlp.experts):
                    q = f"{p}mlp.e{e}."
                    out.update({q + "gate": (l.mlp.ff, W), q + "up": (l.mlp.ff, W), q + "down": (W, l.mlp.ff)})
                out[p + "mlp.router"] = (l.mlp.experts, W)
            out.update({p + "rg1": (W, W), p + "rg1.b": (W,)})
            if l.mlp:
                out.update({p + "rg2": (W, W), p + "rg2.b": (W,)})
        out.update({"final.norm": (), "head": (self.vocab_size, W)})
        return out

    def param_count(self) -> int:
        total = 0
        for shape in self.tensor_shapes().values():
            n = 1
            for s in shape:
                n *= s
            total += n
        return total

    def to_dict(self) -> dict:
        return asdict(self)

    def with_(self, **kw) -> "LayeredConfig":
        return replace(self, **kw)


def _positive(**kw) -> None:
    for k, v in kw.items():
        if v <= 0:
            raise ValueError(f"{k} must be positive, got {v}")


def _mixer(kind: str, m: dict) -> Mixer:
    if kind == LatentMixer.kind:
        x = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]))
        _positive(heads=x.heads, dim=x.dim, vdim=x.vdim, kv_rank=x.kv_rank)
        return x
    if kind == DeltaMixer.kind:
        x = DeltaMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        _positive(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, conv=x.taps)
        if x.heads % x.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        return x
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp(m: Optional[dict]) -> Optional[MoeSpec]:
    if m is None:
        return None
    if m.get("kind", "moe") != "moe":
        raise ValueError(f"unknown feed-forward kind {m.get('kind')!r}")
    r = m["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    x = MoeSpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), int(g["count"]), int(g["keep"]))
    _positive(experts=x.experts, top=x.top, ff=x.ff, groups=x.groups, keep=x.keep)
    if x.experts % x.groups or x.keep > x.groups or x.top > x.experts // x.groups * x.keep:
        raise ValueError("router groups do not fit the expert count")
    return x


def from_layer_list(source) -> LayeredConfig:
    """`config.json` (a path, its directory, or the parsed object) -> LayeredConfig.  The inner widths of the delta
    mixers' low-rank projections are not in the file; the loader takes them from the tensors."""
    if isinstance(source, dict):
        c = source
    else:
        p = Path(source)
        c = json.loads((p / "config.json" if p.is_dir() else p).read_text())
    layers = tuple(LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in c["layers"])
    if not layers:
        raise ValueError("a model needs at least one layer")
    cfg = LayeredConfig(int(c["vocab"]), int(c["width"]), layers, float(c["norm"]["eps"]),
                        float(c.get("logit_softcap") or 0.0), name=str(c.get("architecture", "gitozen")).lower())
    _positive(vocab=cfg.vocab_size, width=cfg.width)
    return cfg


def to_layer_list(cfg: LayeredConfig) -> dict:
    """The `config.json` object of a configuration."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, LatentMixer):
            mx = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale}
        else:
            mx = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
        ff = None
        if l.mlp:
            ff = {"kind": "moe", "expert": {"ff": l.mlp.ff}, "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
            if l.mlp.groups > 1:
                ff["router"]["groups"] = {"count": l.mlp.groups, "keep": l.mlp.keep}
        layers.append({"type": m.kind, "mixer": mx, "mlp": ff})
    return {"architecture": "Gitozen", "vocab": cfg.vocab_size, "width": cfg.width, "norm": {"eps": cfg.norm_eps},
            "logit_softcap": cfg.logit_softcap or None, "layers": layers}


def tiny_gitozen() -> LayeredConfig:
    """Small shape for fixtures and the command line: both mixers, grouped heads, a layer without feed-forward."""
    moe = MoeSpec(experts=6, top=2, ff=40, groups=3, keep=2)
    lat = LatentMixer(heads=3, dim=24, vdim=16, kv_rank=40, scale=0.2)
    dlt = DeltaMixer(heads=4, kv_heads=2, dim=16, vdim=24, taps=3, decay_rank=12, gate_rank=8)
    return LayeredConfig(vocab_size=512, width=96, layers=(LayerSpec(dlt, moe), LayerSpec(lat, moe), LayerSpec(dlt, None),
                                                           LayerSpec(lat, moe)), logit_softcap=20.0)


def gitozen_lite(n_layers: int = 27) -> LayeredConfig:
    """Layers of a served model's size (the widths of DeepSeek-V2-Lite): three of four mixers are delta mixers."""
    moe = MoeSpec(experts=64, top=6, ff=1408, groups=8, keep=3)
    lat = LatentMixer(heads=16, dim=128, vdim=128, kv_rank=512, scale=128 ** -0.5)
    dlt = DeltaMixer(heads=16, kv_heads=16, dim=128, vdim=128, taps=4, decay_rank=128, gate_rank=128)
    return LayeredConfig(vocab_size=102400, width=2048, layers=tuple(LayerSpec(lat if i % 4 == 3 else dlt, moe)
                                                                     for i in range(n_layers)),
                         logit_softcap=30.0, name="gitozen-lite")


def gitozen_latent_lite(n_layers: int = 27) -> LayeredConfig:
    """The same with latent attention in every layer: the layer stack closest to DeepSeek-V2-Lite's."""
    base = gitozen_lite(n_layers)
    lat = LayerSpec(LatentMixer(heads=16, dim=128, vdim=128, kv_rank=512, scale=128 ** -0.5), base.layers[0].mlp)
    return base.with_(layers=(lat,) * n_layers, name="gitozen-latent-lite")


PRESETS = {"tiny-gitozen": tiny_gitozen, "gitozen-lite": gitozen_lite, "gitozen-latent-lite": gitozen_latent_lite}
