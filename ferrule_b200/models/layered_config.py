"""Layer-list models: every layer names its own mixer and feed-forward, with its own sizes.

`LayeredConfig` is a sequence of `LayerSpec`s over one residual width (a 32-bit residual stream) and a block form:

  PARALLEL_GATED  one RMS norm feeds the mixer and the feed-forward, both results are gated element by element
  OUTPUT_NORM     the mixer, then the feed-forward, each reading the stream itself; a norm (layer norm with weight and
                  bias) on the sublayer's output before it is added.  With `canon_taps` the mixer reads the stream plus
                  a short causal convolution of it
  SANDWICH_NORM   the mixer, then the feed-forward, each between two grouped RMS norms: one on its input, one on its
                  output before that is added to the stream
  PRE_NORM        the mixer, then the feed-forward, each behind an RMS norm of its own.  With `token_shift` the mixer's
                  normalised input moves towards the previous token's, element by element

`loop` runs a range of layers several times in a row with the same weights: `runs` is the sequence of layers a token
passes, and every run has its own cache plane and state.  The embedding is added to the stream again before every pass
but the first.  A layer may instead name another one whose weights it uses (`weights_of`); it is a layer of its own in every
other respect.

Mixers:

  LatentMixer     latent attention: keys and values are linear images of one normalised latent row per token (the only
                  thing cached), causal softmax, one output gate per head; optionally queries through a latent of their own,
                  a rotated key part shared by the heads, a sliding window
  AttentionMixer  grouped-query attention inside position-aligned chunks: query and key norm over the whole
                  projection, partial rotation, value norm, values mixed with those of the first mixing layer
  WindowMixer     grouped-query attention over a sliding window (and kept first tokens) with query and key norm per head:
                  optionally projection biases, keys that double as values, a distance bias per head, scores mixed
                  across heads, an output gate, two score maps whose outputs are subtracted, rotation, a soft cap on the
                  scores, mean keys and values of the blocks before the window, softmax weights mixed across heads
  DeltaMixer      gated delta rule: short causal convolutions, unit-norm queries and keys, one decay per key channel
                  or per head, a [dim, vdim] state per head, gated per-head output norm
  MambaMixer      selective scan: short causal convolution, per-channel step sizes, an [inner, state] diagonal recurrence
  Mamba2Mixer     scan with one decay per head: short causal convolution, a [state, vdim] matrix per head, gated group norm

Feed-forward: routed experts (softmax scores, group-limited top-k; optionally clamped inputs, a gated shared expert), dense
with GELU or gated with tanh GELU, or none.

`from_layer_list` reads the `config.json` of the architectures whose checkpoints are stored this way: Gitozen
(PARALLEL_GATED; latent attention, delta rule with channel decays, experts), Supisun (OUTPUT_NORM; chunked attention,
selective scan, delta rule with head decays, dense feed-forward, learned positions), Vedadra (SANDWICH_NORM; window
attention with mixed heads, differential window attention, gated dense feed-forward, looped layers) and Vogunex (PRE_NORM with
token shift; window attention with pooled blocks and mixed weights, rotated latent attention, head-decay scan, dense
feed-forward or experts with a shared one, shared weights).
"""
from __future__ import annotations

import json
from dataclasses import asdict, dataclass, replace
from pathlib import Path
from typing import Callable, Dict, Optional, Tuple, Union


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    q_rank: int = 0                # > 0: queries are an image of a normalised latent of this width
    rot_dim: int = 0               # rotated dimensions per head (neighbours paired) beside the `dim` others
    rot_base: float = 0.0
    window: int = 0                # a query sees itself and the window - 1 tokens before it (0: all of them)

    kind = "latent_attention"

    @property
    def split_row(self) -> bool:
        """Whether the rotated part has feature blocks of its own behind the latent's, which the values do not span."""
        return 0 < self.rot_dim <= 64 and self.kv_rank <= 512 < pad_to(self.kv_rank + self.rot_dim, 64)

    @property
    def rot_offset(self) -> int:
        """Column of the rotated part in a cache row."""
        return 512 if self.split_row else self.kv_rank

    @property
    def row_dim(self) -> int:
        """Features per cache row, padded to what the attention kernels take."""
        return 576 if self.split_row else pad_to(self.kv_rank + self.rot_dim, 64)

    @property
    def value_dim(self) -> int:
        """Columns of a cache row that the tensor-core kernels take as its value."""
        return 512 if self.split_row else self.row_dim


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                     # a query sees the keys of its own chunk of positions only
    rot_base: float
    rot_dims: int                  # leading dimensions of a head that are rotated (halves paired)
    v_mix: bool = False

    kind = "attention"
    maps = 1
    window = keep_first = pool = 0
    softcap = score_bound = 0.0
    shared_keys = shared_values = scaled_queries = False

    @property
    def dim_pad(self) -> int:
        return pad_to(self.dim, 8)

    @property
    def vdim_pad(self) -> int:
        return pad_to(self.vdim, 8)

    @property
    def value_width(self) -> int:
        return self.vdim_pad

    @property
    def v_offset(self) -> int:
        """First value column of a cache row: [kv_heads][dim_pad] keys | [kv_heads][vdim_pad] values."""
        return self.kv_heads * self.dim_pad

    @property
    def row_dim(self) -> int:
        return pad_to(self.kv_heads * (self.dim_pad + self.vdim_pad), 8)

    @property
    def key_width(self) -> int:
        """Width of a query row as the attention kernels take it."""
        return self.dim_pad


@dataclass(frozen=True)
class WindowMixer:
    """Position i sees j <= i with i - j < window or j < keep_first.  `maps` = 2: two query / key pairs per head over the
    same values; the head's output is rms(a1 - lambda a2) * (1 - diff).  `mix_heads`: score_h <- sum_g T[h, g] score_g."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    keep_first: int = 0
    maps: int = 1
    diff: float = 0.0              # maps = 2: base of lambda
    biases: str = ""               # projections with a bias: letters of q, k, v and o
    tied_values: bool = False      # the values are the projected keys (before their norm)
    head_temps: bool = False       # one factor per head on its scores
    distance_bias: bool = False    # score_h -= 2^(-8 (h + 1) / heads) (i - j)
    mix_heads: bool = False
    gate: bool = False             # output multiplied by sigmoid(W_g h), element by element
    norm_weights: bool = True      # on the query and key norm
    rot_base: float = 0.0
    rot_dims: int = 0              # leading dimensions of a head that are rotated (halves paired)
    softcap: float = 0.0           # score <- softcap tanh(score / softcap)
    pool: int = 0                  # every block of `pool` tokens wholly before the window is seen as its mean key and value
    mix_weights: bool = False      # weight_h <- sum_g T[h, g] weight_g, after the softmax

    chunk = 0
    scaled_queries = True          # the scale is part of the queries the attention kernels read

    @property
    def kind(self) -> str:
        return "attention" if self.maps == 1 else "attention_2"

    @property
    def dim_pad(self) -> int:
        return pad_to(self.dim, 8)

    @property
    def vdim_pad(self) -> int:
        return pad_to(self.vdim, 8)

    @property
    def shared_keys(self) -> bool:
        """Every query row meets the keys of all kv heads side by side: sum_g T[h, g] q_g . k_kv(g) is one product of a
        mixed query with the concatenated keys."""
        return self.mix_heads

    @property
    def score_bound(self) -> float:
        """No scaled score is larger (0: unknown): without norm weights queries and keys have the length sqrt(dim), means of
        keys are not longer.  (Rounding them to bf16 adds at most a hundredth.)"""
        return 0.0 if self.norm_weights or self.mix_heads else 1.01 * self.dim * abs(self.scale)

    @property
    def shared_values(self) -> bool:
        """Every query row meets the values of all kv heads side by side: sum_g T[h, g] w_g . v_kv(h) needs every head's
        weights on the values of every kv head."""
        return self.mix_weights

    @property
    def value_width(self) -> int:
        """Value columns of a query row's output."""
        return (self.kv_heads if self.shared_values else 1) * self.vdim_pad

    @property
    def key_width(self) -> int:
        return (self.kv_heads if self.shared_keys else self.maps) * self.dim_pad

    @property
    def v_offset(self) -> int:
        """First value column of a cache row: [kv_heads][maps][dim_pad] keys | [kv_heads][vdim_pad] values."""
        return self.kv_heads * self.maps * self.dim_pad

    @property
    def row_dim(self) -> int:
        return pad_to(self.v_offset + self.kv_heads * self.vdim_pad, 8)


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int = 16           # inner width of the two low-rank projections (a checkpoint's tensors say which);
    gate_rank: int = 16            # 0: one full projection
    head_decay: bool = False       # one decay per head instead of one per key channel
    gate: str = "sigmoid"          # output gate's activation: sigmoid or silu

    @property
    def kind(self) -> str:
        return "delta" if self.head_decay else "channel_delta"

    @property
    def low_rank(self) -> bool:
        return self.decay_rank > 0

    @property
    def channels(self) -> int:
        """Convolved channels: q | k | v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class MambaMixer:
    inner: int
    state: int
    dt_rank: int
    taps: int

    kind = "mamba1"
    heads = 1

    @property
    def inner_pad(self) -> int:
        return pad_to(self.inner, 8)


@dataclass(frozen=True)
class Mamba2Mixer:
    """S <- exp(-exp(A) dt) S + dt B x^T, y = S^T C + D x per head (a head of group g reads B_g and C_g); the output is
    rms(y silu(z)) in `norm_groups` equal parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    norm_groups: int = 1

    kind = "mamba2"

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def inner_pad(self) -> int:
        return pad_to(self.inner, 8)

    @property
    def bc_pad(self) -> int:
        return pad_to(self.groups * self.state, 8)

    @property
    def channels(self) -> int:
        """Convolved channels: x | B | C, each padded."""
        return self.inner_pad + 2 * self.bc_pad


@dataclass(frozen=True)
class MoeSpec:
    """Expert: W_down (g sigmoid(alpha g) (u + shift)) with g = min(W_gate x, limit), u = clamp(W_up x, +-limit)."""
    experts: int
    top: int
    ff: int
    groups: int = 1
    keep: int = 1
    limit: float = 0.0             # 0: not clamped
    alpha: float = 1.0
    shift: float = 0.0
    renormalize: bool = False      # the weights of the chosen experts sum to one
    router_bias: bool = False      # on the logits
    shared_ff: int = 0             # > 0: an expert of this width for every token, times sigmoid(W_sg x)
    shared_limit: float = 0.0


@dataclass(frozen=True)
class DenseSpec:
    """W_down gelu(W_up x), the exact (error-function) GELU; gated: W_down (gelu(W_gate x) * W_up x), the tanh form."""
    ff: int
    gated: bool = False
    biases: bool = False

    experts = top = 0


Mixer = Union[LatentMixer, AttentionMixer, WindowMixer, DeltaMixer, MambaMixer, Mamba2Mixer]

PARALLEL_GATED = "parallel_gated"
OUTPUT_NORM = "output_norm"
SANDWICH_NORM = "sandwich_norm"
PRE_NORM = "pre_norm"


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    mlp: Union[MoeSpec, DenseSpec, None]
    weights_of: int = -1           # the layer whose tensors this one uses, -1: its own


@dataclass(frozen=True)
class Loop:
    """Layers start .. stop - 1 run `times` times in a row."""
    start: int
    stop: int
    times: int


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
    max_position: int = 1 << 20         # without positional encoding the cache is the only limit
    block: str = PARALLEL_GATED
    canon_taps: int = 0                 # OUTPUT_NORM: taps of the mixers' input convolution, 0: none
    learned_positions: bool = False     # a table of `max_position` vectors is added to the embedding
    norm_groups: int = 1                # SANDWICH_NORM: parts of a row with an RMS norm of their own
    loop: Optional[Loop] = None         # SANDWICH_NORM
    embed_scale: float = 1.0            # PRE_NORM: factor on the embedding
    token_shift: bool = False           # PRE_NORM: the mixers' inputs move towards the previous token's

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
    def runs(self) -> Tuple[int, ...]:
        """Layers in the order a token passes them."""
        n, l = len(self.layers), self.loop
        if l is None:
            return tuple(range(n))
        return (*range(l.start), *(tuple(range(l.start, l.stop)) * l.times), *range(l.stop, n))

    @property
    def pass_starts(self) -> Tuple[int, ...]:
        """Runs that begin a pass of the loop other than the first."""
        l = self.loop
        return () if l is None else tuple(l.start + k * (l.stop - l.start) for k in range(1, l.times))

    def owner(self, layer: int) -> int:
        """The layer whose tensors `layer` uses."""
        w = self.layers[layer].weights_of
        return layer if w < 0 else w

    def first_layers(self, n: int) -> "LayeredConfig":
        """The same model cut off behind its first `n` layers."""
        l = self.loop
        if l is not None:
            l = Loop(l.start, min(l.stop, n), l.times) if l.start < n else None
        return replace(self, layers=self.layers[:n], loop=l)

    def cycled(self, n: int) -> "LayeredConfig":
        """A model of `n` layers that repeats this one's."""
        whole = replace(self, layers=tuple(self.layers[i % len(self.layers)] for i in range(n)))
        return whole.first_layers(n)

    @property
    def latent_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, LatentMixer))

    @property
    def delta_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, DeltaMixer))

    @property
    def attention_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, AttentionMixer))

    @property
    def window_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, WindowMixer))

    @property
    def mamba_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, MambaMixer))

    @property
    def mamba2_layers(self) -> Tuple[int, ...]:
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, Mamba2Mixer))

    @property
    def cache_layers(self) -> Tuple[int, ...]:
        """Layers with a row per token in the paged pool."""
        return tuple(i for i, l in enumerate(self.layers) if isinstance(l.mixer, (LatentMixer, AttentionMixer, WindowMixer)))

    @property
    def cache_runs(self) -> Tuple[int, ...]:
        """Runs with a plane of their own in the paged pool, in the order of the planes."""
        cached = set(self.cache_layers)
        return tuple(r for r, i in enumerate(self.runs) if i in cached)

    @property
    def first_value_layer(self) -> int:
        """The layer whose values the later value-mixing layers mix in, -1: none."""
        return next((i for i in self.attention_layers if self.layers[i].mixer.v_mix), -1)

    @property
    def kv_row_dim(self) -> int:
        """Row width of the paged pool: the widest row of any layer."""
        return max((self.layers[i].mixer.row_dim for i in self.cache_layers), default=64)

    def plane_dim(self, layer: int) -> int:
        """Row width of a layer's planes: latent layers their own, the others the widest of them."""
        if isinstance(self.layers[layer].mixer, LatentMixer):
            return self.layers[layer].mixer.row_dim
        return max(self.layers[i].mixer.row_dim for i in self.cache_layers if i not in self.latent_layers)

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
        gated = self.block == PARALLEL_GATED
        out: Dict[str, Tuple[int, ...]] = {"embed": (self.vocab_size, W)}
        if self.learned_positions:
            out["pos"] = (self.max_position, W)
        for i, l in enumerate(self.layers):
            p, m = f"l{self.owner(i)}.", l.mixer
            x = p + "mix."
            if gated:
                out[p + "norm1"] = ()
            elif self.block == PRE_NORM:
                names = ("norm1",) + (("norm2",) if l.mlp else ()) + (("shift",) if self.token_shift else ())
                out.update({p + n: (W,) for n in names})
            elif self.block == SANDWICH_NORM:
                names = ("norm1", "norm2", "norm1b", "norm2b") if l.mlp else ("norm1", "norm1b")
                out.update({p + n: (W,) for n in names})
            else:
                for n in ("norm1", "norm2")[:2 if l.mlp else 1]:
                    out.update({p + n: (W,), p + n + ".b": (W,)})
            if isinstance(m, LatentMixer):
                if m.q_rank:
                    out.update({x + "dq": (m.q_rank, W), x + "dq.norm": (m.q_rank,),
                                x + "uq": (m.heads * (m.dim + m.rot_dim), m.q_rank)})
                else:
                    out[x + "q"] = (m.heads * (m.dim + m.rot_dim), W)
                out.update({x + "dkv": (m.kv_rank + m.rot_dim, W), x + "dkv.norm": (m.kv_rank,),
                            x + "uk": (m.heads * m.dim, m.kv_rank), x + "uv": (m.heads * m.vdim, m.kv_rank),
                            x + "g": (m.heads, W), x + "o": (W, m.heads * m.vdim)})
            elif isinstance(m, AttentionMixer):
                nq, nk, nv = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
                out.update({x + "q": (nq, W), x + "k": (nk, W), x + "v": (nv, W), x + "q.norm": (nq,), x + "k.norm": (nk,)})
                if m.v_mix:
                    out[x + "vmix"] = ()
                out[x + "o"] = (W, m.heads * m.vdim)
            elif isinstance(m, WindowMixer):
                nq, nk, nv = m.heads * m.maps * m.dim, m.kv_heads * m.maps * m.dim, m.kv_heads * m.vdim
                for name, n in (("q", nq), ("k", nk)) + (() if m.tied_values else (("v", nv),)):
                    out[x + name] = (n, W)
                    if name in m.biases:
                        out[x + name + ".b"] = (n,)
                if m.norm_weights:
                    out.update({x + "q.norm": (m.dim,), x + "k.norm": (m.dim,)})
                if m.maps == 2:
                    out.update({x + n: (m.dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
                if m.mix_heads or m.mix_weights:
                    out[x + "talk"] = (m.heads, m.heads)
                if m.head_temps:
                    out[x + "temp"] = (m.heads,)
                if m.gate:
                    out[x + "g"] = (m.heads * m.vdim, W)
                out[x + "o"] = (W, m.heads * m.vdim)
                if "o" in m.biases:
                    out[x + "o.b"] = (W,)
            elif isinstance(m, Mamba2Mixer):
                c = m.inner + 2 * m.groups * m.state
                out.update({x + "in": (m.inner + c + m.heads, W), x + "conv": (c, m.taps), x + "conv.b": (c,),
                            x + "dt_bias": (m.heads,), x + "A_log": (m.heads,), x + "D": (m.heads,), x + "norm": (m.inner,),
                            x + "o": (W, m.inner)})
            elif isinstance(m, MambaMixer):
                out.update({x + "in": (2 * m.inner, W), x + "conv": (m.inner, m.taps), x + "conv.b": (m.inner,),
                            x + "x": (m.dt_rank + 2 * m.state, m.inner), x + "dt": (m.inner, m.dt_rank),
                            x + "dt.b": (m.inner,), x + "A_log": (m.inner, m.state), x + "D": (m.inner,),
                            x + "o": (W, m.inner)})
            else:
                nk, nv = m.kv_heads * m.dim, m.heads * m.vdim
                out.update({x + "q": (nk, W), x + "q.conv": (nk, m.taps), x + "k": (nk, W), x + "k.conv": (nk, m.taps),
                            x + "v": (nv, W), x + "v.conv": (nv, m.taps), x + "b": (m.heads, W), x + "A_log": (m.heads,),
                            x + "norm": (m.vdim,)})
                decays = m.heads if m.head_decay else m.heads * m.dim
                if m.low_rank:
                    out.update({x + "a1": (m.decay_rank, W), x + "a2": (decays, m.decay_rank), x + "dt_bias": (decays,),
                                x + "g1": (m.gate_rank, W), x + "g2": (nv, m.gate_rank)})
                else:
                    out.update({x + "a": (decays, W), x + "dt_bias": (decays,), x + "g": (nv, W)})
                out[x + "o"] = (W, nv)
            if isinstance(l.mlp, MoeSpec):
                for e in range(l.mlp.experts):
                    q = f"{p}mlp.e{e}."
                    out.update({q + "gate": (l.mlp.ff, W), q + "up": (l.mlp.ff, W), q + "down": (W, l.mlp.ff)})
                out[p + "mlp.router"] = (l.mlp.experts, W)
                if l.mlp.router_bias:
                    out[p + "mlp.router.b"] = (l.mlp.experts,)
                if l.mlp.shared_ff:
                    q, f = p + "mlp.shared.", l.mlp.shared_ff
                    out.update({q + "gate": (f, W), q + "up": (f, W), q + "down": (W, f), q + "sg": (1, W)})
            elif l.mlp:
                if l.mlp.gated:
                    out[p + "mlp.gate"] = (l.mlp.ff, W)
                out.update({p + "mlp.up": (l.mlp.ff, W), p + "mlp.down": (W, l.mlp.ff)})
                if l.mlp.biases:
                    out.update({p + "mlp.up.b": (l.mlp.ff,), p + "mlp.down.b": (W,)})
            if gated:
                out.update({p + "rg1": (W, W), p + "rg1.b": (W,)})
                if l.mlp:
                    out.update({p + "rg2": (W, W), p + "rg2.b": (W,)})
            if self.canon_taps:
                out[p + "canon1"] = (W, self.canon_taps)
        if gated:
            out["final.norm"] = ()
        elif self.block in (SANDWICH_NORM, PRE_NORM):
            out["final.norm"] = (W,)
        else:
            out.update({"final.norm": (W,), "final.norm.b": (W,)})
        out["head"] = (self.vocab_size, W)
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


def _grouped(heads: int, kv_heads: int) -> None:
    if heads % kv_heads:
        raise ValueError("heads must be a multiple of kv_heads")


def _latent(m: dict) -> LatentMixer:
    x = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]))
    _positive(heads=x.heads, dim=x.dim, vdim=x.vdim, kv_rank=x.kv_rank)
    return x


def _rotated_latent(m: dict) -> LatentMixer:
    x = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]), int(m["q_rank"]),
                    int(m["rot_dim"]), float(m["rot"]["base"]), int(m["mask"]["size"]))
    _positive(heads=x.heads, dim=x.dim, vdim=x.vdim, kv_rank=x.kv_rank, q_rank=x.q_rank, rot_dim=x.rot_dim, rot_base=x.rot_base,
              window=x.window)
    if x.rot_dim % 2 or int(m["rot"].get("dims", x.rot_dim)) != x.rot_dim:
        raise ValueError("rot.dims must be rot_dim, an even number")
    return x


def _attention(m: dict) -> AttentionMixer:
    x = AttentionMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]),
                       int(m["mask"]["size"]), float(m["rot"]["base"]), int(m["rot"]["dims"]), bool(m.get("v_mix", False)))
    _positive(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, chunk=x.chunk, rot_base=x.rot_base)
    _grouped(x.heads, x.kv_heads)
    if not 0 <= x.rot_dims <= x.dim or x.rot_dims % 2:
        raise ValueError("rot.dims must be even and at most dim")
    return x


def _window(m: dict, **form) -> WindowMixer:
    mask = m["mask"]
    x = WindowMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), int(mask["size"]),
                    int(mask.get("keep_first") or 0), diff=float(m.get("diff") or 0.0), **form)
    _positive(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, window=x.window)
    _grouped(x.heads, x.kv_heads)
    if x.keep_first < 0:
        raise ValueError("mask.keep_first must not be negative")
    if x.tied_values and x.dim != x.vdim:
        raise ValueError("values that are the keys have the keys' width")
    return x


def _pooled_window(m: dict) -> WindowMixer:
    rot = m["rot"]
    x = _window(m, rot_base=float(rot["base"]), rot_dims=int(rot["dims"]), softcap=float(m.get("softcap") or 0.0),
                pool=int(m["mask"]["pool"]), **POOLED_WINDOW)
    _positive(rot_base=x.rot_base, pool=x.pool)
    if not 0 <= x.rot_dims <= x.dim or x.rot_dims % 2:
        raise ValueError("rot.dims must be even and at most dim")
    if x.softcap < 0:
        raise ValueError("softcap must not be negative")
    return x


def _mamba2(m: dict) -> Mamba2Mixer:
    x = Mamba2Mixer(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["conv"]),
                    int(m.get("norm_groups") or 1))
    _positive(heads=x.heads, vdim=x.vdim, state=x.state, groups=x.groups, conv=x.taps, norm_groups=x.norm_groups)
    if x.heads % x.groups or x.inner % x.norm_groups:
        raise ValueError("groups must divide the heads and norm_groups the inner width")
    return x


def _mamba(m: dict) -> MambaMixer:
    x = MambaMixer(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
    _positive(inner=x.inner, state=x.state, dt_rank=x.dt_rank, conv=x.taps)
    return x


def _delta(m: dict, **form) -> DeltaMixer:
    x = DeltaMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]), **form)
    _positive(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, conv=x.taps)
    _grouped(x.heads, x.kv_heads)
    return x


HEAD_DELTA = dict(decay_rank=0, gate_rank=0, head_decay=True, gate="silu")

TALKING_WINDOW = dict(biases="qko", tied_values=True, head_temps=True, distance_bias=True, mix_heads=True, gate=True)

POOLED_WINDOW = dict(biases="qkv", norm_weights=False, mix_weights=True)


def _dense(m: dict, **form) -> DenseSpec:
    d = DenseSpec(int(m["ff"]), **form)
    _positive(ff=d.ff)
    return d


def _moe(m: dict, **form) -> MoeSpec:
    r = m["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    x = MoeSpec(int(r["experts"]), int(r["top"]), int(m["expert"]["ff"]), int(g["count"]), int(g["keep"]), **form)
    _positive(experts=x.experts, top=x.top, ff=x.ff, groups=x.groups, keep=x.keep)
    if x.experts % x.groups or x.keep > x.groups or x.top > x.experts // x.groups * x.keep:
        raise ValueError("router groups do not fit the expert count")
    return x


CLAMPED_EXPERT = dict(alpha=1.702, shift=1.0, renormalize=True, router_bias=True)


def _shared_moe(m: dict) -> MoeSpec:
    sh = m.get("shared") or {"ff": 0}
    x = _moe(m, limit=float(m["expert"].get("limit") or 0.0), shared_ff=int(sh["ff"]),
             shared_limit=float(sh.get("limit") or 0.0), **CLAMPED_EXPERT)
    if x.limit < 0 or x.shared_limit < 0 or x.shared_ff < 0:
        raise ValueError("limits and sizes of experts must not be negative")
    return x


@dataclass(frozen=True)
class Design:
    """What an architecture's name fixes: its block form, the mixers its layers may name (type -> reader) and the kinds of
    feed-forward (kind -> reader)."""
    name: str
    block: str
    mixers: Dict[str, Callable[[dict], Mixer]]
    feed_forward: Dict[str, Callable[[dict], Union[MoeSpec, DenseSpec]]]


DESIGNS = {d.name: d for d in (
    Design("Gitozen", PARALLEL_GATED, {"latent_attention": _latent, "channel_delta": _delta}, {"moe": _moe}),
    Design("Supisun", OUTPUT_NORM, {"attention": _attention, "mamba1": _mamba, "delta": lambda m: _delta(m, **HEAD_DELTA)},
           {"dense": _dense}),
    Design("Vedadra", SANDWICH_NORM, {"attention": lambda m: _window(m, **TALKING_WINDOW),
                                      "attention_2": lambda m: _window(m, maps=2)},
           {"dense": lambda m: _dense(m, gated=True)}),
    Design("Vogunex", PRE_NORM, {"attention": _pooled_window, "latent_attention": _rotated_latent, "mamba2": _mamba2},
           {"dense": lambda m: _dense(m, biases=True), "moe": _shared_moe}))}

ARCHITECTURES = tuple(n.lower() for n in DESIGNS)       # registry names of the layer-list architectures


def _mlp(m: Optional[dict], readers: dict):
    if m is None:
        return None
    kind = m.get("kind", next(iter(readers)))
    if kind not in readers:
        raise ValueError(f"unknown feed-forward kind {kind!r}")
    return readers[kind](m)


def _shared_weights(layers: list, entries: list) -> list:
    """Layers that use another one's tensors, with the layer that has them."""
    out = list(layers)
    for i, e in enumerate(entries):
        j = e.get("weights_of")
        if j is None:
            continue
        for _ in entries:
            j = int(j)
            if not 0 <= j < len(entries) or j == i:
                raise ValueError(f"layer {i} uses the weights of layer {j}, which is none of the others")
            if entries[j].get("weights_of") is None:
                break
            j = entries[j]["weights_of"]
        else:
            raise ValueError(f"layer {i}: no layer has the weights it uses")
        if layers[j] != layers[i]:
            raise ValueError(f"layer {i} uses the weights of layer {j}, whose sizes differ")
        out[i] = replace(layers[i], weights_of=j)
    return out


def _loop(c: dict, n_layers: int) -> Optional[Loop]:
    l = c.get("loop")
    if not l:
        return None
    x = Loop(int(l["start"]), int(l["stop"]), int(l["times"]))
    if not 0 <= x.start < x.stop <= n_layers or x.times < 1:
        raise ValueError(f"loop {l} does not fit {n_layers} layers")
    return x


def from_layer_list(source) -> LayeredConfig:
    """`config.json` (a path, its directory, or the parsed object) -> LayeredConfig.  The inner widths of the delta
    mixers' low-rank projections are not in the file; the loader takes them from the tensors."""
    if isinstance(source, dict):
        c = source
    else:
        p = Path(source)
        c = json.loads((p / "config.json" if p.is_dir() else p).read_text())
    arch = str(c.get("architecture", "Gitozen"))
    if arch not in DESIGNS:
        raise ValueError(f"unknown layer-list architecture {arch!r}")
    d = DESIGNS[arch]
    layers = []
    for l in c["layers"]:
        if l["type"] not in d.mixers:
            raise ValueError(f"unknown mixer type {l['type']!r}")
        layers.append(LayerSpec(d.mixers[l["type"]](l["mixer"]), _mlp(l.get("mlp"), d.feed_forward)))
    if not layers:
        raise ValueError("a model needs at least one layer")
    if d.block == PRE_NORM:
        layers = _shared_weights(layers, c["layers"])
    elif any(l.get("weights_of") is not None for l in c["layers"]):
        raise ValueError(f"{arch} layers have weights of their own")
    cfg = LayeredConfig(int(c["vocab"]), int(c["width"]), tuple(layers), float(c["norm"]["eps"]),
                        float(c.get("logit_softcap") or 0.0), name=arch.lower(), block=d.block)
    if d.block == OUTPUT_NORM:
        cfg = cfg.with_(max_position=int(c["max_positions"]), learned_positions=True, canon_taps=int(c["canon"]["taps"]))
        _positive(max_positions=cfg.max_position, taps=cfg.canon_taps)
    if d.block == PRE_NORM:
        cfg = cfg.with_(embed_scale=float((c.get("embedding") or {}).get("scale", 1.0)), token_shift=True)
    if d.block == SANDWICH_NORM:
        cfg = cfg.with_(norm_groups=int(c["norm"].get("groups") or 1), loop=_loop(c, len(layers)))
        _positive(groups=cfg.norm_groups)
        if cfg.width % cfg.norm_groups:
            raise ValueError("norm.groups must divide the width")
    elif c.get("loop"):
        raise ValueError(f"{arch} layers do not loop")
    _positive(vocab=cfg.vocab_size, width=cfg.width)
    shapes = {(m.kv_heads, m.vdim) for m in (layers[i].mixer for i in cfg.attention_layers) if m.v_mix}
    if len(shapes) > 1:
        raise ValueError("value-mixing layers must agree on kv_heads and vdim")
    return cfg


def to_layer_list(cfg: LayeredConfig) -> dict:
    """The `config.json` object of a configuration."""
    layers = []
    for l in cfg.layers:
        m = l.mixer
        if isinstance(m, LatentMixer):
            mx = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale}
            if m.q_rank:
                mx.update(q_rank=m.q_rank, rot_dim=m.rot_dim, rot={"base": m.rot_base, "dims": m.rot_dim}, mask={"size": m.window})
        elif isinstance(m, Mamba2Mixer):
            mx = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.taps,
                  "norm_groups": m.norm_groups}
        elif isinstance(m, AttentionMixer):
            mx = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                  "mask": {"size": m.chunk}, "rot": {"base": m.rot_base, "dims": m.rot_dims}, "v_mix": m.v_mix}
        elif isinstance(m, WindowMixer):
            mx = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                  "mask": {"size": m.window, **({"keep_first": m.keep_first} if m.keep_first else {})}}
            if m.maps == 2:
                mx["diff"] = m.diff
            if m.pool:
                mx["mask"]["pool"] = m.pool
                mx.update(rot={"base": m.rot_base, "dims": m.rot_dims}, softcap=m.softcap or None)
        elif isinstance(m, MambaMixer):
            mx = {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.taps}
        else:
            mx = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps}
        ff = None
        if isinstance(l.mlp, DenseSpec):
            ff = {"kind": "dense", "ff": l.mlp.ff}
        elif l.mlp:
            ff = {"kind": "moe", "expert": {"ff": l.mlp.ff}, "router": {"experts": l.mlp.experts, "top": l.mlp.top}}
            if l.mlp.groups > 1:
                ff["router"]["groups"] = {"count": l.mlp.groups, "keep": l.mlp.keep}
            if cfg.block == PRE_NORM:
                ff["expert"]["limit"] = l.mlp.limit or None
                ff["shared"] = {"ff": l.mlp.shared_ff, "limit": l.mlp.shared_limit or None} if l.mlp.shared_ff else None
        layers.append({"type": m.kind, "mixer": mx, "mlp": ff, **({"weights_of": l.weights_of} if l.weights_of >= 0 else {})})
    out = {"vocab": cfg.vocab_size, "width": cfg.width, "norm": {"eps": cfg.norm_eps}, "layers": layers}
    if cfg.block == OUTPUT_NORM:
        return {"architecture": "Supisun", **out, "max_positions": cfg.max_position, "canon": {"taps": cfg.canon_taps}}
    if cfg.block == PRE_NORM:
        return {"architecture": "Vogunex", **out, "embedding": {"scale": cfg.embed_scale}}
    if cfg.block == SANDWICH_NORM:
        out["norm"] = {"eps": cfg.norm_eps, "groups": cfg.norm_groups}
        return {"architecture": "Vedadra", **out, "loop": asdict(cfg.loop) if cfg.loop else None}
    return {"architecture": "Gitozen", **out, "logit_softcap": cfg.logit_softcap or None}


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


def _gitozen_dense(name: str, width: int, heads: int, dim: int, ff: int, n_layers: int) -> LayeredConfig:
    """One expert of the given inner width that takes every token: a dense feed-forward.  Sizes beside the supisun-*
    presets: the same widths, heads, depth and about as many parameters."""
    lat = LatentMixer(heads=heads, dim=dim, vdim=dim, kv_rank=512, scale=dim ** -0.5)
    dlt = DeltaMixer(heads=heads, kv_heads=heads, dim=dim, vdim=dim, taps=4, decay_rank=128, gate_rank=128)
    return LayeredConfig(vocab_size=102400, width=width, layers=tuple(
        LayerSpec(lat if i % 4 == 3 else dlt, MoeSpec(experts=1, top=1, ff=ff)) for i in range(n_layers)), name=name)


def gitozen_dense_small(n_layers: int = 24) -> LayeredConfig:
    return _gitozen_dense("gitozen-dense-small", 1024, 8, 128, 2048, n_layers)


def gitozen_dense_lite(n_layers: int = 27) -> LayeredConfig:
    return _gitozen_dense("gitozen-dense-lite", 2048, 16, 128, 4608, n_layers)


def gitozen_dense_wide(n_layers: int = 32) -> LayeredConfig:
    return _gitozen_dense("gitozen-dense-wide", 4096, 32, 128, 7680, n_layers)


def _supisun(vocab: int, width: int, layers, max_position: int, taps: int = 4, eps: float = 1e-6,
             name: str = "supisun") -> LayeredConfig:
    return LayeredConfig(vocab_size=vocab, width=width, layers=tuple(layers), norm_eps=eps, name=name,
                         max_position=max_position, block=OUTPUT_NORM, canon_taps=taps, learned_positions=True)


def tiny_supisun() -> LayeredConfig:
    """Small shape for fixtures and the command line: all three mixers, grouped heads, a layer without feed-forward."""
    att = AttentionMixer(heads=6, kv_heads=2, dim=24, vdim=16, scale=0.2, chunk=40, rot_base=10000.0, rot_dims=16, v_mix=True)
    mam = MambaMixer(inner=112, state=8, dt_rank=6, taps=4)
    dlt = DeltaMixer(heads=4, kv_heads=2, dim=16, vdim=24, taps=3, **HEAD_DELTA)
    ff = DenseSpec(160)
    return _supisun(512, 96, (LayerSpec(att, ff), LayerSpec(mam, ff), LayerSpec(dlt, None), LayerSpec(att, ff)), 4096, taps=3)


def _supisun_attention_stack(name: str, width: int, heads: int, kv_heads: int, dim: int, ff: int, n_layers: int) -> LayeredConfig:
    """Chunked attention in every layer and no input convolution: the stack closest to the vedadra-* presets."""
    att = AttentionMixer(heads, kv_heads, dim, dim, dim ** -0.5, 8192, 500000.0, dim, False)
    return _supisun(102400, width, (LayerSpec(att, DenseSpec(ff)) for _ in range(n_layers)), 32768, taps=1, name=name)


def supisun_attention_small(n_layers: int = 24) -> LayeredConfig:
    return _supisun_attention_stack("supisun-attention-small", 1024, 8, 4, 128, 4608, n_layers)


def supisun_attention_lite(n_layers: int = 27) -> LayeredConfig:
    return _supisun_attention_stack("supisun-attention-lite", 2048, 16, 4, 128, 9216, n_layers)


def supisun_attention_wide(n_layers: int = 32) -> LayeredConfig:
    return _supisun_attention_stack("supisun-attention-wide", 4096, 32, 4, 128, 18432, n_layers)


def tiny_vedadra() -> LayeredConfig:
    """Small shape for fixtures and the command line: both mixers, grouped heads, a layer without feed-forward, a loop."""
    att = WindowMixer(heads=6, kv_heads=2, dim=24, vdim=24, scale=0.2, window=20, **TALKING_WINDOW)
    dif = WindowMixer(heads=4, kv_heads=2, dim=16, vdim=40, scale=0.25, window=36, keep_first=3, maps=2, diff=0.6)
    ff = DenseSpec(160, True)
    return LayeredConfig(512, 96, (LayerSpec(dif, ff), LayerSpec(att, ff), LayerSpec(dif, None), LayerSpec(att, ff)), 1e-6,
                         name="vedadra", block=SANDWICH_NORM, norm_groups=3, loop=Loop(1, 3, 2))


def _vedadra_stack(name: str, width: int, heads: int, kv_heads: int, dim: int, ff: int, n_layers: int) -> LayeredConfig:
    """Layers of a served model's size, `n_layers` runs of which three are a second pass: every third mixer differential,
    its maps of the other heads' width and half as many heads with values twice as wide."""
    att = WindowMixer(heads, kv_heads, dim, dim, dim ** -0.5, 1024, **TALKING_WINDOW)
    dif = WindowMixer(heads // 2, kv_heads, dim, 2 * dim, dim ** -0.5, 4096, keep_first=4, maps=2, diff=0.5)
    n = n_layers - 3
    return LayeredConfig(102400, width, tuple(LayerSpec(dif if i % 3 == 2 else att, DenseSpec(ff, True)) for i in range(n)), 1e-6,
                         name=name, block=SANDWICH_NORM, norm_groups=4, loop=Loop(n // 3, n // 3 + 3, 2))


def vedadra_small(n_layers: int = 24) -> LayeredConfig:
    return _vedadra_stack("vedadra-small", 1024, 8, 4, 128, 3072, n_layers)


def vedadra_lite(n_layers: int = 27) -> LayeredConfig:
    """The widths of DeepSeek-V2-Lite (and of supisun-attention-lite)."""
    return _vedadra_stack("vedadra-lite", 2048, 16, 4, 128, 6144, n_layers)


def vedadra_wide(n_layers: int = 32) -> LayeredConfig:
    return _vedadra_stack("vedadra-wide", 4096, 32, 4, 128, 12288, n_layers)


def _supisun_stack(name: str, width: int, heads: int, kv_heads: int, dim: int, ff: int, n_layers: int) -> LayeredConfig:
    """Layers of a served model's size: out of eight, three attention, three selective-scan and two delta mixers."""
    att = AttentionMixer(heads, kv_heads, dim, dim, dim ** -0.5, 8192, 500000.0, dim, True)
    mam = MambaMixer(inner=2 * width, state=16, dt_rank=width // 16, taps=4)
    dlt = DeltaMixer(heads, heads, dim, dim, 4, **HEAD_DELTA)
    order = (att, mam, dlt, mam, att, mam, dlt, att)
    return _supisun(102400, width, (LayerSpec(order[i % 8], DenseSpec(ff)) for i in range(n_layers)), 32768, name=name)


def supisun_small(n_layers: int = 24) -> LayeredConfig:
    return _supisun_stack("supisun-small", 1024, 8, 4, 128, 4096, n_layers)


def supisun_lite(n_layers: int = 27) -> LayeredConfig:
    """The widths of DeepSeek-V2-Lite (and of gitozen-lite)."""
    return _supisun_stack("supisun-lite", 2048, 16, 4, 128, 8192, n_layers)


def supisun_wide(n_layers: int = 32) -> LayeredConfig:
    return _supisun_stack("supisun-wide", 4096, 32, 8, 128, 14336, n_layers)


def _vogunex(vocab: int, width: int, layers, eps: float = 1e-6, embed_scale: float = 1.0, name: str = "vogunex") -> LayeredConfig:
    return LayeredConfig(vocab, width, tuple(layers), eps, name=name, block=PRE_NORM, embed_scale=embed_scale, token_shift=True)


def tiny_vogunex() -> LayeredConfig:
    """Small shape for fixtures and the command line: all three mixers, both feed-forwards, a layer without one, shared
    weights."""
    att = WindowMixer(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.2, window=20, rot_base=10000.0, rot_dims=16, softcap=15.0,
                      pool=6, **POOLED_WINDOW)
    lat = LatentMixer(heads=3, dim=24, vdim=16, kv_rank=40, scale=0.18, q_rank=56, rot_dim=8, rot_base=10000.0, window=36)
    mam = Mamba2Mixer(heads=6, vdim=16, state=24, groups=2, taps=4, norm_groups=3)
    moe = MoeSpec(experts=6, top=2, ff=40, limit=3.0, shared_ff=56, shared_limit=5.0, **CLAMPED_EXPERT)
    ff = DenseSpec(160, biases=True)
    return _vogunex(512, 96, (LayerSpec(att, ff), LayerSpec(lat, moe), LayerSpec(att, ff, weights_of=0), LayerSpec(mam, moe),
                              LayerSpec(mam, None)), 1e-5, 2.0)


def _vogunex_stack(name: str, width: int, heads: int, kv_heads: int, ff, n_layers: int) -> LayeredConfig:
    """Layers of a served model's size: out of eight, three attention, three head-decay scan and two latent mixers."""
    att = WindowMixer(heads, kv_heads, 128, 128, 128 ** -0.5, 1024, rot_base=500000.0, rot_dims=128, softcap=30.0, pool=16,
                      **POOLED_WINDOW)
    lat = LatentMixer(heads, 128, 128, 512, 192 ** -0.5, q_rank=3 * width // 4, rot_dim=64, rot_base=500000.0, window=4096)
    mam = Mamba2Mixer(heads=width // 32, vdim=64, state=128, groups=1, taps=4)
    order = (att, mam, lat, mam, att, mam, lat, att)
    return _vogunex(102400, width, (LayerSpec(order[i % 8], ff) for i in range(n_layers)), name=name)


def vogunex_small(n_layers: int = 24) -> LayeredConfig:
    return _vogunex_stack("vogunex-small", 1024, 8, 4, DenseSpec(4096, biases=True), n_layers)


def vogunex_lite(n_layers: int = 27) -> LayeredConfig:
    """The widths of supisun-lite."""
    return _vogunex_stack("vogunex-lite", 2048, 16, 4, DenseSpec(8192, biases=True), n_layers)


def vogunex_wide(n_layers: int = 32) -> LayeredConfig:
    return _vogunex_stack("vogunex-wide", 4096, 32, 8, DenseSpec(14336, biases=True), n_layers)


def vogunex_moe_lite(n_layers: int = 27) -> LayeredConfig:
    """The widths and experts of gitozen-lite, and a shared expert."""
    moe = MoeSpec(experts=64, top=6, ff=1408, limit=7.0, shared_ff=1408, shared_limit=7.0, **CLAMPED_EXPERT)
    return _vogunex_stack("vogunex-moe-lite", 2048, 16, 4, moe, n_layers)


PRESETS = {"tiny-gitozen": tiny_gitozen, "gitozen-lite": gitozen_lite, "gitozen-latent-lite": gitozen_latent_lite,
           "gitozen-dense-small": gitozen_dense_small, "gitozen-dense-lite": gitozen_dense_lite,
           "gitozen-dense-wide": gitozen_dense_wide,
           "tiny-supisun": tiny_supisun, "supisun-small": supisun_small, "supisun-lite": supisun_lite,
           "supisun-wide": supisun_wide, "supisun-attention-small": supisun_attention_small,
           "supisun-attention-lite": supisun_attention_lite, "supisun-attention-wide": supisun_attention_wide,
           "tiny-vedadra": tiny_vedadra, "vedadra-small": vedadra_small, "vedadra-lite": vedadra_lite,
           "vedadra-wide": vedadra_wide, "tiny-vogunex": tiny_vogunex, "vogunex-small": vogunex_small,
           "vogunex-lite": vogunex_lite, "vogunex-wide": vogunex_wide, "vogunex-moe-lite": vogunex_moe_lite}


def preset_architecture(preset: str) -> str:
    """Registry name of the architecture a preset belongs to."""
    return next(a for a in ARCHITECTURES if a in preset)
