"""Supisun on the sm_100a kernels: every kernel against the plain equations, whole models in 32 bits and in bf16 against
an independent oracle (whole prompts, portions, decoding, mixed batches, reused pages and slots), generation through
the engine with captured decode graphs and look-ahead."""
import random
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from ferrule_b200.models.layered_config import (OUTPUT_NORM, AttentionMixer, DenseSpec, LayeredConfig, LayerSpec,
                                                MambaMixer)
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.runtime.engine import Engine, EngineConfig, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
import supisun_oracle as SO  # noqa: E402
from supisun_configs import CONFIGS, delta  # noqa: E402

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 2e-2, F32: 3e-5}


@pytest.fixture(scope="module")
def ops():
    from ferrule_b200.ops import kernels, layered
    return kernels, layered


@pytest.fixture(autouse=True)
def _status_clean():
    yield
    if torch.cuda.is_available():
        from ferrule_b200.ops import _lib
        torch.cuda.synchronize()
        assert _lib.read_status()[0] == 0


def rnd(*shape, dtype=F32, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed * 7919 + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(BF).to(dtype).cuda()


def near(got, want, dtype, scale=None):
    got, want = got.double().cpu(), want.double().cpu()
    d = (got - want).abs().max() / (want.abs().max() if scale is None else scale)
    assert d < TOL[dtype], float(d)


def i32(*x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def packed(lens, old):
    """Row-to-sequence tables of a packed batch; sequence s reads state 2 s (when `old`) and writes state 2 s + 1."""
    start = np.concatenate([[0], np.cumsum(lens)])
    return dict(row_seq=i32(*[s for s, n in enumerate(lens) for _ in range(n)]), seq_start=i32(*start.tolist()),
                state_in=i32(*[2 * s if o else -1 for s, o in enumerate(old)]),
                state_out=i32(*[2 * s + 1 for s in range(len(lens))]), n_seqs=len(lens))


LENS, OLD = [1, 40, 2, 17, 3, 16, 4], [True, True, False, False, True, True, False]


def ldiv8(n):
    return (n + 7) // 8 * 8


# ------------------------------------------------------------------ row operators
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim", [52, 300, 2048, 4100])
@pytest.mark.parametrize("rms", [False, True])
def test_norm_and_residual_addition(ops, dtype, dim, rms):
    KL, T, pad = ops[1], 5, ldiv8(dim)
    z = lambda *s, **kw: torch.nn.functional.pad(rnd(*s, **kw), (0, pad - s[-1])).contiguous()
    x, y, wb = z(T, dim, seed=1), z(T, dim, dtype=dtype, seed=2), z(2, dim, seed=3)
    y[1] += 40.0 * (torch.arange(pad, device="cuda") < dim)                 # a mean far above the deviation
    act = torch.full((T, pad), 7.0, dtype=dtype, device="cuda")
    yd, w = y.double().cpu()[:, :dim], wb.double().cpu()[:, :dim]
    normed = SO.rms(yd, 1e-5) * w[0] if rms else SO.layer_norm(yd, w[0], w[1], 1e-5)
    want = x.double().cpu()[:, :dim] + normed
    KL.add_normed(x, y, wb, dim, 1e-5, act=act, rms=rms)
    near(x[:, :dim], want, F32)                                             # the stream is 32-bit either way
    assert torch.equal(act, x.to(dtype)) and not x[:, dim:].any()
    rows = i32(4, 0, 4)
    out = torch.full((3, pad), 7.0, dtype=dtype, device="cuda")
    KL.norm_rows(x, rows, wb, out, dim, 1e-5, rms=rms)
    xs = x.double().cpu()[[4, 0, 4], :dim]
    near(out[:, :dim], SO.rms(xs, 1e-5) * w[0] if rms else SO.layer_norm(xs, w[0], w[1], 1e-5), dtype)
    assert not out[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,taps", [(52, 4), (2048, 3), (72, 1), (300, 6)])
def test_embedding_with_positions_and_the_fused_input_convolution(ops, dtype, dim, taps):
    """Decode form: one row per sequence, the convolution's earlier inputs in the state."""
    KL, pad, old = ops[1], ldiv8(dim), [True, False, True, True, False]
    z = lambda *s, **kw: torch.nn.functional.pad(rnd(*s, **kw), (0, pad - s[-1])).contiguous()
    table, pos, w = z(33, dim, dtype=dtype), z(50, dim, dtype=dtype, seed=1), z(taps, dim, seed=2)
    tail = z(11, max(taps - 1, 1), dim, seed=3)
    before, p = tail.clone(), packed([1] * 5, old)
    ids, at = i32(3, 32, 0, 3, 9), i32(0, 49, 7, 1, 2)
    x = torch.full((5, pad), 7.0, device="cuda")
    h = torch.full((5, pad), 7.0, dtype=dtype, device="cuda")
    KL.embed_stream(ids, table, x, dim, positions=at, pos_table=pos, canon=(w, tail, p["state_in"], p["state_out"], h))
    assert torch.equal(x, table[ids.long()].float() + pos[at.long()].float())
    for s in range(5):
        prev = before[2 * s, :taps - 1] if old[s] else torch.zeros(taps - 1, pad, device="cuda")
        seq = torch.cat([prev, x[s:s + 1]]).double().cpu()
        near(h[s], (seq + SO.causal_conv(seq, w.double().cpu().T))[-1], dtype)
        if taps > 1:
            assert torch.equal(tail[2 * s + 1], seq[1:].float().cuda()) and torch.equal(tail[2 * s], before[2 * s])
    # and behind a sublayer
    y, wb, tail2 = z(5, dim, dtype=dtype, seed=4), z(2, dim, seed=5), before.clone()
    want = x.clone()
    KL.add_normed(want, y, wb, dim, 1e-5)
    KL.add_normed(x, y, wb, dim, 1e-5, canon=(w, tail2, p["state_in"], p["state_out"], h))
    assert torch.equal(x, want)
    seq = torch.cat([before[0, :taps - 1], x[:1]]).double().cpu()
    near(h[0], (seq + SO.causal_conv(seq, w.double().cpu().T))[-1], dtype)


@pytest.mark.parametrize("form", ["stream", "stream32", "bf16", "fp32"])
@pytest.mark.parametrize("channels,taps", [(56, 4), (2048, 4), (304, 3), (64, 2), (40, 1), (72, 7)])
def test_short_convolution_of_packed_sequences(ops, form, channels, taps):
    KL, T = ops[1], sum(LENS)
    ti = BF if form == "bf16" else F32
    to = F32 if form in ("fp32", "stream32") else BF
    x = rnd(T, channels + 16, dtype=ti)[:, 8:8 + channels]
    w, bias = rnd(taps, channels, seed=1), rnd(channels, seed=2)
    tail = rnd(2 * len(LENS), max(taps - 1, 1), channels, dtype=ti, seed=3)
    before, out = tail.clone(), torch.full((T, channels), 7.0, dtype=to, device="cuda")
    stream = form.startswith("stream")
    KL.short_conv(x, w, tail, out, **packed(LENS, OLD), bias=None if stream else bias, residual=stream, silu=not stream)
    at = 0
    for s, n in enumerate(LENS):
        prev = before[2 * s, :taps - 1] if OLD[s] else torch.zeros(taps - 1, channels, dtype=ti, device="cuda")
        seq = torch.cat([prev, x[at:at + n]])
        sd = seq.double().cpu()
        y = SO.causal_conv(sd, w.double().cpu().T, None if stream else bias.double().cpu())
        y = sd + y if stream else torch.nn.functional.silu(y)
        near(out[at:at + n], y[taps - 1:], to)
        if taps > 1:
            assert torch.equal(tail[2 * s + 1], seq[len(seq) - taps + 1:]) and torch.equal(tail[2 * s], before[2 * s])
        at += n


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows", [3, 40, 300])
def test_gelu_epilogue(ops, dtype, rows):
    K = ops[0]
    x, w = rnd(rows, 72, dtype=dtype), rnd(136, 72, dtype=dtype, scale=0.3)
    z = x.double() @ w.double().T
    near(K.gemm(x, w, epilogue=K.EPI_GELU), 0.5 * z * (1 + torch.erf(z / 2 ** 0.5)), dtype)


# ------------------------------------------------------------------ selective scan
def scan_case(dtype, m, lens, old, seed=0):
    T, Ip = sum(lens), m.inner_pad
    img = type("Img", (), {})()
    img.a_log2 = -torch.exp(rnd(m.state, Ip, seed=seed) * 0.7) * 1.4426950408889634
    img.dt_bias, img.d_skip = rnd(Ip, seed=seed + 1) - 2, rnd(Ip, seed=seed + 2)
    off_c = ldiv8(m.state) + 8
    case = dict(x=rnd(T, Ip, dtype=dtype, seed=seed + 3), z=rnd(T, Ip + 24, dtype=dtype, seed=seed + 4)[:, 16:16 + Ip],
                bc=rnd(T, off_c + ldiv8(m.state), dtype=dtype, seed=seed + 5), off_b=8, off_c=off_c,
                dt=rnd(T, Ip, seed=seed + 6), img=img, states=rnd(2 * len(lens) + 1, m.state, Ip, seed=seed + 7))
    tables = packed(lens, old)
    del tables["row_seq"]
    return {**case, **tables}


def scan_want(case, m, lens, old):
    d = lambda t: t.double().cpu()
    dt = torch.nn.functional.softplus(d(case["dt"]) + d(case["img"].dt_bias), threshold=1e9)
    A = d(case["img"].a_log2).T * np.log(2.0)
    outs, states, at = [], [], 0
    for s, n in enumerate(lens):
        r = slice(at, at + n)
        bc = d(case["bc"])[r]
        y, S = SO.selective_scan(d(case["x"])[r], dt[r], A, bc[:, 8:8 + m.state], bc[:, case["off_c"]:case["off_c"] + m.state],
                                 d(case["img"].d_skip), d(case["states"][2 * s]).T if old[s] else None)
        outs.append(y * torch.nn.functional.silu(d(case["z"])[r]))
        states.append(S.T)
        at += n
    return torch.cat(outs), states


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("inner,state", [(72, 16), (40, 5), (264, 32), (64, 8), (96, 64), (33, 100), (8, 1)])
@pytest.mark.parametrize("decode", [False, True])
def test_selective_scan(ops, dtype, inner, state, decode):
    KL, m = ops[1], MambaMixer(inner, state, 4, 4)
    lens, old = ([1] * 5, [True, False, True, True, False]) if decode else (LENS, OLD)
    case = scan_case(dtype, m, lens, old)
    before, want = case["states"].clone(), scan_want(case, m, lens, old)
    out = torch.full((sum(lens), m.inner_pad), 5.0, dtype=dtype, device="cuda")
    KL.selective_scan(out=out, **case)
    near(out, want[0], dtype)
    for s in range(len(lens)):
        near(case["states"][2 * s + 1], want[1][s], F32, scale=1.0 + want[1][s].abs().max())
        assert torch.equal(case["states"][2 * s], before[2 * s])
    assert torch.equal(case["states"][-1], before[-1])


def test_selective_scan_portions_carry_the_state_over_long_runs(ops):
    """600 tokens in portions equal one pass; slowly decaying states remember the first token."""
    KL, m = ops[1], MambaMixer(48, 16, 4, 4)
    case = scan_case(F32, m, [600], [False])
    case["img"].a_log2[::2] = -1e-3
    want, states = scan_want(case, m, [600], [False])
    at, cur, r, outs = 0, -1, random.Random(0), []
    while at < 600:
        n = min(r.choice([1, 2, 3, 15, 16, 17, 64, 130]), 600 - at)
        nxt = 1 - cur if cur >= 0 else 0
        sub = {**case, **{k: case[k][at:at + n] for k in ("x", "z", "bc", "dt")}, "seq_start": i32(0, n), "state_in": i32(cur),
               "state_out": i32(nxt)}
        outs.append(KL.selective_scan(out=torch.zeros(n, m.inner_pad, device="cuda"), **sub))
        at, cur = at + n, nxt
    near(torch.cat(outs), want, F32)
    near(case["states"][cur], states[0], F32)


# ------------------------------------------------------------------ delta rule with one decay per head
def delta_case(dtype, m, lens, old, seed=0):
    T, nk, nv = sum(lens), m.kv_heads * m.dim, m.heads * m.vdim
    off, at = {}, 0
    for name, n in (("q", nk), ("k", nk), ("v", nv), ("a", m.heads), ("g", nv), ("b", m.heads)):
        off[name] = at
        at += ldiv8(n)
    img = type("Img", (), {})()
    img.off_gate = 0
    img.conv, img.a_neg = rnd(m.taps, m.channels, seed=seed + 1), -torch.exp(rnd(m.heads, seed=seed + 2))
    img.dt_bias, img.o_norm = rnd(m.heads, seed=seed + 3) - 2, rnd(m.vdim, seed=seed + 4)
    n_states = 2 * len(lens) + 1
    return dict(proj=rnd(T, at, dtype=dtype, seed=seed + 5), off=off, ag=None, img=img, mixer=m, eps=1e-5,
                state=rnd(n_states, m.heads, m.dim, m.vdim, seed=seed + 7),
                tail=rnd(n_states, max(m.taps - 1, 1), m.channels, dtype=dtype, seed=seed + 8), **packed(lens, old))


def delta_want(case, lens, old):
    m, off, img = case["mixer"], case["off"], case["img"]
    d = lambda t: t.double().cpu()
    nk, nv, keep, F = m.kv_heads * m.dim, m.heads * m.vdim, m.taps - 1, torch.nn.functional
    proj = d(case["proj"])
    raw = torch.cat([proj[:, off["q"]:off["q"] + nk], proj[:, off["k"]:off["k"] + nk], proj[:, off["v"]:off["v"] + nv]], 1)
    share, outs, states, at = [h // (m.heads // m.kv_heads) for h in range(m.heads)], [], [], 0
    for s, n in enumerate(lens):
        r = slice(at, at + n)
        before = d(case["tail"][2 * s, :keep]) if old[s] else torch.zeros(keep, m.channels, dtype=torch.float64)
        y = F.silu(SO.causal_conv(torch.cat([before, raw[r]]), d(img.conv).T))[keep:]
        q, k, v = y[:, :nk].view(n, -1, m.dim), y[:, nk:2 * nk].view(n, -1, m.dim), y[:, 2 * nk:].view(n, m.heads, m.vdim)
        g = SO.head_decay(proj[r, off["a"]:off["a"] + m.heads], torch.log(-d(img.a_neg)), d(img.dt_bias))
        beta = torch.sigmoid(proj[r, off["b"]:off["b"] + m.heads])
        o, S = SO.delta_recurrence((SO.unit(q) / m.dim ** 0.5)[:, share], SO.unit(k)[:, share], v, g, beta,
                                   d(case["state"][2 * s]) if old[s] else None)
        gate = F.silu(proj[r, off["g"]:off["g"] + nv]).view(n, m.heads, m.vdim)
        outs.append((SO.rms(o, case["eps"]) * d(img.o_norm) * gate).reshape(n, -1))
        states.append(S)
        at += n
    return torch.cat(outs), states


DELTAS = [delta(3, 3, 64, 48, 4), delta(4, 2, 20, 12, 3), delta(6, 1, 8, 4, 1), delta(2, 2, 72, 33, 5), delta(2, 1, 128, 128, 4),
          delta(1, 1, 130, 100, 2), delta(2, 2, 31, 64, 4)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", DELTAS, ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}t{m.taps}")
@pytest.mark.parametrize("decode", [False, True])
def test_delta_rule_with_head_decay(ops, dtype, m, decode):
    KL = ops[1]
    lens, old = ([1] * 5, [True, False, True, True, False]) if decode else (LENS, OLD)
    if decode and not KL.delta_decode_supported(m):
        pytest.skip("served by the prefill form")
    case = delta_case(dtype, m, lens, old)
    before, (want, states) = case["state"].clone(), delta_want(case, lens, old)
    out = torch.full((sum(lens), ldiv8(m.heads * m.vdim)), 5.0, dtype=dtype, device="cuda")
    KL.delta_rule(out=out, scratch=KL.DeltaScratch(sum(lens), [m], "cuda"), decode=decode, **case)
    near(out[:, :m.heads * m.vdim], want, dtype)
    for s in range(len(lens)):
        near(case["state"][2 * s + 1], states[s], F32, scale=1.0 + states[s].abs().max())
        assert torch.equal(case["state"][2 * s], before[2 * s])


# ------------------------------------------------------------------ attention
def attention_rows(m, lens, page, seed=0):
    """Paged pool with shuffled pages; query rows around every page and chunk border."""
    g = random.Random(seed)
    per = [(n + page - 1) // page for n in lens]
    ids = list(range(sum(per) + 3))
    g.shuffle(ids)
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([ids.pop() for _ in range(n)])
    edges = lambda n, c: {k * c + o for k in range(n // c + 1) for o in (-1, 0, 1)}
    rows = [(s, p) for s, n in enumerate(lens) for p in sorted(edges(n, page) | edges(n, m.chunk) | {n - 1}) if 0 <= p < n]
    return sum(per) + 3, table, rows


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", [AttentionMixer(6, 2, 20, 12, 0.3, 10, 5000.0, 12, True), AttentionMixer(4, 4, 64, 64, 0.2, 24, 1e4, 64),
                               AttentionMixer(3, 1, 30, 130, 0.3, 17, 50.0, 2, True), AttentionMixer(8, 2, 128, 128, 0.1, 512, 1e6, 0)],
                         ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}c{m.chunk}")
def test_attention_norms_rotation_values_and_cache_append(ops, dtype, m):
    KL, T, eps = ops[1], 9, 1e-5
    H, G, D, V, dp, vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_pad, m.vdim_pad
    proj = torch.zeros(T, H * dp + G * (dp + vp) + 8, dtype=dtype, device="cuda")
    q, k, v = proj[:, :H * dp], proj[:, H * dp:(H + G) * dp], proj[:, (H + G) * dp:(H + G) * dp + G * vp]
    qs, ks, vs = rnd(T, H, D, dtype=dtype), rnd(T, G, D, dtype=dtype, seed=1), rnd(T, G, V, dtype=dtype, seed=2)
    q.unflatten(1, (H, dp))[..., :D], k.unflatten(1, (G, dp))[..., :D], v.unflatten(1, (G, vp))[..., :V] = qs, ks, vs
    img = type("Img", (), {})()
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).reshape(-1).contiguous()
    qn, kn = 1 + 0.3 * rnd(H, D, seed=3), 1 + 0.3 * rnd(G, D, seed=4)
    img.q_norm, img.k_norm, img.v_mix = pad(qn, dp), pad(kn, dp), 0.35
    row_dim = m.row_dim + 16
    pool = torch.full((3, 5, row_dim), 9.0, dtype=dtype, device="cuda")
    first = rnd(3, 5, row_dim, dtype=dtype, seed=5)
    slots = torch.tensor([5, 0, 14, -1, 2, 9, 1, 8, 13], device="cuda")
    # row t of the plain rotation is position t
    from ferrule_b200.models.layered import rotation_frequencies
    a = torch.arange(T, dtype=torch.float64)[:, None] * rotation_frequencies(m.rot_base, m.rot_dims)
    tables = (torch.cos(a).float().cuda(), torch.sin(a).float().cuda())
    KL.gqa_prep(q, k, v, m, img, tables, i32(*range(T)), slots, pool, eps, first_pool=first if m.v_mix else None, first_off=16)
    d = lambda t: t.double().cpu()
    whole = lambda t, w: (SO.rms(d(t).reshape(T, -1), eps) * d(w).reshape(-1)).view(t.shape)
    near(q.unflatten(1, (H, dp))[..., :D], SO.rotate(whole(qs, qn), m.rot_base, m.rot_dims), dtype)
    want_k, want_v = SO.rotate(whole(ks, kn), m.rot_base, m.rot_dims), SO.rms(d(vs), eps)
    flat, keep = pool.view(-1, row_dim), slots >= 0
    at = slots[keep]
    if m.v_mix:
        fv = d(first).view(-1, row_dim)[slots.clamp(min=0).cpu(), 16:16 + G * vp].view(T, G, vp)[..., :V]
        want_v = 0.65 * want_v + 0.35 * fv
    near(flat[at, :G * dp].view(-1, G, dp)[..., :D], want_k[keep.cpu()], dtype)
    near(flat[at, G * dp:G * (dp + vp)].view(-1, G, vp)[..., :V], want_v[keep.cpu()], dtype)
    assert (flat[[i for i in range(15) if i not in slots.tolist()]] == 9.0).all()


ATTENTIONS = [AttentionMixer(6, 2, 20, 12, 0.9, 10, 1.0, 0), AttentionMixer(3, 3, 64, 64, 0.9, 37, 1.0, 0),
              AttentionMixer(8, 1, 128, 128, 0.9, 64, 1.0, 0), AttentionMixer(5, 1, 48, 80, 0.9, 96, 1.0, 0),
              AttentionMixer(4, 2, 136, 200, 0.9, 1000, 1.0, 0), AttentionMixer(2, 1, 300, 40, 0.9, 50, 1.0, 0),
              AttentionMixer(16, 4, 128, 128, 0.9, 130, 1.0, 0)]


def attention_case(m, dtype, page, lens, rows=None):
    n_pages, table, picked = attention_rows(m, lens, page)
    rows = picked if rows is None else rows
    pool = torch.zeros(n_pages, page, m.row_dim + 8, dtype=dtype, device="cuda")
    pool[..., :m.v_offset].unflatten(2, (m.kv_heads, m.dim_pad))[..., :m.dim] = rnd(n_pages, page, m.kv_heads, m.dim, dtype=dtype)
    pool[..., m.v_offset:m.v_offset + m.kv_heads * m.vdim_pad].unflatten(2, (m.kv_heads, m.vdim_pad))[..., :m.vdim] = \
        rnd(n_pages, page, m.kv_heads, m.vdim, dtype=dtype, seed=1)
    q = torch.zeros(len(rows), m.heads, m.dim_pad, dtype=dtype, device="cuda")
    q[..., :m.dim] = rnd(len(rows), m.heads, m.dim, dtype=dtype, scale=0.3, seed=2)
    flat = pool.view(-1, pool.shape[-1])
    # one score stands out: the first key of the chunk, the key just before it (not visible), the last key
    for i, (s, p) in enumerate(rows):
        lo = p // m.chunk * m.chunk
        for h, t in enumerate((lo, lo - 1, p)):
            if t >= 0 and h < m.heads:
                g = h // (m.heads // m.kv_heads)
                key = flat[int(table[s, t // page]) * page + t % page, g * m.dim_pad:g * m.dim_pad + m.dim].float()
                q[i, h, :m.dim] = (key * (20.0 / float(key.norm() ** 2))).to(dtype)
    fd, want = flat.double().cpu(), []
    for i, (s, p) in enumerate(rows):
        t = torch.arange(p // m.chunk * m.chunk, p + 1)
        kv = fd[table[s, t // page].long() * page + t % page]
        for h in range(m.heads):
            g = h // (m.heads // m.kv_heads)
            w = torch.softmax(kv[:, g * m.dim_pad:g * m.dim_pad + m.dim] @ q[i, h, :m.dim].double().cpu() * m.scale, 0)
            v0 = m.v_offset + g * m.vdim_pad
            want.append(w @ kv[:, v0:v0 + m.vdim])
    return pool, table.cuda(), q, rows, torch.stack(want).view(len(rows), m.heads, m.vdim)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("m", ATTENTIONS, ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}c{m.chunk}")
def test_attention_in_chunks(ops, dtype, m, page):
    KL = ops[1]
    pool, table, q, rows, want = attention_case(m, dtype, page, [1, 40, 200])
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=dtype, device="cuda")
    KL.gqa_attention(q.flatten(1), m, pool, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), page, out)
    near(out.view(len(rows), m.heads, -1)[..., :m.vdim], want, dtype)


@pytest.mark.parametrize("page,splits,early", [(16, 1, False), (64, 2, False), (8, 4, True), (16, 8, True)])
@pytest.mark.parametrize("m", [m for m in ATTENTIONS if max(m.dim, m.vdim) <= 256] + [AttentionMixer(40, 2, 64, 64, 0.9, 300, 1.0, 0)],
                         ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}c{m.chunk}")
def test_attention_of_few_rows(ops, m, page, splits, early):
    KL = ops[1]
    pool, table, q, rows, want = attention_case(m, BF, page, [1, 40, 300])
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=BF, device="cuda")
    KL.gqa_decode(q.flatten(1), m, pool, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), page, out, splits=splits,
                  decode_only=early)
    near(out.view(len(rows), m.heads, -1)[..., :m.vdim], want, BF)


@pytest.mark.parametrize("page", [8, 16, 64, 128])
@pytest.mark.parametrize("m", [m for m in ATTENTIONS if max(m.dim, m.vdim) <= 256] + [AttentionMixer(14, 2, 256, 256, 0.9, 90, 1.0, 0)],
                         ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}c{m.chunk}")
def test_prompt_attention_on_tensor_cores(ops, m, page):
    """Tiles that start and end anywhere: inside a chunk, at its border, over several chunks; portions that continue."""
    K, KL = ops
    parts = ((90, 0), (70, 130), (33, 27), (1, 64))
    rows = [(s, p0 + i) for s, (n, p0) in enumerate(parts) for i in range(n)]
    pool, table, q, rows, want = attention_case(m, BF, page, [p0 + n for n, p0 in parts], rows)
    segs, r0 = [], 0
    for s, (n, p0) in enumerate(parts):
        segs.append((s, r0, n, p0))
        r0 += n
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=BF, device="cuda")
    assert KL.gqa_tc_group(m, BF, page) == m.heads // m.kv_heads
    for group in {m.heads // m.kv_heads, min(2 * m.heads // m.kv_heads, 128)}:      # also tiles another layer's groups limit
        tiles, rest = K.prefill_tiles(segs, group, 2)
        assert rest == [(len(rows) - 1, len(rows))]
        KL.gqa_prefill_tc(q.flatten(1), m, pool, table, torch.from_numpy(tiles).cuda().contiguous(), len(tiles), 128 // group, page, out)
        got = out.view(len(rows), m.heads, -1)
        near(got[:-1, :, :m.vdim], want[:-1], BF)
        assert (got[-1] == 7.0).all()


# ------------------------------------------------------------------ whole models
_memo = {}


def model(name, dtype, gain=1.6):
    key = (name, dtype)
    if key not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=F32, gain=gain)
        _memo[key] = (cfg, pack_weights(cfg, lambda n: t(n).to(device="cuda", dtype=dtype)), SO.Oracle(cfg, t))
    return _memo[key]


def engine(name, dtype, pages=24, page=16, slots=4, cls=ReplayEngine, rows=None, **kw):
    cfg, w, oracle = model(name, dtype)
    n = pages * page
    runner = LayeredRunner(w, n_pages=pages, page_size=page, max_rows=rows or n, max_seqs=slots, max_seq_len=n + page, full_logit_rows=64)
    sched = SchedulerConfig(max_active_sequences=slots, max_decode_batch=slots, max_batch_tokens=rows or n, prefill_chunk_size=rows or n,
                            ctx_size=n + page, **kw)
    return cls(runner, EngineConfig(scheduler=sched, kv_pages=pages, page_size=page)), oracle, cfg


def prompt(cfg, n, seed):
    r = random.Random(seed)
    return [r.randrange(cfg.vocab_size) for _ in range(n)]


def same(got, want, dtype):
    """Root mean square over a row's logits; most rows are well inside (a norm over nearly equal values amplifies the
    rounding of a few)."""
    e = np.sqrt(((np.asarray(got) - want.float().numpy()) ** 2).mean(1)) / float(want.std())
    mid, most = (5e-6, 1e-4) if dtype == F32 else (0.05, 0.4)
    assert np.median(e) < mid and e.max() < most, (float(np.median(e)), float(e.max()))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_token_by_token(name, dtype):
    eng, oracle, cfg = engine(name, dtype)
    toks = prompt(cfg, 75, 1)
    want = oracle.logits(toks)
    same(eng.replay([ReplayEntry("w", toks, list(range(75)))], ["w"])[0], want, dtype)
    rows = [eng.replay([ReplayEntry("d", [t], [0])])[0] for t in toks]
    same(np.concatenate(rows), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("sizes", [[2], [3, 2], [16], [1, 9, 2, 33]])
def test_portions_of_any_size(sizes, dtype):
    eng, oracle, cfg = engine("all", dtype)
    toks = prompt(cfg, 130, 3)
    want, at, k, rows = oracle.logits(toks), 0, 0, []
    while at < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - at)
        k += 1
        rows.append(eng.replay([ReplayEntry("a", toks[at:at + n], list(range(n)))])[0])
        at += n
    same(np.concatenate(rows), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page,chunk", [(8, 24), (64, 50), (16, 16)])
def test_a_token_is_seen_exactly_inside_its_chunk(page, chunk, decoded, dtype):
    """One attention layer and no convolution: a changed token changes the logits of its own chunk behind it, no others."""
    cfg = LayeredConfig(vocab_size=50, width=32, layers=(LayerSpec(AttentionMixer(4, 2, 16, 16, 0.5, chunk, 50.0, 8), DenseSpec(24)),),
                        norm_eps=1e-5, name="supisun", max_position=200, block=OUTPUT_NORM, canon_taps=1, learned_positions=True)
    w = pack_weights(cfg, lambda n, t=RandomTensors(cfg, seed=3, dtype=F32, gain=1.5): t(n).to(device="cuda", dtype=dtype))
    runner = LayeredRunner(w, n_pages=160 // page + 1, page_size=page, max_rows=160, max_seqs=1, max_seq_len=160, full_logit_rows=64)
    eng = ReplayEngine(runner, EngineConfig(scheduler=SchedulerConfig(1, 1, 160, 160, ctx_size=160), kv_pages=160 // page + 1,
                                            page_size=page))
    toks = prompt(cfg, 110, 5)

    def logits(seq):
        # the head in one portion; the tail decoded token by token, or in a second portion
        cuts = [(0, 60)] + ([(i, 1) for i in range(60, 110)] if decoded else [(60, 50)])
        out = [eng.replay([ReplayEntry("a", seq[i:i + n], list(range(n)))], ["a"] if i + n == 110 else [])[0] for i, n in cuts]
        return np.concatenate(out)

    base = logits(toks)
    edges = sorted({k * chunk + o for k in range(3) for o in (-1, 0, 1)} | {page - 1, page})
    for t in (e for e in edges if 0 <= e < 110):
        seq = list(toks)
        seq[t] = (seq[t] + 7) % cfg.vocab_size
        changed = np.abs(logits(seq) - base).max(1) > 1e-3
        want = np.array([p >= t and p // chunk == t // chunk for p in range(110)])
        assert not changed[~want].any() and changed[want].mean() > 0.9 and changed[t], t


@pytest.mark.parametrize("dtype", [F32, BF])
def test_mixed_batches_reuse_pages_and_slots(dtype):
    rnd_ = random.Random(4)
    eng, oracle, cfg = engine("all", dtype, pages=8)
    todo = [(f"q{i}", prompt(cfg, rnd_.randrange(1, 60), 100 + i)) for i in range(12)]
    live, got = {}, {}
    pages = lambda n: (n + 15) // 16
    while todo or live:
        while todo and len(live) < 4 and sum(pages(len(t)) for t, _ in live.values()) + pages(len(todo[0][1])) <= 8:
            rid, t = todo.pop(0)
            live[rid] = (t, 0)
        entries, end = [], []
        for rid in list(live):
            t, at = live[rid]
            if rnd_.random() < 0.25:
                continue
            n = min(rnd_.choice([1, 1, 2, 3, 20]), len(t) - at)
            entries.append(ReplayEntry(rid, t[at:at + n], list(range(n))))
            live[rid] = (t, at + n)
            if at + n == len(t):
                end.append(rid)
        rnd_.shuffle(entries)
        for e, rows in zip(entries, eng.replay(entries, end)):
            got.setdefault(e.request_id, (live[e.request_id][0], []))[1].append(rows)
        for rid in end:
            del live[rid]
    for t, rows in got.values():
        same(np.concatenate(rows), oracle.logits(t), dtype)
    assert eng.kv.free_pages == 8 and eng.scheduler.slots.available == 4


@pytest.mark.parametrize("chunk", [3, 64])
def test_greedy_generation_with_graphs_and_look_ahead(chunk):
    """In 32 bits the engine's own loop (scheduler, captured decode graphs, look-ahead) gives the oracle's tokens."""
    eng, oracle, cfg = engine("all", F32, cls=Engine)
    eng.cfg.scheduler.prefill_chunk_size = chunk
    ps = {f"r{i}": prompt(cfg, n, 50 + i) for i, n in enumerate((1, 2, 37, 9, 26, 5))}
    toks = {}
    for r, p in ps.items():
        eng.submit(GenerateRequest(r, p, max_new_tokens=24, ignore_eos=True))
    eng.run_until_idle(lambda ev: toks.setdefault(ev.request_id, []).append(ev.token) if isinstance(ev, TokenEvent) else None)
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 24), r
    assert eng.runner.stats.graph_steps > 0 and eng.runner.stats.lookahead_hits > 0 and eng.kv.free_pages == 24
