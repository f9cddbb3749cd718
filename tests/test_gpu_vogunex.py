"""Vogunex on the sm_100a kernels: every kernel against the plain equations, whole models in 32 bits and in bf16 against an
independent oracle (whole prompts, portions, decoding, mixed batches, reused pages and slots), generation through the engine
with captured decode graphs and look-ahead."""
import random
import sys
from dataclasses import replace
from pathlib import Path

import numpy as np
import pytest
import torch

from ferrule_b200.models.layered_config import Mamba2Mixer, to_layer_list
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.runtime.engine import Engine, EngineConfig, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
import vogunex_oracle as VO  # noqa: E402
from vogunex_configs import CONFIGS, FF, latent, moe, pooled, vogunex  # noqa: E402

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


def dbl(t):
    return t.double().cpu()


def pad8(n):
    return (n + 7) // 8 * 8


# ------------------------------------------------------------------ row operators
def batch_of(lens, fresh, buffers=3):
    """Packed sequences: sequence s reads state index `buffers * s` (none when fresh) and writes the next."""
    start = [0]
    for n in lens:
        start.append(start[-1] + n)
    row_seq = i32(*[s for s, n in enumerate(lens) for _ in range(n)])
    return (row_seq, i32(*start), i32(*[-1 if f else buffers * s for s, f in enumerate(fresh)]),
            i32(*[buffers * s + 1 for s in range(len(lens))]), len(lens))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim", [60, 256, 1000, 4100])
@pytest.mark.parametrize("lens", [(1, 1, 1), (5,), (1, 30, 2, 9, 1)])
def test_residual_addition_norm_and_token_shift(ops, dtype, dim, lens):
    KL, T, pad, eps = ops[1], sum(lens), pad8(dim), 1e-3
    z = lambda *s, **kw: torch.nn.functional.pad(rnd(*s, **kw), (0, pad - s[-1])).contiguous()
    cut = lambda t: dbl(t)[..., :dim]
    x, y, table = z(T, dim, seed=1), z(T, dim, dtype=dtype, seed=2), z(11, dim, dtype=dtype, seed=3)
    norm, shift, plane = z(dim, seed=4), z(dim, seed=5), z(9 * 3, dim, seed=6)
    ffn, shared, gate = z(T * 4, dim, dtype=dtype, seed=7).view(T, 4, pad), z(T, dim, dtype=dtype, seed=8), rnd(T, 3, seed=9)[:, 1:2]
    ids = i32(*[(7 * i) % 11 for i in range(T)])
    fresh = [s % 2 == 0 for s in range(len(lens))]
    seqs = batch_of(lens, fresh)
    stream = {"y": (cut(x) + cut(y), dict(y=y)), "embedding": (cut(table)[ids.long().cpu()] * 1.5, dict(ids=ids, table=table, scale=1.5)),
              "experts": (cut(x) + cut(ffn)[:, :3].sum(1), dict(ffn=ffn, topk=3)),
              "shared expert": (cut(x) + cut(ffn)[:, :2].sum(1) + torch.sigmoid(dbl(gate)) * cut(shared),
                                dict(ffn=ffn, topk=2, shared=shared, shared_gate=gate))}
    for name, (want, args) in stream.items():
        src = None if name == "embedding" else x
        for form in ("tail", "norm", "shift"):
            out, act, state = torch.full_like(x, 7.0), torch.full((T, pad), 7.0, dtype=dtype, device="cuda"), plane.clone()
            kw = {} if form == "tail" else dict(norm=norm, act=act)
            if form == "shift":
                kw.update(shift=shift, plane=state, seqs=seqs)
            KL.pre_norm_step(src, out, dim=dim, eps=eps, like=act, **args, **kw)
            near(out[:, :dim], want, F32)
            assert not out[:, dim:].any()
            if form == "tail":
                continue
            h = VO.rms(want, eps) * cut(norm)
            if form == "shift":
                for s, n in enumerate(lens):
                    a = int(seqs[1][s])
                    first = torch.zeros(1, dim, dtype=torch.float64) if fresh[s] else cut(plane)[3 * s:3 * s + 1]
                    near(state[3 * s + 1, :dim], h[a + n - 1], F32)              # the state is the row before its own shift
                    before = torch.cat([first, h[a:a + n - 1]])
                    h[a:a + n] = (h[a:a + n] + (before - h[a:a + n]) * cut(shift)) if n == 1 else torch.cat(
                        [h[a:a + 1] + (first - h[a:a + 1]) * cut(shift), VO.token_shift(h[a:a + n], cut(shift))[1:]])
                untouched = [i for i in range(27) if i not in [3 * s + 1 for s in range(len(lens))]]
                assert torch.equal(state[untouched], plane[untouched])
            near(act[:, :dim], h, dtype)
            assert not act[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,groups", [(60, 3), (52, 13), (300, 2), (2048, 1), (4096, 8)])
def test_group_norm_of_activation_rows(ops, dtype, dim, groups):
    KL, pad = ops[1], pad8(dim)
    x, w = rnd(5, pad, dtype=dtype), torch.nn.functional.pad(rnd(dim, seed=1), (0, pad - dim)).contiguous()
    x *= (3.0 ** (torch.arange(pad) // (dim // groups) % 5)).cuda().to(dtype)
    want = VO.part_norm(dbl(x)[:, :dim], groups, 1e-3) * dbl(w)[:dim]
    assert KL.group_norm_rows(x, w, x, dim, groups, 1e-3) is x
    near(x[:, :dim], want, dtype)
    assert not x[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows", [3, 40, 300])
def test_biases_and_clamped_units_in_gemm_epilogues(ops, dtype, rows):
    K = ops[0]
    x, w, b = rnd(rows, 72, dtype=dtype), rnd(272, 72, dtype=dtype, scale=0.3), rnd(272, seed=5)
    z = dbl(x) @ dbl(w).T
    near(K.gemm(x, w, bias=b), z + dbl(b), dtype)
    near(K.gemm(x, w, bias=b, out=torch.empty(rows, 272, device="cuda")), z + dbl(b), F32)
    near(K.gemm(x, w, bias=b, epilogue=K.EPI_GELU), VO.gelu(z + dbl(b)), dtype)
    near(K.gemm(x, w[:199], bias=b), (z + dbl(b))[:, :199], dtype)                       # odd widths
    g, u = z[:, :136], z[:, 136:]
    unit = lambda g, u, a, s: g * torch.sigmoid(a * g) * (u + s)
    near(K.gemm(x, w, epilogue=K.EPI_SWIGLU), unit(g, u, 1, 0), dtype)
    near(K.gemm(x, w, epilogue=K.EPI_SWIGLU, act_limit=1.5, act_alpha=1.702, act_shift=1.0),
         unit(g.clamp(max=1.5), u.clamp(-1.5, 1.5), 1.702, 1), dtype)
    long_k = rnd(rows, 2048, dtype=dtype), rnd(64, 2048, dtype=dtype, scale=0.1)          # few tiles: the bias joins once
    near(K.gemm(*long_k, bias=b), dbl(long_k[0]) @ dbl(long_k[1]).T + dbl(b)[:64], dtype)


@pytest.mark.parametrize("T,E,k", [(1, 4, 4), (16, 12, 3), (60, 64, 6)])
def test_router_with_logit_bias_and_a_shared_experts_gate(ops, T, E, k):
    K = ops[0]
    x, w, b = rnd(T, 96, dtype=BF), rnd(E + 1, 96, dtype=BF, scale=0.2), rnd(E, seed=3, scale=2.0)
    z = dbl(x) @ dbl(w).T
    want = VO.route(z[:, :E] + dbl(b), k)
    for static in (False, True):
        if static:
            counts = torch.zeros(E, dtype=torch.int32, device="cuda")
            plan = K.static_plan(64, E, counts)
            idx, wts, gate = i32(*[0] * (T * k)).view(T, k), torch.zeros(T, k, device="cuda"), torch.zeros(T, 1, device="cuda")
            K.router_append(x, w, k, 0, plan, 0, E, idx, wts, torch.zeros(plan.cap_rows, 96, dtype=BF, device="cuda"), normalize=True,
                            dst_slots=k, logit_bias=b, extra=gate)
            near(gate, z[:, E:], F32)
        else:
            idx, wts = K.router_topk((x.float() @ w.float().T)[:, :E], k, 0, normalize=True, logit_bias=b)
        near(torch.zeros(T, E).scatter(1, idx.long().cpu(), wts.cpu()), want, F32)


# ------------------------------------------------------------------ queries, keys, values
PREPS = [pooled(6, 3, 20, 12, 0.3, 9, 4, 8), pooled(1, 1, 33, 10, 0.5, 9, 7), pooled(8, 2, 128, 128, 0.1, 9, 16), pooled(4, 4, 12, 24, 0.4, 9, 3, 0)]


def ids_of(m):
    return f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}w{m.window}p{m.pool}"


def rotation(base, dims, n=400):
    a = VO.angles(n, base, dims)
    return torch.cos(a).float().cuda().contiguous(), torch.sin(a).float().cuda().contiguous()


def rotated_at(turn, x, positions, base, dims):
    """x [n, heads, d] at the given positions."""
    far = torch.zeros(max(positions) + 1, *x.shape[1:], dtype=torch.float64)
    out = torch.empty_like(x)
    for i, p in enumerate(positions):
        far[p] = x[i]
        out[i] = turn(far, base, dims)[p]
    return out


class Img:
    q_norm = k_norm = q_bias = k_bias = None

    def __init__(self, m):
        self.q_mix = torch.full((m.heads,), m.scale).cuda()
        self.talk = (torch.eye(m.heads).cuda() + 0.4 * rnd(m.heads, m.heads, seed=8)).contiguous()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", PREPS, ids=ids_of)
def test_rotation_head_norms_and_cache_append(ops, dtype, m):
    KL, T, eps = ops[1], 9, 1e-4
    H, G, D, V, dp, vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_pad, m.vdim_pad
    off = {"q": 0, "k": H * dp, "v": (H + G) * dp}
    proj = torch.zeros(T, (H + G) * dp + G * vp + 8, dtype=dtype, device="cuda")
    qs, ks, vs = rnd(T, H, D, dtype=dtype), rnd(T, G, D, dtype=dtype, seed=1), rnd(T, G, V, dtype=dtype, seed=2)
    ks[:, 0] *= 8                                       # heads of very different size: every head has its own norm
    for name, t, n in (("q", qs, dp), ("k", ks, dp), ("v", vs, vp)):
        proj[:, off[name]:off[name] + t.shape[1] * n].unflatten(1, (-1, n))[..., :t.shape[2]] = t
    pos = [0, 1, 2, 77, 5, 300, 399, 8, 13]
    pool = torch.full((3, 5, m.row_dim + 16), 9.0, dtype=dtype, device="cuda")
    slots = torch.tensor([5, 0, 14, -1, 2, 9, 1, 8, 13], device="cuda")
    q = proj[:, :H * dp]                                # in place
    KL.head_prep(proj, off, m, Img(m), slots, pool, eps, q, rotation(m.rot_base, m.rot_dims), i32(*pos))
    turn = lambda t: VO.rms(rotated_at(VO.rotate_halves, dbl(t), pos, m.rot_base, m.rot_dims), eps)
    near(q.unflatten(1, (H, dp))[..., :D], turn(qs) * m.scale, dtype)
    flat, keep = pool.view(15, -1), (slots >= 0).cpu()
    at = slots[slots >= 0]
    near(flat[at, :G * dp].unflatten(1, (G, dp))[..., :D], turn(ks)[keep], dtype)
    near(flat[at, m.v_offset:m.v_offset + G * vp].unflatten(1, (-1, vp))[..., :V], dbl(vs)[keep], dtype)
    assert (flat[[i for i in range(15) if i not in slots.tolist()]] == 9.0).all()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("page,P", [(8, 3), (8, 8), (16, 40), (64, 1)])
def test_mean_rows_of_blocks(ops, dtype, page, P):
    """A launch for any batch, and the tail of the append for single rows: exactly the blocks that end with the batch's rows."""
    KL, m = ops[1], pooled(4, 2, 16, 8, 0.3, 9, P)
    lens, div = (90, 41, 80), 3
    per = [(n + page - 1) // page for n in lens]
    ids = list(range(sum(per) + 2))
    random.Random(1).shuffle(ids)
    table = torch.zeros(3, max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([ids.pop() for _ in range(n)])
    pool = rnd(sum(per) + 2, page, m.row_dim, dtype=dtype)
    flat = dbl(pool).flatten(0, 1)
    stride = 90 // P + 2
    mean = torch.full((5, stride, m.row_dim), 9.0, dtype=dtype, device="cuda")
    slots = i32(3 * 4 + 1, -1, 2)                       # buffer numbers of slots 4 and 0; a sequence without a slot
    rows = [(0, p) for p in range(30, 90)] + [(1, 40)] + [(2, p) for p in range(80)] + [(0, -1)]
    KL.pool_blocks(m, pool, (mean, div, slots), i32(*[p for _, p in rows]), i32(*[s for s, _ in rows]), table.cuda(), page)
    written = set()
    for s, p in rows:
        if s != 1 and p >= 0 and (p + 1) % P == 0:
            t = [int(table[s, j // page]) * page + j % page for j in range(p + 1 - P, p + 1)]
            slot = {0: 4, 2: 0}[s]
            near(mean[slot, p // P], flat[t].mean(0), dtype)
            written.add((slot, p // P))
    assert written and all((mean[a, b] == 9.0).all() for a in range(5) for b in range(stride) if (a, b) not in written)
    # one row per sequence, behind the append of that row itself
    H, G, dp, vp = 4, 2, m.dim_pad, m.vdim_pad
    proj = rnd(3, (H + G) * dp + G * vp, dtype=dtype)
    last = [max(p for p in range(n) if (p + 1) % P == 0) for n in lens]
    where = torch.tensor([int(table[s, p // page]) * page + p % page for s, p in enumerate(last)], device="cuda")
    mean.fill_(9.0)
    KL.head_prep(proj, {"q": 0, "k": H * dp, "v": (H + G) * dp}, m, Img(m), where, pool, 1e-5, proj[:, :H * dp],
                 rotation(m.rot_base, m.rot_dims), i32(*last), ((mean, div, slots), i32(*last), i32(0, 1, 2), table.cuda(), page))
    flat = dbl(pool).flatten(0, 1)
    for s, slot in ((0, 4), (2, 0)):
        t = [int(table[s, j // page]) * page + j % page for j in range(last[s] + 1 - P, last[s] + 1)]
        near(mean[slot, last[s] // P], flat[t].mean(0), dtype)
    assert int((mean != 9.0).any(-1).sum()) == 2


# ------------------------------------------------------------------ attention with pooled blocks and mixed weights
ATTENTIONS = [pooled(6, 3, 20, 12, 0.3, 9, 4), pooled(1, 1, 64, 40, 0.3, 1, 1), pooled(8, 2, 128, 128, 0.3, 70, 16),
              pooled(20, 4, 40, 16, 0.3, 130, 7), pooled(16, 4, 128, 128, 0.3, 64, 5, softcap=30.0), pooled(6, 2, 64, 80, 0.3, 17, 40),
              pooled(40, 2, 24, 64, 0.3, 33, 3), pooled(4, 4, 72, 136, 0.3, 20, 64, softcap=0.0), pooled(3, 3, 16, 200, 0.3, 300, 2),
              pooled(12, 3, 48, 48, 0.2, 100, 16, softcap=20.0)]


def attention_case(m, dtype, page, lens, rows=None, seed=0):
    """Paged pool with shuffled pages and mean rows in slots; query rows around every page border, window edge and block edge.
    One score stands out per head: that of the oldest token in the window, of the one before it, of the last block seen, of the
    next block, of the first block, of the row itself."""
    g = random.Random(seed)
    per = [(n + page - 1) // page for n in lens]
    ids = list(range(sum(per) + 3))
    g.shuffle(ids)
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([ids.pop() for _ in range(n)])
    if rows is None:
        edge = {m.window, m.pool, m.window + m.pool, m.window + 2 * m.pool}
        rows = [(s, p) for s, n in enumerate(lens)
                for p in sorted({k * page + o for k in range(n // page + 1) for o in (-1, 0)} | {e + o for e in edge for o in (-2, -1, 0, 1)}
                                | {n - 1}) if 0 <= p < n]
    H, G, D, V, dp, vp = m.heads, m.kv_heads, m.dim, m.vdim, m.dim_pad, m.vdim_pad
    pool = torch.zeros(sum(per) + 3, page, m.row_dim + 8, dtype=dtype, device="cuda")
    # a kernel may rely on a bound of the scores that the norms of queries and keys give: such mixers get normalised ones
    bounded = 0 < m.score_bound <= 0.7 * m.softcap
    keys = rnd(*pool.shape[:2], G, D)
    pool[..., :G * dp].unflatten(2, (G, dp))[..., :D] = (VO.rms(keys, 0.0) if bounded else keys).to(dtype)
    pool[..., m.v_offset:m.v_offset + G * vp].unflatten(2, (G, vp))[..., :V] = rnd(*pool.shape[:2], G, V, dtype=dtype, seed=1)
    flat, img = dbl(pool).flatten(0, 1), Img(m)
    slot = lambda s, t: int(table[s, t // page]) * page + t % page
    # mean rows: sequence s in slot n - 1 - s; rows no sequence has are large, so that reading one shows
    n, stride = len(lens), max(lens) // m.pool + 3
    mean = torch.full((n, stride, m.row_dim + 8), 50.0, dtype=dtype, device="cuda")
    for s, length in enumerate(lens):
        for b in range(length // m.pool):
            mean[n - 1 - s, b] = flat[[slot(s, b * m.pool + i) for i in range(m.pool)]].mean(0).to(dtype)
    means = dbl(mean)
    q = dbl(rnd(len(rows), H, D, scale=0.3, seed=2))
    want = torch.zeros(len(rows), H, V, dtype=torch.float64)
    for i, (s, p) in enumerate(rows):
        lo = max(p - m.window + 1, 0)
        blocks = lo // m.pool
        key = {"old": lo, "before": lo - 1, "self": p}
        targets = [flat[slot(s, t)] if t >= 0 else None for t in key.values()]
        targets += [means[n - 1 - s, b] if 0 <= b < lens[s] // m.pool else None for b in (blocks - 1, blocks, 0)]
        for h, t in enumerate(targets):
            if t is not None and h < H:
                kv = h // (H // G)
                t = t[kv * dp:kv * dp + D]
                q[i, h] = t * (8.0 / float(t.norm() ** 2))
        if bounded:
            q[i] *= D ** 0.5 * m.scale / q[i].norm(dim=-1, keepdim=True)
        qi = q[i].to(dtype).double()
        kv = torch.cat([means[n - 1 - s, :blocks], flat[[slot(s, t) for t in range(lo, p + 1)]]])
        w = []
        for h in range(H):
            c = h // (H // G) * dp
            w.append(torch.softmax(VO.softcap(kv[:, c:c + D] @ qi[h], m.softcap), 0))
        w = VO.mixed_weights(torch.stack(w), dbl(img.talk))
        for h in range(H):
            c = m.v_offset + h // (H // G) * vp
            want[i, h] = w[h] @ kv[:, c:c + V]
    rows_q = torch.nn.functional.pad(q, (0, dp - D)).flatten(1).to(dtype).cuda()
    return pool, table.cuda(), rows_q, rows, want, dict(mean=(mean, 3, i32(*[3 * (n - 1 - s) + s % 3 for s in range(n)]))), img.talk


def check_rows(out, want, m, dtype):
    near(out.unflatten(1, (m.heads, -1))[..., :m.vdim], want, dtype)
    assert not out.unflatten(1, (m.heads, -1))[..., m.vdim:].any()


def rows_of(m, rows, dtype):
    return (torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=dtype, device="cuda"),
            torch.full((len(rows), m.heads * m.value_width), 7.0, dtype=dtype, device="cuda"),
            i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]))


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("m", ATTENTIONS, ids=ids_of)
def test_attention_in_windows_and_blocks(ops, dtype, m, page):
    KL = ops[1]
    pool, table, q, rows, want, form, talk = attention_case(m, dtype, page, [1, 40, 200])
    out, o, seq, pos = rows_of(m, rows, dtype)
    KL.gqa_attention(q, m, pool, table, seq, pos, page, o, **form)
    check_rows(KL.value_mix(o, talk, m, out), want, m, dtype)


@pytest.mark.parametrize("page,splits,early", [(16, 1, False), (64, 2, False), (8, 4, True), (16, 8, True)])
@pytest.mark.parametrize("m", ATTENTIONS, ids=ids_of)
def test_attention_of_few_rows(ops, m, page, splits, early):
    KL = ops[1]
    assert KL.gqa_decode_supported(m, BF, page)
    pool, table, q, rows, want, form, talk = attention_case(m, BF, page, [1, 40, 300])
    out, _, seq, pos = rows_of(m, rows, BF)
    splits = min(splits, {1: 8, 2: 4, 3: 2}[(m.heads + 15) // 16])
    KL.gqa_decode(q, m, pool, table, seq, pos, page, out, splits=splits, decode_only=early, talk=talk, **form)
    check_rows(out, want, m, BF)


@pytest.mark.parametrize("page", [8, 64, 128])
@pytest.mark.parametrize("m", ATTENTIONS, ids=ids_of)
def test_prompt_attention_on_tensor_cores(ops, m, page):
    """Tiles that start and end anywhere: inside a window, at its edge, in the middle of a block; portions that continue."""
    K, KL = ops
    parts = ((90, 0), (70, 130), (33, 27), (1, 64), (2, 400))
    rows = [(s, p0 + i) for s, (n, p0) in enumerate(parts) for i in range(n)]
    pool, table, q, rows, want, form, talk = attention_case(m, BF, page, [p0 + n for n, p0 in parts], rows)
    segs, r0 = [], 0
    for s, (n, p0) in enumerate(parts):
        segs.append((s, r0, n, p0))
        r0 += n
    per = KL.gqa_tc_group(m, BF, page)
    assert per == m.heads // m.kv_heads
    for group in {per, min(2 * per, 128)}:               # also tiles another layer's groups limit
        out, o, _, _ = rows_of(m, rows, BF)
        tiles, rest = K.prefill_tiles(segs, group, 2)
        assert rest == [(len(rows) - 3, len(rows) - 2)]
        KL.gqa_prefill_tc(q, m, pool, table, torch.from_numpy(tiles).cuda().contiguous(), len(tiles), 128 // group, page, o, **form)
        KL.value_mix(o, talk, m, out)
        keep = [i for i in range(len(rows)) if i != len(rows) - 3]
        check_rows(out[keep], want[keep], m, BF)
        assert (o[-3] == 7.0).all()


# ------------------------------------------------------------------ latent attention
LATENTS = [latent(3, 12, 20, 26, 30, 6, 11), latent(16, 8, 8, 500, 16, 40, 70), latent(8, 8, 8, 448, 24, 64, 1),
           latent(1, 24, 33, 15, 9, 2, 64), latent(5, 16, 8, 130, 24, 10, 65), latent(2, 8, 8, 600, 8, 16, 33)]
lat_ids = lambda m: f"{m.heads}x{m.kv_rank}r{m.rot_dim}w{m.window}"


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", LATENTS, ids=lat_ids)
def test_latent_rows_and_turned_queries(ops, dtype, m):
    KL, T, eps = ops[1], 7, 1e-3

    class L:
        dq_norm, kv_norm = 1 + 0.3 * rnd(pad8(m.q_rank), seed=3), 1 + 0.3 * rnd(m.row_dim, seed=4)

    off = {"dq": 8, "dkv": 8 + pad8(m.q_rank)}
    proj = rnd(T, off["dkv"] + pad8(m.kv_rank + m.rot_dim) + 8, dtype=dtype)
    before, pos = dbl(proj), [0, 1, 2, 77, 5, 300, 399]
    pool = torch.full((2, 5, m.row_dim), 9.0, dtype=dtype, device="cuda")
    slots, rot = torch.tensor([5, 0, 9, -1, 2, 1, 8], device="cuda"), rotation(m.rot_base, m.rot_dim)
    KL.latent_prep(proj, off, m, L, rot, i32(*pos), slots, pool, eps)
    near(proj[:, 8:8 + m.q_rank], VO.rms(before[:, 8:8 + m.q_rank], eps) * dbl(L.dq_norm)[:m.q_rank], dtype)
    c = before[:, off["dkv"]:off["dkv"] + m.kv_rank]
    k = before[:, None, off["dkv"] + m.kv_rank:off["dkv"] + m.kv_rank + m.rot_dim]
    want = torch.zeros(T, m.row_dim, dtype=torch.float64)
    want[:, :m.kv_rank] = VO.rms(c, eps) * dbl(L.kv_norm)[:m.kv_rank]
    want[:, m.rot_offset:m.rot_offset + m.rot_dim] = rotated_at(VO.rotate_pairs, k, pos, m.rot_base, m.rot_dim)[:, 0]
    flat, keep = pool.view(10, -1), slots >= 0
    near(flat[slots[keep]], want[keep.cpu()], dtype)
    assert not flat[slots[keep]][:, want.abs().sum(0).cuda() == 0].any() and (flat[[3, 4, 6, 7]] == 9.0).all()
    src, q = rnd(T, m.heads * m.rot_dim + 8, dtype=dtype, seed=6)[:, :m.heads * m.rot_dim], rnd(T, m.heads, m.row_dim, dtype=dtype, seed=7)
    want = dbl(q)
    want[..., m.rot_offset:m.rot_offset + m.rot_dim] = rotated_at(VO.rotate_pairs, dbl(src).unflatten(1, (m.heads, -1)), pos, m.rot_base, m.rot_dim)
    KL.latent_turn(src, m, rot, i32(*pos), q)
    near(q, want, dtype)


def latent_case(m, dtype, page, lens, rows):
    g = random.Random(2)
    per = [(n + page - 1) // page for n in lens]
    ids = list(range(sum(per) + 2))
    g.shuffle(ids)
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([ids.pop() for _ in range(n)])
    pool = rnd(sum(per) + 2, page, m.row_dim, dtype=dtype)
    used = torch.zeros(m.row_dim, device="cuda")
    used[:m.kv_rank] = 1
    used[m.rot_offset:m.rot_offset + m.rot_dim] = 1
    pool *= used.to(dtype)
    flat = dbl(pool).flatten(0, 1)
    slot = lambda s, t: int(table[s, t // page]) * page + t % page
    q = dbl(rnd(len(rows), m.heads, m.row_dim, scale=0.2, seed=2)) * dbl(used)
    gate = rnd(len(rows), m.heads + 3, dtype=dtype, seed=5)
    for i, (s, p) in enumerate(rows):                    # one score stands out: the window's oldest key, the one before it, the row
        lo = max(p - m.window + 1, 0)
        for h, t in enumerate((lo, lo - 1, p)):
            if 0 <= t and h < m.heads:
                q[i, h] = flat[slot(s, t)] * (6.0 / m.scale / float(flat[slot(s, t)].norm() ** 2))
    qd = q.to(dtype)
    want = torch.zeros(len(rows), m.heads, m.row_dim, dtype=torch.float64)
    for i, (s, p) in enumerate(rows):
        kv = flat[[slot(s, t) for t in range(max(p - m.window + 1, 0), p + 1)]]
        w = torch.softmax(qd[i].double() @ kv.T * m.scale, -1) * torch.sigmoid(dbl(gate)[i, :m.heads, None])
        want[i] = w @ kv
    return pool, table.cuda(), qd.cuda(), want, gate


@pytest.mark.parametrize("page,splits,early,group", [(16, 1, False, 1), (64, 8, True, 1), (8, 4, False, 1), (16, 1, False, 4)])
@pytest.mark.parametrize("m", LATENTS, ids=lat_ids)
def test_latent_attention_in_windows(ops, m, page, splits, early, group):
    K, KL = ops
    lens = [1, 40, 260]
    edges = lambda n: sorted({e + o for e in (m.window, 2 * m.window, 64, 128, n) for o in (-1, 0, 1)} | {0})
    rows = [(s, p) for s, n in enumerate(lens) for p in edges(n) if 0 <= p < n]
    if group > 1:                                        # consecutive rows of one sequence share a tile
        rows = [(2, p) for p in range(60, 84)]
    for dtype in (F32, BF):
        pool, table, q, want, gate = latent_case(m, dtype, page, lens, rows)
        seq, pos = i32(*[s for s, _ in rows]), i32(*[p for _, p in rows])
        out = torch.full_like(q, 7.0)
        KL.latent_attention(q, pool, table, seq, pos, page, m.scale, out, gate=gate, window=m.window)
        near(out, want, dtype)
    if m.value_dim > 512:
        return
    out = torch.full((len(rows), m.heads, m.value_dim), 7.0, dtype=BF, device="cuda")
    K.mla_attention(q, pool, table, seq, pos, page, m.value_dim, m.row_dim - m.value_dim, m.scale, out, splits=splits,
                    split_tokens=(1 << 29) if splits == 1 else max(64, ((m.window + 64 + splits - 1) // splits + 63) // 64 * 64),
                    decode_only=early, gate=gate, window=m.window, group_rows=group)
    near(out, want[..., :m.value_dim], BF)


@pytest.mark.parametrize("page", [8, 64])
@pytest.mark.parametrize("m", [m for m in LATENTS if m.value_dim == 512], ids=lat_ids)
def test_latent_prompt_attention_on_tensor_cores(ops, m, page):
    K, KL = ops
    parts = ((90, 0), (70, 130), (33, 27), (2, 200))
    rows = [(s, p0 + i) for s, (n, p0) in enumerate(parts) for i in range(n)]
    pool, table, q, want, gate = latent_case(m, BF, page, [p0 + n for n, p0 in parts], rows)
    segs, r0 = [], 0
    for s, (n, p0) in enumerate(parts):
        segs.append((s, r0, n, p0))
        r0 += n
    assert KL.latent_tc_group(m, BF, page) == m.heads
    tiles, _ = K.prefill_tiles(segs, m.heads, 2)
    out = torch.full((len(rows), m.heads, 512), 7.0, dtype=BF, device="cuda")
    K.mla_prefill_tc(q, pool, table, torch.from_numpy(tiles).cuda().contiguous(), len(tiles), page, 512, m.row_dim - 512, m.scale, out,
                     gate=gate, window=m.window)
    near(out, want[..., :512], BF)


# ------------------------------------------------------------------ head-decay scan
SCANS = [Mamba2Mixer(3, 5, 3, 1, 1), Mamba2Mixer(4, 16, 32, 2, 4), Mamba2Mixer(6, 72, 24, 3, 2), Mamba2Mixer(2, 64, 128, 1, 4),
         Mamba2Mixer(2, 40, 60, 1, 4), Mamba2Mixer(1, 128, 200, 1, 2), Mamba2Mixer(5, 8, 8, 5, 3)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("lens", [(1, 1, 1, 1), (1, 300, 2, 64, 1, 65), (17, 129)])
@pytest.mark.parametrize("m", SCANS, ids=lambda m: f"{m.heads}x{m.vdim}n{m.state}g{m.groups}")
def test_scan_in_steps_chunks_and_tokens(ops, dtype, lens, m):
    """Decays from nearly one to nearly zero; states carried in and out, for sequences that start and that go on."""
    KL, T, H, V, N, G = ops[1], sum(lens), m.heads, m.vdim, m.state, m.groups
    fresh = [s % 3 == 1 for s in range(len(lens))]
    _, start, sin, sout, n = batch_of(lens, fresh)
    xbc = rnd(T, m.channels + 8, dtype=dtype, scale=0.7)
    off = {"z": 0, "dt": m.inner_pad}
    proj = rnd(T, m.inner_pad + pad8(H) + 8, dtype=dtype, seed=1)

    class I:
        off_b, off_c = m.inner_pad, m.inner_pad + m.bc_pad
        dt_bias, d_skip = rnd(H, seed=2) - 1.5, rnd(H, seed=3)
        a_neg = -torch.logspace(-3, 1.5, H).cuda() if H > 1 else torch.full((1,), -0.3).cuda()

    states = rnd(3 * n, H, N, V, seed=4)
    X, Bs, Cs = dbl(xbc)[:, :m.inner].view(T, H, V), dbl(xbc)[:, I.off_b:I.off_b + G * N].view(T, G, N), dbl(xbc)[:, I.off_c:I.off_c + G * N].view(T, G, N)
    dt = VO.softplus(dbl(proj)[:, off["dt"]:off["dt"] + H] + dbl(I.dt_bias))
    A, D, rep = dbl(I.a_neg), dbl(I.d_skip), H // G
    want, ends = torch.zeros(T, H, V, dtype=torch.float64), []
    for s, length in enumerate(lens):
        S = torch.zeros(H, N, V, dtype=torch.float64) if fresh[s] else dbl(states)[3 * s]
        for t in range(int(start[s]), int(start[s]) + length):
            S = torch.exp(A * dt[t])[:, None, None] * S + dt[t][:, None, None] * Bs[t].repeat_interleave(rep, 0)[:, :, None] * X[t][:, None]
            want[t] = torch.einsum("hnv,hn->hv", S, Cs[t].repeat_interleave(rep, 0)) + D[:, None] * X[t]
        ends.append(S)
    want = want.flatten(1) * VO.silu(dbl(proj)[:, :m.inner])
    for by_token in (False, True):
        plane, out = states.clone(), torch.full((T, m.inner_pad), 7.0, dtype=dtype, device="cuda")
        KL.head_scan(xbc, proj, off, m, I, plane, start, sin, sout, n, out, long_seqs=0 if by_token else sum(k > 1 for k in lens),
                     by_token=by_token)
        for h in range(H):                               # head by head: decays differ by orders of magnitude
            near(out[:, h * V:(h + 1) * V], want[:, h * V:(h + 1) * V], dtype)
        assert not out[:, m.inner:].any()
        for s, S in enumerate(ends):
            d = (dbl(plane[3 * s + 1]) - S).abs().amax((1, 2)) / S.abs().amax((1, 2))
            assert float(d.max()) < 3e-5, (s, d)          # the state is 32-bit in bf16 models too
        untouched = [i for i in range(3 * n) if i % 3 != 1]
        assert torch.equal(plane[untouched], states[untouched])


# ------------------------------------------------------------------ whole models
_memo = {}


def model(name, dtype, gain=1.6):
    key = (name, dtype)
    if key not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=F32, gain=gain)
        _memo[key] = (cfg, pack_weights(cfg, lambda n: t(n).to(device="cuda", dtype=dtype)), VO.Oracle(to_layer_list(cfg), t))
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
    """Root mean square over a row's logits; most rows are well inside (norms and routers amplify the rounding of a few)."""
    e = np.sqrt(((np.asarray(got) - want.float().numpy()) ** 2).mean(1)) / float(want.std())
    mid, most = (5e-6, 1e-4) if dtype == F32 else (0.05, 0.6)
    assert np.median(e) < mid and e.max() < most, (float(np.median(e)), float(e.max()))


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_token_by_token(name, dtype):
    eng, oracle, cfg = engine(name, dtype)
    toks = prompt(cfg, 100, 1)
    want = oracle.logits(toks)
    same(eng.replay([ReplayEntry("w", toks, list(range(100)))], ["w"])[0], want, dtype)
    rows = [eng.replay([ReplayEntry("d", [t], [0])])[0] for t in toks]
    same(np.concatenate(rows), want, dtype)


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_stream_after_every_layer(name):
    cfg, w, oracle = model(name, F32)
    eng = engine(name, F32, pages=8, slots=1)[0]

    class Tap:
        seen = []

        def write(self, layer, stage, t):
            self.seen.append(t[:, :cfg.width].double().cpu())

        def wants(self, *_):
            return True

    eng.runner.fwd.tap = Tap()
    toks = prompt(cfg, 19, 2)
    got = eng.replay([ReplayEntry("a", toks, [18])], ["a"])[0]
    assert len(Tap.seen) == cfg.n_layers
    for x, want in zip(Tap.seen, oracle.layers(toks)):
        assert (x - want).abs().max() < 3e-4 * max(1.0, float(want.abs().max()))
    same(got, oracle.logits(toks)[18:], F32)
    Tap.seen.clear()


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


def seen(m, p, t):
    """Whether the query at p sees the token at t, itself or in its block."""
    if p < t:
        return False
    if p - t < m.window:
        return True
    return bool(getattr(m, "pool", 0)) and t // m.pool * m.pool + m.pool - 1 <= p - m.window


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page,mixer", [(8, pooled(4, 2, 16, 8, 0.5, 24, 6, softcap=0.5)),
                                        (64, pooled(2, 2, 16, 24, 0.5, 50, 16, softcap=0.5)),
                                        (16, pooled(3, 1, 16, 8, 0.5, 16, 16, softcap=0.5)),
                                        (16, pooled(2, 1, 64, 64, 0.5, 1, 7, softcap=0.5)), (16, latent(4, 16, 16, 40, 24, 8, 23)), (64, latent(16, 16, 16, 480, 24, 32, 64))],
                         ids=lambda x: f"{x.kind}{x.window}p{getattr(x, 'pool', 0)}" if hasattr(x, "kind") else str(x))
def test_a_token_is_seen_exactly_in_windows_and_blocks(page, mixer, decoded, dtype):
    """One layer without a shift and with scores that are nearly equal (no row of a tile makes another one rescale): a changed
    token changes the logits of the rows that see it, and no others."""
    cfg = vogunex(50, 32, 1e-5, 1.0, (mixer, FF))
    t = RandomTensors(cfg, seed=3, dtype=F32, gain=1.5)
    get = lambda n: torch.zeros_like(t(n)) if n.endswith("shift") else t(n) * (0.05 if n.endswith((".mix.uq", ".mix.dq")) else 1.0)
    w = pack_weights(cfg, lambda n: get(n).to(device="cuda", dtype=dtype))
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
    P = getattr(mixer, "pool", 0) or 1
    for t in sorted({0, 1, P - 1, P, 2 * P, 30, 58, 59, 60, 61, page, page - 1} & set(range(110))):
        seq = list(toks)
        seq[t] = (seq[t] + 7) % cfg.vocab_size
        moved = np.abs(logits(seq) - base).max(1)
        want = np.array([seen(mixer, p, t) for p in range(110)])
        assert not (moved[~want] > 0).any(), t
        assert (moved[want] > 0).mean() > (0.95 if dtype == F32 else 0.6) and moved[t] > 1e-3, t


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


@pytest.mark.parametrize("name", ["attention", "scan"])
def test_long_decoding(name):
    """150 decoded tokens slide every window and complete many blocks."""
    eng, oracle, cfg = engine(name, F32, pages=12, slots=1, cls=Engine, rows=64)
    p, toks = prompt(cfg, 5, 21), []
    eng.submit(GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True))
    eng.run_until_idle(lambda ev: toks.append(ev.token) if isinstance(ev, TokenEvent) else None)
    seq = p + toks
    assert toks == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]


def test_one_table_of_tiles_per_kind_of_attention():
    """Attention groups of 4 and latent heads of 16 have tiles of their own; bf16, all on tensor cores."""
    cfg = vogunex(90, 64, 1e-5, 1.0, (pooled(8, 2, 32, 32, 0.3, 40, 8), FF), (latent(16, 16, 16, 512, 32, 64, 50), moe(8, 2, 32, 1.0, 32, 1.0)),
                  (Mamba2Mixer(4, 32, 32, 2, 4), FF))
    cfg = replace(cfg, layers=cfg.layers + (replace(cfg.layers[0], weights_of=0),))
    t = RandomTensors(cfg, seed=9, dtype=F32, gain=1.3)
    w, oracle = pack_weights(cfg, lambda n: t(n).to(device="cuda", dtype=BF)), VO.Oracle(to_layer_list(cfg), t)
    runner = LayeredRunner(w, n_pages=8, page_size=64, max_rows=512, max_seqs=4, max_seq_len=512, full_logit_rows=64)
    assert runner.staging.tc_forms == (4, 16)
    eng = ReplayEngine(runner, EngineConfig(scheduler=SchedulerConfig(4, 4, 512, 512, ctx_size=512), kv_pages=8, page_size=64))
    a, b, c = prompt(cfg, 150, 1), prompt(cfg, 90, 2), prompt(cfg, 40, 3)
    out = [[], [], []]
    for cut in (((0, 1), (0, 50), (0, 20)), ((1, 100), (50, 51), (20, 21)), ((100, 150), (51, 90), (21, 40))):
        got = eng.replay([ReplayEntry(n, s[x:y], list(range(y - x))) for n, s, (x, y) in zip("abc", (a, b, c), cut)])
        for o, rows in zip(out, got):
            o.append(rows)
    for s, o in zip((a, b, c), out):
        same(np.concatenate(o), oracle.logits(s), BF)
