"""Vedadra on the sm_100a kernels: every kernel against the plain equations, whole models in 32 bits and in bf16 against an
independent oracle (whole prompts, portions, decoding, mixed batches, reused pages and slots), generation through the
engine with captured decode graphs and look-ahead."""
import random
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from ferrule_b200.models.layered_config import SANDWICH_NORM, DenseSpec, LayeredConfig, LayerSpec, Loop
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.runtime.engine import Engine, EngineConfig, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
import vedadra_oracle as VO  # noqa: E402
from vedadra_configs import CONFIGS, differential, talking  # noqa: E402

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
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,groups", [(60, 3), (60, 1), (52, 13), (40, 5), (300, 2), (2048, 1), (2048, 4), (4100, 4), (4096, 64)])
def test_grouped_norms_and_residual_addition(ops, dtype, dim, groups):
    KL, T, pad, eps = ops[1], 5, pad8(dim), 1e-3
    z = lambda *s, **kw: torch.nn.functional.pad(rnd(*s, **kw), (0, pad - s[-1])).contiguous()
    # parts of very different size: a norm over the wrong part shows
    size = torch.nn.functional.pad(0.05 * 3.0 ** (torch.arange(dim) // (dim // groups) % 5), (0, pad - dim)).cuda()
    x, y, table = z(T, dim, seed=1), (z(T, dim, seed=2) * size).to(dtype), z(11, dim, dtype=dtype, seed=3)
    bias, w_out, w_in = (z(dim, seed=s) for s in (4, 5, 6))
    ids = i32(10, 0, 3, 3, 7)
    cut = lambda t: dbl(t)[..., :dim]
    kw = dict(dim=dim, eps=eps, groups=groups)
    for form in ("sublayer", "no bias", "new pass", "embedding", "tail"):
        xs, act = x.clone(), torch.full((T, pad), 7.0, dtype=dtype, device="cuda")
        b = None if form == "no bias" else bias
        args = {} if form == "embedding" else dict(y=y, bias=b, out_norm=w_out)
        if form in ("new pass", "embedding"):
            args.update(ids=ids, table=table)
        want = torch.zeros(T, dim, dtype=torch.float64) if form == "embedding" else cut(x)
        if form != "embedding":
            want = want + VO.group_rms(cut(y) + (0 if b is None else cut(b)), cut(w_out), groups, eps)
        if "ids" in args:
            want = want + cut(table)[ids.long().cpu()]
        if form != "tail":
            args.update(in_norm=w_in, act=act)
        KL.sandwich_step(xs, fresh=form == "embedding", **args, **kw)
        near(xs[:, :dim], want, F32)                                            # the stream is 32-bit either way
        assert not xs[:, dim:].any()
        if form != "tail":
            near(act[:, :dim], VO.group_rms(want, cut(w_in), groups, eps), dtype)
            assert not act[:, dim:].any()
    out = torch.full((3, pad), 7.0, dtype=dtype, device="cuda")
    KL.sandwich_rows(x, i32(4, 0, 4), w_in, out, dim, eps, groups)
    near(out[:, :dim], VO.group_rms(cut(x)[[4, 0, 4]], cut(w_in), groups, eps), dtype)
    assert not out[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows", [3, 40, 300])
def test_gated_gelu_epilogue(ops, dtype, rows):
    K = ops[0]
    x, w = rnd(rows, 72, dtype=dtype), rnd(272, 72, dtype=dtype, scale=0.5)
    z = dbl(x) @ dbl(w).T
    near(K.gemm(x, w, epilogue=K.EPI_GEGLU), VO.gelu_tanh(z[:, :136]) * z[:, 136:], dtype)


# ------------------------------------------------------------------ queries, keys, values
PREPS = [talking(6, 3, 20, 0.3, 9), talking(1, 1, 64, 0.5, 9), talking(8, 2, 128, 0.1, 9), talking(4, 4, 12, 0.4, 9),
         differential(4, 2, 12, 20, 0.5, 7, 3, 0.3), differential(3, 1, 128, 256, 0.1, 7, 0, 0.5),
         differential(1, 1, 9, 7, 0.4, 7, 1, 0.5)]


def ids_of(m):
    return f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}m{m.maps}w{m.window}k{m.keep_first}"


class Img:
    def __init__(self, m, seed=0):
        pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).reshape(-1).contiguous()
        self.w = {"q": 1 + 0.3 * rnd(m.dim, seed=seed + 3), "k": 1 + 0.3 * rnd(m.dim, seed=seed + 4)}
        self.q_norm, self.k_norm = pad(self.w["q"], m.dim_pad), pad(self.w["k"], m.dim_pad)
        self.b = {"q": rnd(m.heads, m.dim, seed=seed + 5), "k": rnd(m.kv_heads, m.dim, seed=seed + 6)}
        self.q_bias, self.k_bias = (pad(self.b[n], m.dim_pad) if m.biases else None for n in "qk")
        self.temp, self.talk = 1 + 0.3 * rnd(m.heads, seed=seed + 7), torch.eye(m.heads).cuda() + 0.4 * rnd(m.heads, m.heads, seed=seed + 8)
        self.q_mix = (self.talk * self.temp * m.scale if m.mix_heads else torch.full((m.heads,), m.scale).cuda()).contiguous()
        slopes = torch.tensor([VO.slope(h, m.heads) for h in range(m.heads)]).cuda()
        self.slopes = (self.talk @ slopes).contiguous() if m.distance_bias else None


def wide_queries(q, img, m):
    """Rows of the attention kernels from normalised queries [n, heads * maps, dim]."""
    out = torch.zeros(q.shape[0], m.heads * m.maps, m.key_width // m.dim_pad, m.dim_pad, dtype=q.dtype)
    for h in range(m.heads):
        for mp in range(m.maps):
            if not m.mix_heads:
                out[:, h * m.maps + mp, mp, :m.dim] = q[:, h * m.maps + mp] * m.scale
                continue
            for g in range(m.heads):
                out[:, h, g // (m.heads // m.kv_heads), :m.dim] += dbl(img.q_mix)[h, g] * q[:, g]
    return out.flatten(1)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", PREPS, ids=ids_of)
def test_head_norms_mixing_and_cache_append(ops, dtype, m):
    KL, T, eps = ops[1], 9, 1e-4
    H, G, D, V, dp, vp = m.heads * m.maps, m.kv_heads * m.maps, m.dim, m.vdim, m.dim_pad, m.vdim_pad
    off = {"q": 0, "k": H * dp, "v": (H + G) * dp}
    proj = torch.zeros(T, (H + G) * dp + m.kv_heads * vp + 8, dtype=dtype, device="cuda")
    qs, ks, vs = rnd(T, H, D, dtype=dtype), rnd(T, G, D, dtype=dtype, seed=1), rnd(T, m.kv_heads, V, dtype=dtype, seed=2)
    ks[:, 0] *= 8                                       # heads of very different size: every head has its own norm
    for name, t, n in (("q", qs, dp), ("k", ks, dp), ("v", vs, vp)):
        proj[:, off[name]:off[name] + t.shape[1] * n].unflatten(1, (-1, n))[..., :t.shape[2]] = t
    img = Img(m)
    pool = torch.full((3, 5, m.row_dim + 16), 9.0, dtype=dtype, device="cuda")
    slots = torch.tensor([5, 0, 14, -1, 2, 9, 1, 8, 13], device="cuda")
    out = torch.full((T, H * m.key_width), 7.0, dtype=dtype, device="cuda")
    KL.head_prep(proj, off, m, img, slots, pool, eps, out)
    q, k = dbl(qs), dbl(ks)
    if m.biases:
        q, k = q + dbl(img.b["q"]), k + dbl(img.b["k"])
    near(out, wide_queries(VO.rms(q, eps) * dbl(img.w["q"]), img, m), dtype)
    flat, keep = pool.view(15, -1), (slots >= 0).cpu()
    at = slots[slots >= 0]
    near(flat[at, :G * dp].unflatten(1, (G, dp))[..., :D], (VO.rms(k, eps) * dbl(img.w["k"]))[keep], dtype)
    near(flat[at, m.v_offset:m.v_offset + m.kv_heads * vp].unflatten(1, (-1, vp))[..., :V], (k if m.tied_values else dbl(vs))[keep], dtype)
    assert (flat[[i for i in range(15) if i not in slots.tolist()]] == 9.0).all()


# ------------------------------------------------------------------ attention
ATTENTIONS = [talking(6, 3, 20, 0.3, 9), talking(1, 1, 64, 0.3, 1, 2), talking(8, 2, 128, 0.3, 70, 5), talking(20, 4, 40, 0.3, 130),
              talking(16, 4, 128, 0.3, 64), differential(4, 2, 12, 20, 0.3, 10, 3, 0.4), differential(3, 3, 64, 64, 0.3, 37, 70, 0.8),
              differential(8, 1, 32, 128, 0.3, 96, 0, 0.1), differential(10, 1, 64, 80, 0.3, 1000, 4, 0.5),
              differential(2, 2, 128, 256, 0.3, 1, 1, 0.2)]
WIDE = [talking(9, 9, 96, 0.3, 40), talking(8, 8, 128, 0.3, 100, 3), talking(40, 2, 72, 0.3, 50), talking(32, 4, 128, 0.3, 60),
        talking(4, 2, 200, 0.3, 33)]


def visible(m, p):
    return [j for j in range(p + 1) if p - j < m.window or j < m.keep_first]


def attention_case(m, dtype, page, lens, rows=None, seed=0):
    """Paged pool with shuffled pages; query rows around every page border and window edge.  One score stands out per head:
    that of the oldest visible key, of the key just before it, of the first and the last kept token and the one behind it, of
    the row itself."""
    g = random.Random(seed)
    per = [(n + page - 1) // page for n in lens]
    ids = list(range(sum(per) + 3))
    g.shuffle(ids)
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([ids.pop() for _ in range(n)])
    if rows is None:
        edge = {m.keep_first, m.window, m.window + m.keep_first}
        rows = [(s, p) for s, n in enumerate(lens)
                for p in sorted({k * page + o for k in range(n // page + 1) for o in (-1, 0)} | {e + o for e in edge for o in (-1, 0, 1)}
                                | {n - 1}) if 0 <= p < n]
    H, G, M, D, V, dp, vp = m.heads, m.kv_heads, m.maps, m.dim, m.vdim, m.dim_pad, m.vdim_pad
    pool = torch.zeros(sum(per) + 3, page, m.row_dim + 8, dtype=dtype, device="cuda")
    pool[..., :G * M * dp].unflatten(2, (G * M, dp))[..., :D] = rnd(*pool.shape[:2], G * M, D, dtype=dtype)
    pool[..., m.v_offset:m.v_offset + G * vp].unflatten(2, (G, vp))[..., :V] = rnd(*pool.shape[:2], G, V, dtype=dtype, seed=1)
    flat, img = dbl(pool).flatten(0, 1), Img(m)
    q = dbl(rnd(len(rows), H * M, D, scale=0.3, seed=2))
    slot = lambda s, t: int(table[s, t // page]) * page + t % page
    for i, (s, p) in enumerate(rows):
        lo = max(p - m.window + 1, 0)
        for h, t in enumerate((lo, lo - 1, 0, m.keep_first - 1, m.keep_first, p)):
            if 0 <= t <= p and h < H * M:
                kv = h // M // (H // G) * M + h % M
                key = flat[slot(s, t), kv * dp:kv * dp + D]
                q[i, h] = key * (12.0 / m.scale / float(key.norm() ** 2))
    rows_q = wide_queries(q, img, m).to(dtype)
    want = []
    out_gate = rnd(len(rows), H * vp + 16, dtype=dtype, seed=9)[:, 8:8 + H * vp] if m.gate else None
    qw = rows_q.double().unflatten(1, (H * M, -1))
    for i, (s, p) in enumerate(rows):
        t = torch.tensor(visible(m, p))
        kv = flat[[slot(s, int(j)) for j in t]]
        for h in range(H):
            g = h // (H // G)
            a = []
            for mp in range(M):
                if m.shared_keys:
                    sc = kv[:, :m.key_width] @ qw[i, h]
                else:
                    sc = kv[:, g * m.key_width:(g + 1) * m.key_width] @ qw[i, h * M + mp]
                if m.distance_bias:
                    sc = sc - float(img.slopes[h]) * (p - t).double()
                a.append(torch.softmax(sc, 0) @ kv[:, m.v_offset + g * vp:m.v_offset + g * vp + V])
            want.append(a[0] if M == 1 else VO.map_difference(a[0], a[1], 0.37, m.diff, 1e-4))
    want = torch.stack(want).view(len(rows), H, V)
    if m.gate:
        want = want * torch.sigmoid(dbl(out_gate).unflatten(1, (H, vp))[..., :V])
    form = dict(slopes=img.slopes, gate=out_gate, diff_lambda=0.37 if M == 2 else 0.0, eps=1e-4)
    return pool, table.cuda(), rows_q.cuda(), rows, want, form


def check_rows(out, want, m, dtype):
    near(out.unflatten(1, (m.heads, -1))[..., :m.vdim], want, dtype, scale=None if m.maps == 1 else 1.0)
    assert not out.unflatten(1, (m.heads, -1))[..., m.vdim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("m", ATTENTIONS + WIDE, ids=ids_of)
def test_attention_in_windows(ops, dtype, m, page):
    KL = ops[1]
    pool, table, q, rows, want, form = attention_case(m, dtype, page, [1, 40, 200])
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=dtype, device="cuda")
    KL.gqa_attention(q, m, pool, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), page, out, **form)
    check_rows(out, want, m, dtype)


@pytest.mark.parametrize("page,splits,early", [(16, 1, False), (64, 2, False), (8, 4, True), (16, 8, True)])
@pytest.mark.parametrize("m", ATTENTIONS + WIDE, ids=ids_of)
def test_attention_of_few_rows(ops, m, page, splits, early):
    KL = ops[1]
    assert KL.gqa_decode_supported(m, BF, page)
    pool, table, q, rows, want, form = attention_case(m, BF, page, [1, 40, 300])
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=BF, device="cuda")
    KL.gqa_decode(q, m, pool, table, i32(*[s for s, _ in rows]), i32(*[p for _, p in rows]), page, out, splits=splits,
                  decode_only=early, **form)
    check_rows(out, want, m, BF)


@pytest.mark.parametrize("page", [8, 64, 128])
@pytest.mark.parametrize("m", ATTENTIONS + WIDE, ids=ids_of)
def test_prompt_attention_on_tensor_cores(ops, m, page):
    """Tiles that start and end anywhere: inside a window, at its edge, beside kept tokens; portions that continue."""
    K, KL = ops
    parts = ((90, 0), (70, 130), (33, 27), (1, 64))
    rows = [(s, p0 + i) for s, (n, p0) in enumerate(parts) for i in range(n)]
    pool, table, q, rows, want, form = attention_case(m, BF, page, [p0 + n for n, p0 in parts], rows)
    segs, r0 = [], 0
    for s, (n, p0) in enumerate(parts):
        segs.append((s, r0, n, p0))
        r0 += n
    out = torch.full((len(rows), m.heads * m.vdim_pad), 7.0, dtype=BF, device="cuda")
    per = KL.gqa_tc_group(m, BF, page)
    assert per == m.heads // m.kv_heads * m.maps
    for group in {per, min(2 * per, 128)}:               # also tiles another layer's groups limit
        tiles, rest = K.prefill_tiles(segs, group, 2)
        assert rest == [(len(rows) - 1, len(rows))]
        KL.gqa_prefill_tc(q, m, pool, table, torch.from_numpy(tiles).cuda().contiguous(), len(tiles), 128 // group, page, out, **form)
        check_rows(out[:-1], want[:-1], m, BF)
        assert (out[-1] == 7.0).all()


# ------------------------------------------------------------------ whole models
_memo = {}


def model(name, dtype, gain=1.6):
    key = (name, dtype)
    if key not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=F32, gain=gain)
        _memo[key] = (cfg, pack_weights(cfg, lambda n: t(n).to(device="cuda", dtype=dtype)), VO.Oracle(cfg, t))
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
    """Root mean square over a row's logits; most rows are well inside (norms amplify the rounding of a few)."""
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


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_stream_after_every_run(name):
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
    assert len(Tap.seen) == len(cfg.runs)
    for x, want in zip(Tap.seen, oracle.layers(toks)):
        assert (x - want).abs().max() < 3e-4
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


def edge_config(mixer, loop=None):
    return LayeredConfig(50, 32, (LayerSpec(mixer, DenseSpec(24, True)),), 1e-5, name="vedadra", block=SANDWICH_NORM, norm_groups=2,
                         loop=loop)


def flat_scores(t):
    """Weights whose attention is nearly uniform and whose heads are mixed evenly: every visible key shows."""
    def get(name):
        x = t(name)
        if name.endswith((".mix.q", ".mix.k.norm")):
            return x * 0.05
        return torch.full_like(x, 0.01) if name.endswith(".talk") else x
    return get


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page,mixer", [(8, talking(4, 2, 16, 0.5, 24)), (64, talking(2, 2, 16, 0.5, 50, 3)), (16, talking(3, 1, 16, 0.5, 16)),
                                        (16, differential(2, 1, 16, 16, 0.5, 17, 5, 0.5)), (8, differential(4, 2, 16, 24, 0.5, 40, 1, 0.3))],
                         ids=lambda x: ids_of(x) if hasattr(x, "maps") else str(x))
def test_a_token_is_seen_exactly_in_windows_and_among_the_kept(page, mixer, decoded, dtype):
    """One layer: a changed token changes the logits of the rows that see it, and no others."""
    cfg = edge_config(mixer)
    get = flat_scores(RandomTensors(cfg, seed=3, dtype=F32, gain=1.5))
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
    k, win = mixer.keep_first, mixer.window
    for t in sorted({0, k - 1, k, k + 1, 58, 59, 60, 61, page, page - 1} & set(range(110))):
        seq = list(toks)
        seq[t] = (seq[t] + 7) % cfg.vocab_size
        moved = np.abs(logits(seq) - base).max(1)
        want = np.array([p >= t and (p - t < win or t < k) for p in range(110)])
        assert not (moved[~want] > 0).any(), t
        assert (moved[want] > 0).mean() > (0.95 if dtype == F32 else 0.8) and moved[t] > 1e-3, t


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


def test_long_decoding_and_three_passes():
    """150 decoded tokens slide every window many times over; one layer that runs three times has three cache planes."""
    cfg = edge_config(talking(2, 1, 24, 0.5, 21, 2), Loop(0, 1, 3))
    t = RandomTensors(cfg, seed=5, dtype=F32, gain=1.6)
    w, oracle = pack_weights(cfg, lambda n: t(n).cuda()), VO.Oracle(cfg, t)
    runner = LayeredRunner(w, n_pages=12, page_size=16, max_rows=64, max_seqs=1, max_seq_len=192)
    assert runner.pool.n_layers == 3
    eng = Engine(runner, EngineConfig(scheduler=SchedulerConfig(1, 1, 64, 64, ctx_size=192), kv_pages=12, page_size=16))
    p, toks = prompt(cfg, 5, 21), []
    eng.submit(GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True))
    eng.run_until_idle(lambda ev: toks.append(ev.token) if isinstance(ev, TokenEvent) else None)
    seq = p + toks
    assert toks == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]
