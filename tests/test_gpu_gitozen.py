"""Gitozen on the sm_100a kernels: every kernel against the plain equations, whole models in 32 bits and in bf16 against
an independent oracle (whole prompts, portions, decoding, mixed batches, reused pages and slots), generation through
the engine with captured decode graphs and look-ahead."""
import math
import random
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from ferrule_b200.models.layered_config import DeltaMixer, LatentMixer, LayeredConfig, LayerSpec, MoeSpec
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.ops import reference as ref
from ferrule_b200.runtime.engine import Engine, EngineConfig, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
from gitozen_configs import CONFIGS  # noqa: E402
from gitozen_oracle import Oracle, causal_conv, decay, delta_recurrence, rms, unit  # noqa: E402

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


# ------------------------------------------------------------------ row operators
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,vector", [(52, False), (2048, False), (4100, True)])
def test_embed_norm(ops, dtype, dim, vector):
    KL = ops[1]
    pad = (dim + 7) // 8 * 8
    table = torch.zeros(33, pad, dtype=dtype, device="cuda")
    table[:, :dim] = rnd(33, dim, dtype=dtype)
    ids = torch.tensor([3, 32, 0, 3], dtype=torch.int32, device="cuda")
    g = rnd(dim) if vector else torch.tensor([1.3], device="cuda")
    x, h = torch.full((4, pad), 7.0, device="cuda"), torch.full((4, pad), 7.0, dtype=dtype, device="cuda")
    KL.embed_norm(ids, table, x, g, h, dim, 1e-5)
    assert torch.equal(x[:, :dim], table[ids.long(), :dim].float())
    near(h[:, :dim], rms(x[:, :dim].double(), 1e-5) * g.double(), dtype)
    assert not h[:, dim:].any() and not x[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("dim,topk,gated", [(52, 2, True), (2048, 6, True), (300, 1, False), (64, 0, True)])
def test_gated_residual_norm(ops, dtype, dim, topk, gated):
    KL = ops[1]
    pad, T = (dim + 7) // 8 * 8, 5
    z = lambda *s, **kw: torch.nn.functional.pad(rnd(*s, **kw), (0, pad - s[-1])).contiguous()
    x, mix, g1, g2 = z(T, dim, seed=1), z(T, dim, dtype=dtype, seed=2), z(T, dim, dtype=dtype, seed=3), z(T, dim, dtype=dtype, seed=4)
    b1, b2 = z(dim, seed=5), z(dim, seed=6)
    ffn = z(T, topk, dim, dtype=dtype, seed=7) if topk else None
    h = torch.empty(T, pad, dtype=dtype, device="cuda")
    want = x.double() + mix.double() * (torch.sigmoid(g1.double() + b1.double()) if gated else 1)
    if topk:
        want = want + ffn.double().sum(1) * (torch.sigmoid(g2.double() + b2.double()) if gated else 1)
    kw = dict(gate1=g1, bias1=b1) if gated else {}
    if topk:
        kw.update(ffn=ffn, topk=topk, **(dict(gate2=g2, bias2=b2) if gated else {}))
    KL.gated_residual_norm(x, torch.tensor([0.8], device="cuda"), h, dim, 1e-6, mix=mix, **kw)
    near(x[:, :dim], want[:, :dim], F32)                      # the residual sum is 32-bit whatever the activations are
    near(h[:, :dim], rms(want[:, :dim], 1e-6) * 0.8, dtype)
    assert not h[:, dim:].any()


@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_append_and_softcap(ops, dtype):
    KL = ops[1]
    rank, D, T = 36, 64, 6
    src = rnd(T, 80, dtype=dtype)
    w = torch.zeros(D, device="cuda")
    w[:rank] = rnd(rank)
    slots = torch.tensor([5, -1, 0, 17, 2, 9], dtype=torch.int64, device="cuda")
    pool = torch.full((3, 6, D), 9.0, dtype=dtype, device="cuda")
    KL.latent_append(src, rank, w, 1e-5, slots, pool)
    flat = pool.view(-1, D)
    keep = slots >= 0
    near(flat[slots[keep], :rank], (rms(src[:, :rank].double(), 1e-5) * w[:rank].double())[keep], dtype)
    assert not flat[slots[keep], rank:].any()
    rest = [i for i in range(18) if i not in slots.tolist()]
    assert (flat[rest] == 9.0).all()
    z = rnd(3, 1001, scale=9.0)
    want = 6.0 * torch.tanh(z.double() / 6.0)
    near(KL.softcap_(z, 6.0), want, F32)


@pytest.mark.parametrize("case", ["dense", "batched", "swiglu", "grouped"])
def test_gemm_in_32_bits(ops, case):
    K = ops[0]
    if case == "dense":
        x, w = rnd(70, 131), rnd(90, 131)
        near(K.gemm(x, w), x.double() @ w.double().T, F32)
    elif case == "batched":
        x, w, out = rnd(9, 3 * 24), rnd(3, 40, 24), torch.zeros(9, 120, device="cuda")
        K.gemm(x, w, out=out, x_group_koff=24, out_group_coff=40)
        near(out.view(9, 3, 40), torch.einsum("tgk,gnk->tgn", x.view(9, 3, 24).double(), w.double()), F32)
    elif case == "swiglu":
        x, w = rnd(33, 50), rnd(2 * 72, 50)
        y = x.double() @ w.double().T
        near(K.gemm(x, w, epilogue=K.EPI_SWIGLU), torch.nn.functional.silu(y[:, :72]) * y[:, 72:], F32)
    else:
        T, E, k = 150, 5, 2
        x, w = rnd(T, 40), rnd(E, 48, 40)
        idx = torch.stack([torch.randperm(E, generator=torch.Generator().manual_seed(i))[:k] for i in range(T)]).int().cuda()
        wts = rnd(T, k)
        plan = K.MoePlan.allocate(T * k, E, 128, "cuda")
        K.moe_plan(idx, wts, plan, 0, E, dst_slots=k)
        xg, out = torch.zeros(T * k, 40, device="cuda"), torch.zeros(T * k, 48, device="cuda")
        K.gather_rows(x.view(BF), plan, xg.view(BF), cap_rows=T * k)
        K.gemm(xg, w, out=out, epilogue=K.EPI_SCATTER, plan=plan, scatter_rows=T * k)
        want = torch.einsum("tk,tkn->tkn", wts.double(), torch.einsum("tj,tknj->tkn", x.double(), w.double()[idx.long()]))
        near(out.view(T, k, 48), want, F32)


@pytest.mark.parametrize("E,groups,keep,top", [(10, 2, 1, 3), (6, 3, 2, 2), (64, 8, 3, 6), (5, 5, 2, 2), (7, 1, 1, 3)])
def test_router_groups_by_their_best_expert(ops, E, groups, keep, top):
    K = ops[0]
    logits = rnd(40, E, scale=2.0)
    # a group with one strong expert and weak others must win over one with two good ones
    logits[0] = torch.where(torch.arange(E) % (E // groups) == 0, 0.0, 1.0).cuda()
    logits[0, 0] = 5.0
    idx, w = K.router_topk(logits, top, ref.SCORE_SOFTMAX, n_groups=groups, topk_groups=keep, group_top=1)
    wi, ww = ref.route(logits.cpu(), top, n_groups=groups, topk_groups=keep, group_top=1)
    from gitozen_oracle import choose_experts
    s = torch.softmax(logits.double().cpu(), -1)
    assert idx.tolist() == wi.tolist() == choose_experts(s, MoeSpec(E, top, 1, groups, keep))
    near(w, s.gather(1, idx.long().cpu()), F32)


# ------------------------------------------------------------------ latent attention
def attention_case(dtype, D, heads, page, lens, seed=0):
    """Paged pool of several sequences with shuffled pages; one query row per listed (sequence, position)."""
    g = random.Random(seed)
    per = [(n + page - 1) // page for n in lens]
    pages = list(range(sum(per) + 3))
    g.shuffle(pages)
    kv = rnd(len(pages), page, D, dtype=dtype, seed=seed)
    table = torch.zeros(len(lens), max(per), dtype=torch.int32)
    for s, n in enumerate(per):
        table[s, :n] = torch.tensor([pages.pop() for _ in range(n)])
    rows = [(s, p) for s, n in enumerate(lens) for p in sorted({0, 1, page - 1, page, page + 1, n - 1}) if p < n]
    row_seq = torch.tensor([s for s, _ in rows], dtype=torch.int32).cuda()
    row_pos = torch.tensor([p for _, p in rows], dtype=torch.int32).cuda()
    return kv, table.cuda(), row_seq, row_pos, rnd(len(rows), heads, D, dtype=dtype, scale=0.3, seed=seed + 1), rows


def attend(kv, table, page, q, gate, rows, scale):
    out = torch.zeros(q.shape, dtype=torch.float64)
    flat, tab = kv.view(-1, kv.shape[-1]).double().cpu(), table.cpu()
    for i, (s, p) in enumerate(rows):
        t = torch.arange(p + 1)
        c = flat[tab[s, t // page].long() * page + t % page]
        out[i] = torch.softmax(q[i].double().cpu() @ c.T * scale, -1) @ c * torch.sigmoid(gate[i].double().cpu())[:, None]
    return out


@pytest.mark.parametrize("dtype,D,heads", [(F32, 64, 3), (F32, 192, 1), (F32, 576, 2), (BF, 640, 2), (BF, 64, 5), (BF, 128, 3),
                                           (BF, 192, 16), (BF, 256, 2), (BF, 320, 4), (BF, 384, 1), (BF, 448, 20), (BF, 512, 16)])
def test_latent_attention(ops, dtype, D, heads):
    K, KL = ops
    page = 16
    kv, table, row_seq, row_pos, q, rows = attention_case(dtype, D, heads, page, [1, 40, 16, 150])
    gate = rnd(len(rows), 24, dtype=dtype, seed=5)
    # far keys: for some rows one early token stands out, the first one, the last of a page, the first of a page
    flat = kv.view(-1, D)
    for i, (s, p) in enumerate(rows):
        if p > 100:
            for t in (0, page - 1, page):
                key = flat[int(table[s, t // page]) * page + t % page]
                q[i, t % heads] = (key.float() * (40.0 / float(key.float().norm() ** 2))).to(dtype)
    want = attend(kv, table, page, q, gate[:, :heads], rows, 0.9)
    out = torch.full_like(q, 7.0)
    if dtype == F32 or D > 512:
        KL.latent_attention(q, kv, table, row_seq, row_pos, page, 0.9, out, gate=gate)
        near(out, want, dtype)
        return
    for splits, tokens in ((1, 1 << 20), (2, 128), (8, 64)):
        K.mla_attention(q, kv, table, row_seq, row_pos, page, D, 0, 0.9, out, splits=splits, split_tokens=tokens, gate=gate)
        near(out, want, dtype)


@pytest.mark.parametrize("heads,page", [(16, 64), (4, 16), (1, 32)])
def test_prefill_attention_without_a_rotary_part(ops, heads, page):
    K = ops[0]
    D = 512
    lens = [90, 200]
    kv, table, _, _, _, _ = attention_case(BF, D, heads, page, lens)
    segs, rows, r0 = [], [], 0
    for s, (n, p0) in enumerate(((90, 0), (70, 130))):
        segs.append((s, r0, n, p0))
        rows += [(s, p0 + i) for i in range(n)]
        r0 += n
    q = rnd(len(rows), heads, D, dtype=BF, scale=0.2)
    gate = rnd(len(rows), heads, dtype=BF, seed=3)
    tiles, rest = K.prefill_tiles(segs, heads)
    out = torch.zeros_like(q)
    K.mla_prefill_tc(q, kv, table, torch.from_numpy(tiles).cuda().contiguous(), len(tiles), page, D, 0, 0.8, out, gate=gate)
    assert not rest
    near(out, attend(kv, table, page, q, gate, rows, 0.8), BF)


# ------------------------------------------------------------------ delta rule
def delta_case(dtype, m, lens, old, seed=0):
    """Rows of sequences of the given lengths; `old[i]`: the sequence continues from a random state."""
    T, nk, nv, nd = sum(lens), m.kv_heads * m.dim, m.heads * m.vdim, m.heads * m.dim
    pad = lambda n: (n + 7) // 8 * 8
    off, at = {}, 0
    for name, n in (("q", nk), ("k", nk), ("v", nv), ("b", m.heads)):
        off[name] = at
        at += pad(n)
    img = type("Img", (), {})()
    img.off_gate = pad(nd)
    img.conv, img.a_neg = rnd(m.taps, m.channels, seed=seed + 1), -torch.exp(rnd(m.heads, seed=seed + 2))
    img.dt_bias, img.o_norm = rnd(nd, seed=seed + 3) - 2, rnd(m.vdim, seed=seed + 4)
    n_states = 2 * len(lens) + 1
    case = dict(proj=rnd(T, at, dtype=dtype, seed=seed + 5), off=off, ag=rnd(T, img.off_gate + nv, seed=seed + 6), img=img, mixer=m,
                eps=1e-5, state=rnd(n_states, m.heads, m.dim, m.vdim, seed=seed + 7),
                tail=rnd(n_states, max(m.taps - 1, 1), m.channels, dtype=dtype, seed=seed + 8))
    starts = np.concatenate([[0], np.cumsum(lens)])
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    case.update(seq_start=i32(starts.tolist()), state_in=i32([2 * i if o else -1 for i, o in enumerate(old)]),
                state_out=i32([2 * i + 1 for i in range(len(lens))]), n_seqs=len(lens),
                row_seq=i32([i for i, n in enumerate(lens) for _ in range(n)]))
    return case, lens, old


def delta_want(case, lens, old):
    m, off, img = case["mixer"], case["off"], case["img"]
    nk, nv, keep = m.kv_heads * m.dim, m.heads * m.vdim, m.taps - 1
    proj, ag = case["proj"].double().cpu(), case["ag"].double().cpu()
    raw = torch.cat([proj[:, off["q"]:off["q"] + nk], proj[:, off["k"]:off["k"] + nk], proj[:, off["v"]:off["v"] + nv]], 1)
    conv, share = img.conv.double().cpu().T, [h // (m.heads // m.kv_heads) for h in range(m.heads)]
    outs, states, tails, at = [], [], [], 0
    for i, n in enumerate(lens):
        r = slice(at, at + n)
        before = case["tail"][2 * i, :keep].double().cpu() if old[i] else torch.zeros(keep, m.channels, dtype=torch.float64)
        x = torch.cat([before, raw[r]])
        y = causal_conv(x, conv)[keep:]
        q, k, v = y[:, :nk].view(n, -1, m.dim), y[:, nk:2 * nk].view(n, -1, m.dim), y[:, 2 * nk:].view(n, m.heads, m.vdim)
        g = decay(ag[r, :m.heads * m.dim], torch.log(-img.a_neg.double().cpu()), img.dt_bias.double().cpu(), m.heads)
        beta = torch.sigmoid(proj[r, off["b"]:off["b"] + m.heads])
        S0 = case["state"][2 * i].double().cpu() if old[i] else None
        o, S = delta_recurrence((unit(q) / math.sqrt(m.dim))[:, share], unit(k)[:, share], v, g, beta, S0)
        gate = torch.sigmoid(ag[r, img.off_gate:img.off_gate + nv]).view(n, m.heads, m.vdim)
        outs.append((rms(o, case["eps"]) * img.o_norm.double().cpu() * gate).reshape(n, -1))
        states.append(S)
        tails.append(x[x.shape[0] - keep:])
        at += n
    return torch.cat(outs), states, tails


MIXERS = [DeltaMixer(3, 3, 64, 48, 4), DeltaMixer(4, 2, 20, 12, 3), DeltaMixer(6, 1, 8, 4, 1), DeltaMixer(2, 2, 72, 33, 5),
          DeltaMixer(2, 1, 128, 128, 4), DeltaMixer(1, 1, 130, 100, 2), DeltaMixer(3, 3, 128, 160, 4), DeltaMixer(2, 2, 31, 64, 4)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m", MIXERS, ids=lambda m: f"{m.heads}x{m.kv_heads}x{m.dim}x{m.vdim}t{m.taps}")
@pytest.mark.parametrize("decode", [False, True])
def test_delta_rule(ops, dtype, m, decode):
    KL = ops[1]
    lens, old = ([1] * 5, [True, False, True, True, False]) if decode else ([1, 40, 2, 17, 3, 16], [True, True, False, False, True, True])
    if decode and not KL.delta_decode_supported(m):
        pytest.skip("served by the prefill form")
    case, lens, old = delta_case(dtype, m, lens, old)
    before = case["state"].clone(), case["tail"].clone()
    out = torch.full((sum(lens), (m.heads * m.vdim + 7) // 8 * 8), 5.0, dtype=dtype, device="cuda")
    want, states, tails = delta_want(case, lens, old)
    scratch = KL.DeltaScratch(sum(lens), [m], "cuda")
    KL.delta_rule(out=out, scratch=scratch, decode=decode, **case)
    near(out[:, :m.heads * m.vdim], want, dtype)
    for i in range(len(lens)):
        near(case["state"][2 * i + 1], states[i], F32, scale=1.0 + states[i].abs().max())
        if m.taps > 1:
            near(case["tail"][2 * i + 1, :m.taps - 1], tails[i], dtype)
        assert torch.equal(case["state"][2 * i], before[0][2 * i]) and torch.equal(case["tail"][2 * i], before[1][2 * i])
    assert torch.equal(case["state"][-1], before[0][-1])


def test_delta_rule_portions_carry_the_state_over_long_runs(ops):
    """600 tokens in portions of changing size equal one pass; slowly decaying channels remember the first token."""
    KL = ops[1]
    m = DeltaMixer(2, 1, 64, 32, 4)
    case, lens, old = delta_case(F32, m, [600], [False])
    case["ag"][:, :m.heads * m.dim:2] = -9.0                     # every other key channel hardly forgets
    want, states, _ = delta_want(case, lens, old)
    scratch = KL.DeltaScratch(600, [m], "cuda")
    at, cur, r = 0, -1, random.Random(0)
    outs = []
    while at < 600:
        n = min(r.choice([1, 2, 3, 15, 16, 17, 64, 130]), 600 - at)
        nxt = 1 - max(cur, 0) if cur >= 0 else 0
        sub = {**case, "proj": case["proj"][at:at + n], "ag": case["ag"][at:at + n]}
        i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")
        sub.update(seq_start=i32(0, n), state_in=i32(cur), state_out=i32(nxt), row_seq=torch.zeros(n, dtype=torch.int32, device="cuda"))
        out = torch.zeros(n, m.heads * m.vdim, device="cuda")
        KL.delta_rule(out=out, scratch=scratch, decode=n == 1, **sub)
        outs.append(out)
        at, cur = at + n, nxt
    near(torch.cat(outs), want, F32)
    near(case["state"][cur], states[0], F32)


def test_state_rotation(ops):
    i, o = torch.tensor([-1, 7, 3], dtype=torch.int32).cuda(), torch.tensor([0, 8, -1], dtype=torch.int32).cuda()
    ops[1].state_rotate(i, o, 3)
    assert i.tolist() == [0, 8, 3] and o.tolist() == [1, 6, -1]


# ------------------------------------------------------------------ whole models
WIDE = LayeredConfig(vocab_size=200, width=128, layers=(
    LayerSpec(LatentMixer(16, 24, 16, 512, 0.4), MoeSpec(9, 2, 48, 3, 1)),
    LayerSpec(DeltaMixer(2, 1, 128, 128, 4, 16, 16), MoeSpec(16, 4, 24, 4, 2))), logit_softcap=8.0)
ALL = {**CONFIGS, "wide": WIDE}
_memo = {}


def model(name, dtype):
    if (name, dtype) not in _memo:
        cfg = ALL[name]
        raw = RandomTensors(cfg, seed=11, gain=1.6)
        w = pack_weights(cfg, lambda n: raw(n).to(dtype).cuda())
        _memo[name, dtype] = (cfg, w)
        _memo.setdefault(name, Oracle(cfg, raw))
    return (*_memo[name, dtype], _memo[name])


def engine(name, dtype, pages=20, page=16, slots=4, cls=ReplayEngine, chunk=None, **kw):
    cfg, w, oracle = model(name, dtype)
    n = pages * page
    runner = LayeredRunner(w, n_pages=pages, page_size=page, max_rows=n, max_seqs=slots, max_seq_len=n + page, full_logit_rows=32, **kw)
    sched = SchedulerConfig(max_active_sequences=slots, max_decode_batch=slots, max_batch_tokens=n,
                            prefill_chunk_size=chunk or n, ctx_size=n + page)
    return cls(runner, EngineConfig(scheduler=sched, kv_pages=pages, page_size=page)), oracle, cfg


def prompt(cfg, n, seed):
    r = random.Random(seed)
    return [r.randrange(cfg.vocab_size) for _ in range(n)]


def same(got, want, dtype):
    d = torch.from_numpy(np.asarray(got)).double() - want
    d = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    if dtype == F32:
        assert d.max() < 1e-4, float(d.max())
        return
    # bf16 rounding can turn a close call between two experts: that moves one row, a wrong key or state moves many
    bf16_errors.extend(d.tolist())


bf16_errors = []


@pytest.fixture(autouse=True)
def _few_close_calls():
    bf16_errors.clear()
    yield
    if bf16_errors:
        d = sorted(bf16_errors)
        assert d[len(d) // 2] < 2e-2 and sum(e > 6e-2 for e in d) <= 0.08 * len(d), (d[len(d) // 2], d[-5:])


def feed(eng, rid, toks, sizes):
    at, k, out = 0, 0, []
    while at < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - at)
        k += 1
        out.append(eng.replay([ReplayEntry(rid, toks[at:at + n], list(range(n)))], [rid] if at + n == len(toks) else [])[0])
        at += n
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", list(ALL))
def test_prompts_portions_and_decoding_match_the_oracle(ops, name, dtype):
    eng, oracle, cfg = engine(name, dtype)
    toks = prompt(cfg, 83, 1)
    want = oracle.logits(toks)
    for sizes in ([83], [1], [2], [16, 3], [70, 1, 1, 1, 1]):
        same(feed(eng, "a", toks, sizes), want, dtype)
    assert eng.kv.free_pages == 20


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("name", ["both", "wide"])
def test_mixed_batches_reuse_pages_and_slots(ops, name, dtype):
    rnd_ = random.Random(3)
    eng, oracle, cfg = engine(name, dtype, pages=9)
    todo = [(f"q{i}", prompt(cfg, rnd_.choice([1, 5, 17, 33, 60]), 200 + i)) for i in range(12)]
    live = {}
    need = lambda t: (len(t) + 15) // 16
    while todo or live:
        while todo and len(live) < 4 and sum(need(t) for t, _ in live.values()) + need(todo[0][1]) <= 9:
            rid, t = todo.pop(0)
            live[rid] = (t, 0)
        entries, end = [], []
        for rid, (t, at) in list(live.items()):
            if rnd_.random() < 0.2:
                continue
            n = min(rnd_.choice([1, 1, 2, 16, 40]), len(t) - at)
            entries.append(ReplayEntry(rid, t[at:at + n], list(range(n))))
            live[rid] = (t, at + n)
            end += [rid] if at + n == len(t) else []
        for e, rows in zip(entries, eng.replay(entries, end)):
            t, at = live[e.request_id]
            same(rows, oracle.logits(t)[at - len(e.tokens):at], dtype)
        for rid in end:
            del live[rid]
    assert eng.kv.free_pages == 9 and eng.scheduler.slots.available == 4


@pytest.mark.parametrize("lookahead", [True, False])
@pytest.mark.parametrize("name", ["both", "delta"])
def test_greedy_generation_in_32_bits_equals_the_oracle(ops, name, lookahead):
    eng, oracle, cfg = engine(name, F32, cls=Engine, chunk=9, lookahead=lookahead)
    ps = {f"r{i}": prompt(cfg, n, 40 + i) for i, n in enumerate((1, 20, 3, 31, 8, 2))}
    toks = {}
    for r, p in ps.items():
        eng.submit(GenerateRequest(r, p, max_new_tokens=6 + len(p) % 5, ignore_eos=True))
    eng.run_until_idle(lambda ev: toks.setdefault(ev.request_id, []).append(ev.token) if isinstance(ev, TokenEvent) else None)
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 6 + len(p) % 5), r
    st = eng.runner.stats
    assert st.graph_steps > 0 and eng.kv.free_pages == 20 and (not lookahead or st.lookahead_hits > 0)


def test_long_generation_in_bf16_follows_the_logits_of_its_own_tokens(ops):
    """150 tokens decoded by captured graphs: each one is (nearly) the best token after the ones before it."""
    eng, oracle, cfg = engine("wide", BF, cls=Engine)
    p, toks = prompt(cfg, 30, 9), []
    eng.submit(GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True))
    eng.run_until_idle(lambda ev: toks.append(ev.token) if isinstance(ev, TokenEvent) else None)
    z = oracle.logits(p + toks)[len(p) - 1:-1]
    gap = (z.max(-1).values - z[torch.arange(len(toks)), torch.tensor(toks)]) / z.std()
    assert len(toks) == 150 and gap.quantile(0.97) < 0.1 and (gap == 0).double().mean() > 0.85
