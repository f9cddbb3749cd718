"""Supisun on the CPU path: configuration and checkpoint handling, the reference forward against an independent oracle,
state and page bookkeeping, generation through the engine, replay of token streams and the trace runner program."""
import json
import random
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from ferrule_b200.io.layered_checkpoint import export_layered, load_layered
from ferrule_b200.io.safetensors import CheckpointError
from ferrule_b200.models.families import Family, TensorRole, classify, detect_family
from ferrule_b200.models.layered_config import (OUTPUT_NORM, AttentionMixer, DenseSpec, LayeredConfig, LayerSpec, from_layer_list,
                                                tiny_supisun, to_layer_list)
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.models.registry import architecture_of
from ferrule_b200.models.state_pool import RecurrentStatePool
from ferrule_b200.models.support import EnginePlan, ParallelismPlan, PolicySet
from ferrule_b200.runtime.engine import Engine, EngineConfig, FinishEvent, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import FinishReason, GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
import supisun_oracle as SO  # noqa: E402
from supisun_configs import CONFIGS  # noqa: E402

_memo = {}


def model(name, gain=1.6):
    if (name, gain) not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=torch.float32, gain=gain)
        _memo[name, gain] = (cfg, pack_weights(cfg, t), SO.Oracle(cfg, t))
    return _memo[name, gain]


def make_engine(cfg, w, pages=24, page=8, slots=4, cls=ReplayEngine, **kw):
    n = pages * page
    runner = LayeredRunner(w, n_pages=pages, page_size=page, max_rows=n, max_seqs=slots, max_seq_len=n + page)
    sched = SchedulerConfig(max_active_sequences=slots, max_decode_batch=slots, max_batch_tokens=n, prefill_chunk_size=n,
                            ctx_size=n + page, **kw)
    return cls(runner, EngineConfig(scheduler=sched, kv_pages=pages, page_size=page))


def engine(name, **kw):
    cfg, w, oracle = model(name)
    return make_engine(cfg, w, **kw), oracle, cfg


def prompt(cfg, n, seed):
    r = random.Random(seed)
    return [r.randrange(cfg.vocab_size) for _ in range(n)]


def same(got, want, tol=1e-4):
    """Root mean square over a row's logits (a norm over nearly equal values amplifies the rounding of a few rows)."""
    d = np.sqrt(((np.asarray(got) - want.float().numpy()) ** 2).mean(1)) / float(want.std())
    assert d.max() < tol, d.max()


# ------------------------------------------------------------------ configuration, checkpoint, registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_configuration_round_trip(name):
    cfg = CONFIGS[name]
    assert from_layer_list(json.loads(json.dumps(to_layer_list(cfg)))) == cfg
    assert detect_family(cfg.tensor_shapes()) == Family.SUPISUN
    assert all(classify(n, Family.SUPISUN).role != TensorRole.UNKNOWN for n in cfg.tensor_shapes())


def test_the_first_mixing_layer_gives_the_values():
    assert CONFIGS["all"].first_value_layer == 1 and CONFIGS["mamba"].first_value_layer == -1
    d = to_layer_list(CONFIGS["all"])
    assert "l0.mix.vmix" not in CONFIGS["all"].tensor_shapes() and "l1.mix.vmix" in CONFIGS["all"].tensor_shapes()
    d["layers"][3]["mixer"]["vdim"] = 24
    with pytest.raises(ValueError, match="agree"):
        from_layer_list(d)


def test_checkpoint_directory_loads_and_damage_is_refused(tmp_path):
    cfg, w, _ = model("all")
    export_layered(cfg, RandomTensors(cfg, seed=11, gain=1.6), tmp_path / "m")
    assert architecture_of(str(tmp_path / "m")).name == "supisun"
    got = load_layered(tmp_path / "m", dtype=torch.float32)
    assert got.cfg == cfg and torch.equal(got.pos, w.pos)
    for a, b in zip(got.layers, w.layers):
        for x, y in ((a, b), (a.mixer, b.mixer)):
            for k, v in vars(y).items():
                if isinstance(v, torch.Tensor):
                    assert torch.equal(getattr(x, k), v), k
    c = json.loads((tmp_path / "m" / "config.json").read_text())
    for edit in (lambda d: d.update(width=60), lambda d: d["layers"].append(d["layers"][0]), lambda d: d.pop("canon"),
                 lambda d: d["layers"][1].update(type="channel_delta"), lambda d: d["layers"][0]["mixer"].update(kv_heads=4),
                 lambda d: d["layers"][0]["mixer"]["rot"].update(dims=26), lambda d: d["layers"][2]["mixer"].update(state=6),
                 lambda d: d["layers"][0]["mlp"].update(kind="moe"), lambda d: d.update(max_positions=701),
                 lambda d: d["layers"][0]["mixer"]["mask"].update(size=0)):
        d = json.loads(json.dumps(c))
        edit(d)
        (tmp_path / "m" / "config.json").write_text(json.dumps(d))
        with pytest.raises(CheckpointError):
            load_layered(tmp_path / "m")


def test_support_contract_knows_the_design():
    cfg = tiny_supisun()
    plan = lambda **kw: EnginePlan.from_policies(PolicySet.from_config(cfg, parallelism=ParallelismPlan(**kw)), cfg.n_heads,
                                                 cfg.n_routed_experts, cfg.n_layers, cfg.vocab_size)
    assert plan().is_executable and plan().family == "supisun" and plan().policies.expert.routed == 0
    assert set(plan().policies.kv.planes) == {"kv", "recurrent_state", "input_convolution"}
    assert not plan(tensor_parallel=2).is_executable


def test_state_planes_of_every_kind():
    cfg = CONFIGS["all"]
    p = RecurrentStatePool(cfg, 3, "cpu", torch.bfloat16, buffers=2)
    assert set(p.canon) == set(range(cfg.n_layers)) and all(t.dtype == torch.float32 and t.shape == (6, 2, 56) for t in p.canon.values())
    assert p.state[2].shape == (6, 5, 48) and p.tail[2].shape == (6, 3, 48) and p.tail[2].dtype == torch.bfloat16
    assert p.state[4].shape == (6, 4, 20, 12) and set(p.state) == {2, 4}


# ------------------------------------------------------------------ forward against the oracle
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_token_by_token_match_the_oracle(name):
    eng, oracle, cfg = engine(name)
    toks = prompt(cfg, 41, 1)
    want = oracle.logits(toks)
    same(eng.replay([ReplayEntry("w", toks, list(range(41)))], ["w"])[0], want)
    for i, t in enumerate(toks):
        same(eng.replay([ReplayEntry("d", [t], [0])], ["d"] if i == 40 else [])[0], want[i:i + 1])


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_stream_after_every_layer(name):
    cfg, w, oracle = model(name)
    eng = make_engine(cfg, w, pages=8, slots=1)

    class Tap:
        seen = []

        def write(self, layer, stage, t):
            self.seen.append(t[:, :cfg.width].clone())

        def wants(self, *_):
            return True

    eng.runner.fwd.tap = Tap()
    toks = prompt(cfg, 19, 2)
    eng.replay([ReplayEntry("a", toks, [])], ["a"])
    for got, want in zip(Tap.seen, oracle.layers(toks)):
        assert (got - want.float()).abs().max() < 3e-4
    assert len(Tap.seen) == cfg.n_layers
    Tap.seen.clear()


@pytest.mark.parametrize("sizes", [[2], [3, 2], [7], [8], [1, 9, 2, 16]])
def test_portions_of_any_size_do_not_change_the_logits(sizes):
    eng, oracle, cfg = engine("all")
    toks = prompt(cfg, 45, 3)
    want, at, k = oracle.logits(toks), 0, 0
    while at < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - at)
        k += 1
        same(eng.replay([ReplayEntry("a", toks[at:at + n], list(range(n)))])[0], want[at:at + n])
        at += n


def edge_model(chunk=12):
    """One attention layer and no convolution: a logit depends on the tokens of its own chunk and on nothing else."""
    cfg = LayeredConfig(vocab_size=50, width=32, layers=(LayerSpec(AttentionMixer(4, 2, 16, 16, 0.5, chunk, 50.0, 8), DenseSpec(24)),),
                        norm_eps=1e-5, name="supisun", max_position=200, block=OUTPUT_NORM, canon_taps=1, learned_positions=True)
    t = RandomTensors(cfg, seed=3, dtype=torch.float32, gain=1.5)
    return cfg, pack_weights(cfg, t)


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page", [4, 8])
def test_a_token_is_seen_exactly_inside_its_chunk(decoded, page):
    cfg, w = edge_model()
    toks, chunk = prompt(cfg, 40, 5), 12

    def logits(seq):
        eng = make_engine(cfg, w, page=page)
        if decoded:
            return np.concatenate([eng.replay([ReplayEntry("a", [t], [0])])[0] for t in seq])
        return eng.replay([ReplayEntry("a", seq, list(range(len(seq))))])[0]

    base = logits(toks)
    for t in (0, 3, 4, 11, 12, 13, 23, 24, 35, 36):
        seq = list(toks)
        seq[t] = (seq[t] + 7) % cfg.vocab_size
        changed = np.abs(logits(seq) - base).max(1) > 1e-3
        assert changed.tolist() == [p >= t and p // chunk == t // chunk for p in range(40)], t


def test_the_input_convolution_reaches_back_taps_minus_one_tokens():
    """Recurrence-free and attention-free reach: with chunks of one token only the convolution joins positions."""
    cfg, w = edge_model(chunk=1)
    cfg = cfg.with_(canon_taps=4)
    w = pack_weights(cfg, RandomTensors(cfg, seed=3, dtype=torch.float32, gain=1.5))
    toks = prompt(cfg, 20, 6)
    run_ = lambda seq, eng: np.concatenate([eng.replay([ReplayEntry("a", seq[i:i + n], list(range(n)))])[0]
                                            for i, n in ((0, 2), (2, 5), (7, 1), (8, 1), (9, 11))])
    base = run_(toks, make_engine(cfg, w))
    for t in (0, 1, 5, 8, 12):
        seq = list(toks)
        seq[t] = (seq[t] + 7) % cfg.vocab_size
        changed = np.abs(run_(seq, make_engine(cfg, w)) - base).max(1) > 1e-3
        assert changed.tolist() == [t <= p <= t + 3 for p in range(20)]


def test_mixed_batches_reuse_pages_and_slots():
    """Twelve requests of unequal length through four slots and a pool that is full most of the time: portions beside
    single tokens, requests left out of steps, every logit equal to the request's alone."""
    for seed in (0, 1):
        rnd = random.Random(seed)
        eng, oracle, cfg = engine("all", pages=12)
        todo = [(f"q{i}", prompt(cfg, rnd.randrange(1, 30), 100 + i)) for i in range(12)]
        live = {}
        pages = lambda n: (n + 7) // 8
        while todo or live:
            while todo and len(live) < 4 and sum(pages(len(t)) for t, _ in live.values()) + pages(len(todo[0][1])) <= 12:
                rid, t = todo.pop(0)
                live[rid] = (t, 0)
            entries, end = [], []
            for rid in list(live):
                t, at = live[rid]
                if rnd.random() < 0.25:
                    continue
                n = min(rnd.choice([1, 1, 2, 3, 9]), len(t) - at)
                entries.append(ReplayEntry(rid, t[at:at + n], list(range(n))))
                live[rid] = (t, at + n)
                if at + n == len(t):
                    end.append(rid)
            rnd.shuffle(entries)
            out = eng.replay(entries, end)
            for e, rows in zip(entries, out):
                t, at = live[e.request_id]
                same(rows, oracle.logits(t)[at - len(e.tokens):at])
            for rid in end:
                del live[rid]
        assert eng.kv.free_pages == 12 and eng.scheduler.slots.available == 4
        eng.kv.check_invariants()


# ------------------------------------------------------------------ generation through the engine
def run(eng, reqs):
    toks, fins = {}, {}

    def emit(ev):
        if isinstance(ev, TokenEvent):
            toks.setdefault(ev.request_id, []).append(ev.token)
        elif isinstance(ev, FinishEvent):
            fins[ev.request_id] = ev

    for r in reqs:
        eng.submit(r)
    eng.run_until_idle(emit)
    return toks, fins


@pytest.mark.parametrize("chunk", [3, 8, 64])
def test_greedy_generation_matches_the_oracle(chunk):
    eng, oracle, cfg = engine("all", cls=Engine)
    eng.cfg.scheduler.prefill_chunk_size = chunk
    ps = {f"r{i}": prompt(cfg, n, 50 + i) for i, n in enumerate((1, 2, 17, 9, 26, 5))}
    toks, fins = run(eng, [GenerateRequest(r, p, max_new_tokens=6, ignore_eos=True) for r, p in ps.items()])
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 6)
        assert fins[r].reason == FinishReason.MAX_TOKENS
    assert eng.kv.free_pages == 24


def test_an_aborted_step_leaves_the_committed_state_untouched():
    eng, oracle, cfg = engine("all", cls=Engine)
    p = prompt(cfg, 11, 7)
    fwd, calls = eng.runner.fwd, [0]
    real = fwd.logits_from_hidden

    class Retry(RuntimeError):
        retryable = True

    def flaky(x, b):
        calls[0] += 1
        if calls[0] in (1, 3, 4):                       # the step has written its state and cache rows by now
            raise Retry("scripted")
        return real(x, b)

    fwd.logits_from_hidden = flaky
    toks, _ = run(eng, [GenerateRequest("a", p, max_new_tokens=5, ignore_eos=True)])
    assert toks["a"] == oracle.greedy(p, 5) and eng.stats.aborted_transactions == 3


def test_sessions_continue_from_their_slot():
    eng, oracle, cfg = engine("all", cls=Engine)
    a, b = prompt(cfg, 9, 8), prompt(cfg, 4, 9)
    toks, _ = run(eng, [GenerateRequest("t0", a, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    history = a + toks["t0"]
    other, _ = run(eng, [GenerateRequest("x", b, max_new_tokens=2, ignore_eos=True)])
    assert other["x"] == oracle.greedy(b, 2)
    more, _ = run(eng, [GenerateRequest("t1", b, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    assert more["t1"] == oracle.greedy(history + b, 3)
    assert eng.reset_session("s") and eng.scheduler.slots.available == 4 and eng.kv.free_pages == 24


def test_swapped_out_sequences_come_back():
    eng, oracle, cfg = engine("all", cls=Engine, pages=7)
    eng.cfg.auto_preempt = True
    ps = {f"r{i}": prompt(cfg, 14, 70 + i) for i in range(3)}
    toks, _ = run(eng, [GenerateRequest(r, p, max_new_tokens=30, ignore_eos=True) for r, p in ps.items()])
    assert eng.stats.auto_preemptions > 0
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 30), r


@pytest.mark.parametrize("name", ["mamba", "delta"])
def test_long_decoding_keeps_the_state(name):
    eng, oracle, cfg = engine(name, pages=40, cls=Engine)
    p = prompt(cfg, 5, 21)
    toks, _ = run(eng, [GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True)])
    seq = p + toks["a"]
    assert seq[5:] == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]


def test_a_sequence_ends_at_the_last_learned_position():
    cfg, w = edge_model()
    cfg = cfg.with_(max_position=21)
    w = pack_weights(cfg, RandomTensors(cfg, seed=3, dtype=torch.float32))
    eng = make_engine(cfg, w)
    eng.replay([ReplayEntry("a", prompt(cfg, 21, 1), [20])], ["a"])
    with pytest.raises(Exception, match="exceeds"):
        eng.replay([ReplayEntry("b", prompt(cfg, 22, 1), [])])


# ------------------------------------------------------------------ oracle self-checks
def test_oracle_recurrences_carry_their_state():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.rand(*s, generator=g, dtype=torch.float64)
    q, k, v, d, b = r(9, 2, 5), r(9, 2, 5), r(9, 2, 3), r(9, 2), r(9, 2)
    o, S = SO.delta_recurrence(q, k, v, d, b)
    o1, s1 = SO.delta_recurrence(q[:4], k[:4], v[:4], d[:4], b[:4])
    o2, s2 = SO.delta_recurrence(q[4:], k[4:], v[4:], d[4:], b[4:], s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, S)
    x, dt, A, B, C, D = r(9, 6), r(9, 6), -r(6, 4), r(9, 4), r(9, 4), r(6)
    y, S = SO.selective_scan(x, dt, A, B, C, D)
    y1, s1 = SO.selective_scan(x[:5], dt[:5], A, B[:5], C[:5], D)
    y2, s2 = SO.selective_scan(x[5:], dt[5:], A, B[5:], C[5:], D, s1)
    assert torch.allclose(torch.cat([y1, y2]), y) and torch.allclose(s2, S)


# ------------------------------------------------------------------ the programs
def test_trace_runner_program(tmp_path):
    cfg, _, oracle = model("all")
    export_layered(cfg, RandomTensors(cfg, seed=11, gain=1.6), tmp_path / "m")
    (tmp_path / "out").mkdir()
    a, b = prompt(cfg, 12, 31), prompt(cfg, 5, 32)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [6, 0]}, {"id": "b", "tokens": b, "want": []}], "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": a[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [4]}, {"id": "a", "tokens": a[8:], "want": [3]}], "end": ["a", "c"]}]
    exe = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    r = subprocess.run([sys.executable, str(exe), "--model", str(tmp_path / "m"), "--dtype", "float32", "--device", "cpu", "--out",
                        str(tmp_path / "out"), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda i: np.fromfile(tmp_path / "out" / f"{i}.f32", "<f4").reshape(-1, cfg.vocab_size)
    same(read(0), oracle.logits(a)[[6, 0]])
    same(read(2), torch.stack([oracle.logits(b)[4], oracle.logits(a)[11]]))
    assert not (tmp_path / "out" / "1.f32").exists()


def test_command_line_makes_inspects_and_runs_a_checkpoint(tmp_path):
    def cli(*args):
        r = subprocess.run([sys.executable, "-m", "ferrule_b200", *args], capture_output=True, text=True, timeout=300,
                           cwd=Path(__file__).resolve().parent.parent)
        assert r.returncode == 0, r.stderr
        return r.stdout

    d = str(tmp_path / "fx")
    assert json.loads(cli("make-fixture", "--family", "supisun", "--out", d))["family"] == "supisun"
    assert '"supisun"' in cli("info", d)
    out = json.loads(cli("generate", "--model-dir", d, "--device", "cpu", "--tokens", "5,6,7", "-n", "4", "--ignore-eos", "--json"))
    cfg = tiny_supisun()
    assert out["tokens"] == SO.Oracle(cfg, RandomTensors(cfg, 0)).greedy([5, 6, 7], 4)
