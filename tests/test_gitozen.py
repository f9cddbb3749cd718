"""Gitozen on the CPU path: configuration and checkpoint handling, the reference forward against an independent oracle,
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
from ferrule_b200.models.layered_config import from_layer_list, tiny_gitozen, to_layer_list
from ferrule_b200.models.layered_runner import LayeredRunner
from ferrule_b200.models.layered_weights import RandomTensors, pack_weights
from ferrule_b200.models.registry import architecture_of
from ferrule_b200.models.state_pool import RecurrentStatePool
from ferrule_b200.models.support import EnginePlan, ParallelismPlan, PolicySet
from ferrule_b200.runtime.engine import Engine, EngineConfig, FinishEvent, TokenEvent
from ferrule_b200.runtime.replay import ReplayEngine, ReplayEntry, ReplayError
from ferrule_b200.runtime.scheduler import SchedulerConfig
from ferrule_b200.runtime.session import FinishReason, GenerateRequest

sys.path.insert(0, str(Path(__file__).parent))
from gitozen_configs import CONFIGS  # noqa: E402
from gitozen_oracle import Oracle, delta_recurrence  # noqa: E402

_memo = {}


def model(name, gain=1.6):
    if (name, gain) not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=torch.float32, gain=gain)
        _memo[name, gain] = (cfg, pack_weights(cfg, t), Oracle(cfg, t))
    return _memo[name, gain]


def replay_engine(name, pages=24, page=8, slots=4, cls=ReplayEngine, **kw):
    cfg, w, oracle = model(name)
    n = pages * page
    runner = LayeredRunner(w, n_pages=pages, page_size=page, max_rows=n, max_seqs=slots, max_seq_len=n + page)
    sched = SchedulerConfig(max_active_sequences=slots, max_decode_batch=slots, max_batch_tokens=n, prefill_chunk_size=n,
                            ctx_size=n + page, **kw)
    return cls(runner, EngineConfig(scheduler=sched, kv_pages=pages, page_size=page)), oracle, cfg


def prompt(cfg, n, seed):
    r = random.Random(seed)
    return [r.randrange(cfg.vocab_size) for _ in range(n)]


def same(got, want, tol=3e-5):
    d = np.abs(np.asarray(got) - want.float().numpy()).max() / float(want.std())
    assert d < tol, d


# ------------------------------------------------------------------ configuration, checkpoint, registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_configuration_round_trip(name):
    cfg = CONFIGS[name]
    back = from_layer_list(json.loads(json.dumps(to_layer_list(cfg))))
    for a, b in zip(cfg.layers, back.layers):
        assert a.mlp == b.mlp and a.mixer.heads == b.mixer.heads and a.mixer.dim == b.mixer.dim
    assert (back.width, back.vocab_size, back.norm_eps, back.logit_softcap) == (cfg.width, cfg.vocab_size, cfg.norm_eps,
                                                                                cfg.logit_softcap)
    assert detect_family(cfg.tensor_shapes()) == Family.GITOZEN
    assert all(classify(n, Family.GITOZEN).role != TensorRole.UNKNOWN for n in cfg.tensor_shapes())


def test_checkpoint_directory_loads_and_damage_is_refused(tmp_path):
    cfg, w, _ = model("both")
    t = RandomTensors(cfg, seed=11, gain=1.6)
    export_layered(cfg, t, tmp_path / "m")
    assert architecture_of(str(tmp_path / "m")).name == "gitozen"
    got = load_layered(tmp_path / "m", dtype=torch.float32)
    assert got.cfg.layers[0].mixer.decay_rank == cfg.layers[0].mixer.decay_rank
    for a, b in zip(got.layers, w.layers):
        for k, v in vars(b.mixer).items():
            if isinstance(v, torch.Tensor):
                assert torch.equal(getattr(a.mixer, k), v), k
        assert (a.e_w13 is None) == (b.e_w13 is None) and (a.e_w13 is None or torch.equal(a.e_w13, b.e_w13))
    c = json.loads((tmp_path / "m" / "config.json").read_text())
    for edit in (lambda d: d.update(width=60), lambda d: d["layers"].append(d["layers"][0]), lambda d: d.pop("norm"),
                 lambda d: d["layers"][1].update(type="window"), lambda d: d["layers"][0]["mixer"].update(kv_heads=3),
                 lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4)):
        d = json.loads(json.dumps(c))
        edit(d)
        (tmp_path / "m" / "config.json").write_text(json.dumps(d))
        with pytest.raises(CheckpointError):
            load_layered(tmp_path / "m")
    (tmp_path / "m" / "config.json").write_text(json.dumps({**c, "architecture": "Other"}))
    with pytest.raises(CheckpointError, match="unknown architecture"):
        architecture_of(str(tmp_path / "m"))


def test_support_contract_knows_the_design():
    cfg = tiny_gitozen()
    plan = lambda **kw: EnginePlan.from_policies(PolicySet.from_config(cfg, parallelism=ParallelismPlan(**kw)), cfg.n_heads,
                                                 cfg.n_routed_experts, cfg.n_layers, cfg.vocab_size)
    assert plan().is_executable and plan().family == "gitozen"
    assert not plan(tensor_parallel=2).is_executable


# ------------------------------------------------------------------ state pool
def test_state_pool_buffers_commit_roll_back_and_run_ahead():
    p = RecurrentStatePool(CONFIGS["delta"], 3, "cpu", torch.float32, buffers=3)
    assert p.bind(1, True) == (-1, 3) and p.bind(1, True) == (-1, 3)       # nothing committed: a retry binds alike
    with pytest.raises(RuntimeError):
        p.bind(1, False)
    p.commit(1, 3)
    assert p.bind(1, False) == (3, 4)
    assert p.bind(1, False, ahead=True) == (4, 5)
    assert p.bind(1, False) == (3, 4)                                      # the unpublished step can still be redone
    p.commit(1, 4)
    assert p.bind(1, False) == (4, 5)                                      # what ran ahead bound the same pair
    p.commit(1, 5)
    assert p.bind(1, False) == (5, 3)
    with pytest.raises(ValueError):
        p.commit(0, 5)
    p.release(1)
    assert p.bind(1, True) == (-1, 3)
    # a first step that is a decode step: the step after it is bound before it is published
    assert p.bind(2, True) == (-1, 6) and p.bind(2, False, ahead=True) == (6, 7)


# ------------------------------------------------------------------ forward against the oracle
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_token_by_token_match_the_oracle(name):
    eng, oracle, cfg = replay_engine(name)
    toks = prompt(cfg, 41, 1)
    want = oracle.logits(toks)
    same(eng.replay([ReplayEntry("w", toks, list(range(41)))], ["w"])[0], want)
    for i, t in enumerate(toks):
        row = eng.replay([ReplayEntry("d", [t], [0])], ["d"] if i == 40 else [])[0]
        same(row, want[i:i + 1])


@pytest.mark.parametrize("name", list(CONFIGS))
def test_residual_stream_after_every_layer(name):
    cfg, w, oracle = model(name)
    runner = LayeredRunner(w, n_pages=8, page_size=8, max_rows=32, max_seqs=1, max_seq_len=64)

    class Tap:
        seen = []

        def write(self, layer, stage, t):
            self.seen.append(t[:, :cfg.width].clone())

        def wants(self, *_):
            return True

    runner.fwd.tap = Tap()
    eng = ReplayEngine(runner, EngineConfig(scheduler=SchedulerConfig(1, 1, 32, 32, ctx_size=64), kv_pages=8, page_size=8))
    toks = prompt(cfg, 19, 2)
    eng.replay([ReplayEntry("a", toks, [])], ["a"])
    for got, want in zip(Tap.seen, oracle.layers(toks)):
        assert (got - want.float()).abs().max() < 2e-4
    assert len(Tap.seen) == cfg.n_layers
    Tap.seen.clear()


@pytest.mark.parametrize("sizes", [[2], [3, 2], [7], [8], [1, 9, 2, 16]])
def test_portions_of_any_size_do_not_change_the_logits(sizes):
    eng, oracle, cfg = replay_engine("both")
    toks = prompt(cfg, 45, 3)
    want, at, k = oracle.logits(toks), 0, 0
    while at < len(toks):
        n = min(sizes[k % len(sizes)], len(toks) - at)
        k += 1
        out = eng.replay([ReplayEntry("a", toks[at:at + n], list(range(n)))])[0]
        same(out, want[at:at + n])
        at += n


def test_mixed_batches_reuse_pages_and_slots():
    """Twelve requests of unequal length through four slots and a pool that is full most of the time: portions beside
    single tokens, requests left out of steps, every logit equal to the request's alone."""
    for seed in (0, 1):
        rnd = random.Random(seed)
        eng, oracle, cfg = replay_engine("both", pages=12)
        todo = [(f"q{i}", prompt(cfg, rnd.randrange(1, 30), 100 + i)) for i in range(12)]
        live, used = {}, set()
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
                used.add(eng._live[e.request_id].slot if e.request_id in eng._live else -1)
                same(rows, oracle.logits(t)[at - len(e.tokens):at])
            for rid in end:
                del live[rid]
        assert eng.kv.free_pages == 12 and eng.scheduler.slots.available == 4
        eng.kv.check_invariants()


def test_replay_refuses_what_cannot_run():
    eng, _, cfg = replay_engine("both", pages=2, slots=1)
    eng.replay([ReplayEntry("a", [1, 2], [])])
    with pytest.raises(ReplayError, match="slot"):
        eng.replay([ReplayEntry("b", [1], [])])
    eng, _, cfg = replay_engine("both", pages=2, slots=2)
    with pytest.raises(ReplayError, match="lie outside"):
        eng.replay([ReplayEntry("a", [1, 2], [2])])
    eng.replay([ReplayEntry("a", list(range(9)), [])])
    with pytest.raises(ReplayError, match="pool cannot hold"):
        eng.replay([ReplayEntry("a", list(range(9)), [])])


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
    eng, oracle, cfg = replay_engine("both", cls=Engine)
    eng.cfg.scheduler.prefill_chunk_size = chunk
    ps = {f"r{i}": prompt(cfg, n, 50 + i) for i, n in enumerate((1, 2, 17, 9, 26, 5))}
    toks, fins = run(eng, [GenerateRequest(r, p, max_new_tokens=6, ignore_eos=True) for r, p in ps.items()])
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 6)
        assert fins[r].reason == FinishReason.MAX_TOKENS
    assert eng.kv.free_pages == 24


def test_an_aborted_step_leaves_the_committed_state_untouched():
    eng, oracle, cfg = replay_engine("both", cls=Engine)
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
    toks, fins = run(eng, [GenerateRequest("a", p, max_new_tokens=5, ignore_eos=True)])
    assert toks["a"] == oracle.greedy(p, 5) and eng.stats.aborted_transactions == 3


def test_sessions_continue_from_their_slot_and_forks_are_refused():
    eng, oracle, cfg = replay_engine("both", cls=Engine)
    a, b = prompt(cfg, 9, 8), prompt(cfg, 4, 9)
    toks, _ = run(eng, [GenerateRequest("t0", a, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    history = a + toks["t0"]
    other, _ = run(eng, [GenerateRequest("x", b, max_new_tokens=2, ignore_eos=True)])
    assert other["x"] == oracle.greedy(b, 2)
    more, _ = run(eng, [GenerateRequest("t1", b, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    assert more["t1"] == oracle.greedy(history + b, 3)
    with pytest.raises(ValueError, match="slot"):
        eng.fork_session_exact("s", GenerateRequest("f", [1]))
    assert eng.reset_session("s") and eng.scheduler.slots.available == 4 and eng.kv.free_pages == 24


def test_swapped_out_sequences_come_back():
    eng, oracle, cfg = replay_engine("both", cls=Engine, pages=7)
    eng.cfg.auto_preempt = True
    ps = {f"r{i}": prompt(cfg, 14, 70 + i) for i in range(3)}
    toks, fins = run(eng, [GenerateRequest(r, p, max_new_tokens=30, ignore_eos=True) for r, p in ps.items()])
    assert eng.stats.auto_preemptions > 0
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 30), r


def test_long_decoding_keeps_the_state():
    eng, oracle, cfg = replay_engine("delta", pages=40, cls=Engine)
    p = prompt(cfg, 5, 21)
    toks, _ = run(eng, [GenerateRequest("a", p, max_new_tokens=200, ignore_eos=True)])
    seq = p + toks["a"]
    assert seq[5:] == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]


# ------------------------------------------------------------------ oracle self-checks
def test_oracle_recurrence_carries_its_state():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.rand(*s, generator=g, dtype=torch.float64)
    q, k, v, d, b = r(9, 2, 5), r(9, 2, 5), r(9, 2, 3), r(9, 2, 5), r(9, 2)
    o, S = delta_recurrence(q, k, v, d, b)
    o1, s1 = delta_recurrence(q[:4], k[:4], v[:4], d[:4], b[:4])
    o2, s2 = delta_recurrence(q[4:], k[4:], v[4:], d[4:], b[4:], s1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(s2, S)


# ------------------------------------------------------------------ the trace runner program
def test_trace_runner_program(tmp_path):
    cfg, _, oracle = model("both")
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
