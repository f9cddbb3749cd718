"""Vedadra on the CPU path: configuration and checkpoint handling, the reference forward against an independent oracle,
looped layers, windows and kept tokens, page bookkeeping, generation through the engine, replay of token streams and the
trace runner program."""
import json
import math
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
from ferrule_b200.models.layered_config import (SANDWICH_NORM, DeltaMixer, DenseSpec, LayeredConfig, LayerSpec, Loop,
                                                from_layer_list, preset_architecture, tiny_vedadra, to_layer_list)
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
import vedadra_oracle as VO  # noqa: E402
from vedadra_configs import CONFIGS, differential, talking  # noqa: E402

_memo = {}


def model(name, gain=1.6):
    if (name, gain) not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=torch.float32, gain=gain)
        _memo[name, gain] = (cfg, pack_weights(cfg, t), VO.Oracle(cfg, t))
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
    """Root mean square over a row's logits."""
    d = np.sqrt(((np.asarray(got) - want.float().numpy()) ** 2).mean(1)) / float(want.std())
    assert d.max() < tol, d.max()


# ------------------------------------------------------------------ configuration, checkpoint, registry
@pytest.mark.parametrize("name", list(CONFIGS))
def test_configuration_round_trip(name):
    cfg = CONFIGS[name]
    assert from_layer_list(json.loads(json.dumps(to_layer_list(cfg)))) == cfg
    assert detect_family(cfg.tensor_shapes()) == Family.VEDADRA
    assert all(classify(n, Family.VEDADRA).role != TensorRole.UNKNOWN for n in cfg.tensor_shapes())


def test_runs_of_looped_layers():
    cfg = CONFIGS["all"]
    assert cfg.runs == (0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4) and cfg.pass_starts == (4, 7)
    assert cfg.cache_runs == tuple(range(11))
    assert [i for i, _ in VO.run_order(5, cfg.loop)] == list(cfg.runs)
    assert [r for r, (_, again) in enumerate(VO.run_order(5, cfg.loop)) if again] == list(cfg.pass_starts)
    assert CONFIGS["once"].runs == (0, 1) and CONFIGS["once"].pass_starts == ()
    assert CONFIGS["differential"].runs == (0, 1) and CONFIGS["talking"].pass_starts == (2,)
    cut = cfg.first_layers(3)
    assert cut.runs == (0, 1, 2, 1, 2, 1, 2) and cfg.first_layers(1).loop is None
    assert cfg.cycled(7).runs == (0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4, 5, 6)


def test_a_recurrent_layer_has_a_state_per_run():
    cfg = LayeredConfig(64, 32, (LayerSpec(DeltaMixer(2, 1, 8, 8, 3), None), LayerSpec(talking(2, 1, 8, 0.5, 4), None)),
                        block=SANDWICH_NORM, loop=Loop(0, 2, 2))
    p = RecurrentStatePool(cfg, 3, "cpu", torch.bfloat16, buffers=2)
    assert set(p.state) == {0, 2} and cfg.cache_runs == (1, 3)


def test_configuration_errors():
    good = to_layer_list(CONFIGS["all"])
    for edit, text in ((lambda d: d["loop"].update(stop=6), "loop"), (lambda d: d["loop"].update(start=4), "loop"),
                       (lambda d: d["loop"].update(times=0), "loop"), (lambda d: d["norm"].update(groups=7), "groups"),
                       (lambda d: d["layers"][0]["mixer"].update(vdim=24), "width"),
                       (lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
                       (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "window"),
                       (lambda d: d["layers"][1]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
                       (lambda d: d["layers"][1].update(type="delta"), "mixer type"),
                       (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "feed-forward")):
        d = json.loads(json.dumps(good))
        edit(d)
        with pytest.raises(ValueError, match=text):
            from_layer_list(d)
    d = json.loads(json.dumps(good))
    d["loop"], d["norm"] = None, {"eps": 1e-5}
    assert from_layer_list(d).runs == (0, 1, 2, 3, 4) and from_layer_list(d).norm_groups == 1
    gitozen = {"architecture": "Gitozen", "vocab": 8, "width": 8, "norm": {"eps": 1e-5}, "loop": {"start": 0, "stop": 1, "times": 2},
               "layers": [{"type": "latent_attention", "mixer": {"heads": 1, "dim": 8, "vdim": 8, "kv_rank": 8, "scale": 1.0}}]}
    with pytest.raises(ValueError, match="loop"):
        from_layer_list(gitozen)


def test_checkpoint_directory_loads_and_damage_is_refused(tmp_path):
    cfg, w, _ = model("all")
    export_layered(cfg, RandomTensors(cfg, seed=11, gain=1.6), tmp_path / "m")
    assert architecture_of(str(tmp_path / "m")).name == "vedadra"
    got = load_layered(tmp_path / "m", dtype=torch.float32)
    assert got.cfg == cfg
    for a, b in zip(got.layers, w.layers):
        for x, y in ((a, b), (a.mixer, b.mixer)):
            for k, v in vars(y).items():
                if k != "mixer":
                    assert torch.equal(getattr(x, k), v) if isinstance(v, torch.Tensor) else getattr(x, k) == v, k
    assert load_layered(tmp_path / "m", max_layers=2).cfg.runs == (0, 1, 1, 1)
    c = json.loads((tmp_path / "m" / "config.json").read_text())
    for edit in (lambda d: d.update(width=63), lambda d: d["layers"].append(d["layers"][0]), lambda d: d.pop("norm"),
                 lambda d: d["layers"][1]["mixer"].update(heads=2), lambda d: d["layers"][0]["mlp"].update(ff=73),
                 lambda d: d["layers"][0]["mixer"].pop("mask")):
        d = json.loads(json.dumps(c))
        edit(d)
        (tmp_path / "m" / "config.json").write_text(json.dumps(d))
        with pytest.raises(CheckpointError):
            load_layered(tmp_path / "m")


def test_support_contract_knows_the_design():
    cfg = tiny_vedadra()
    plan = lambda **kw: EnginePlan.from_policies(PolicySet.from_config(cfg, parallelism=ParallelismPlan(**kw)), cfg.n_heads,
                                                 cfg.n_routed_experts, cfg.n_layers, cfg.vocab_size)
    assert plan().is_executable and plan().family == "vedadra" and plan().policies.kv.planes == ("kv",)
    assert not plan(tensor_parallel=2).is_executable
    assert preset_architecture("tiny-vedadra") == "vedadra" and preset_architecture("supisun-attention-lite") == "supisun"


def test_constants_of_a_layer_are_folded_exactly():
    cfg, w, oracle = model("all")
    T, m, img = oracle.T, cfg.layers[0].mixer, w.layers[0].mixer
    p = "l0.mix."
    assert torch.allclose(img.q_mix.double(), T(p + "talk") * T(p + "temp") * m.scale)
    slopes = torch.tensor([VO.slope(h, m.heads) for h in range(m.heads)], dtype=torch.float64)
    assert torch.allclose(img.slopes.double(), T(p + "talk") @ slopes)
    d = w.layers[1].mixer
    assert math.isclose(d.diff_lambda, float(VO.map_weight(T, "l1.mix.", cfg.layers[1].mixer.diff)), rel_tol=1e-6)
    assert cfg.layers[1].mixer.key_width == 2 * 16 and m.key_width == 3 * 24 and w.layers[1].w_up is None


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
def test_residual_stream_after_every_run(name):
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
    assert len(Tap.seen) == len(cfg.runs)
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


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page,mixer", [(4, talking(4, 2, 16, 0.5, 12)), (8, talking(2, 1, 16, 0.5, 9, 3)), (8, differential(2, 1, 16, 16, 0.5, 10, 4, 0.5)),
                                        (4, differential(4, 2, 16, 24, 0.5, 1, 1, 0.3))],
                         ids=lambda x: f"{x.kind}w{x.window}k{x.keep_first}" if hasattr(x, "maps") else str(x))
def test_a_token_is_seen_exactly_in_windows_and_among_the_kept(decoded, page, mixer):
    """One layer whose scores are nearly equal: a changed token changes the rows that see it, and no others."""
    cfg = LayeredConfig(50, 32, (LayerSpec(mixer, DenseSpec(24, True)),), 1e-5, name="vedadra", block=SANDWICH_NORM, norm_groups=2)
    t = RandomTensors(cfg, seed=3, dtype=torch.float32, gain=1.5)
    flat = lambda n: t(n) * 0.05 if n.endswith((".mix.q", ".k.norm")) else torch.full_like(t(n), 0.01) if n.endswith("talk") else t(n)
    w = pack_weights(cfg, flat)
    toks = prompt(cfg, 40, 5)

    def logits(seq):
        eng = make_engine(cfg, w, page=page)
        if decoded:
            return np.concatenate([eng.replay([ReplayEntry("a", [t], [0])])[0] for t in seq])
        return eng.replay([ReplayEntry("a", seq, list(range(len(seq))))])[0]

    base = logits(toks)
    for t0 in (0, 1, 2, 3, 4, 7, 8, 12, 20, 30):
        seq = list(toks)
        seq[t0] = (seq[t0] + 7) % cfg.vocab_size
        changed = np.abs(logits(seq) - base).max(1) > 1e-5
        assert changed.tolist() == [p >= t0 and (p - t0 < mixer.window or t0 < mixer.keep_first) for p in range(40)], t0


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


def test_sessions_and_swapped_out_sequences():
    eng, oracle, cfg = engine("talking", cls=Engine)
    a, b = prompt(cfg, 9, 8), prompt(cfg, 4, 9)
    toks, _ = run(eng, [GenerateRequest("t0", a, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    more, _ = run(eng, [GenerateRequest("t1", b, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    assert more["t1"] == oracle.greedy(a + toks["t0"] + b, 3)
    eng, oracle, cfg = engine("talking", cls=Engine, pages=7)
    eng.cfg.auto_preempt = True
    ps = {f"r{i}": prompt(cfg, 14, 70 + i) for i in range(3)}
    toks, _ = run(eng, [GenerateRequest(r, p, max_new_tokens=30, ignore_eos=True) for r, p in ps.items()])
    assert eng.stats.auto_preemptions > 0
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 30), r


def test_long_decoding_slides_every_window():
    eng, oracle, cfg = engine("differential", pages=40, cls=Engine)
    p = prompt(cfg, 5, 21)
    toks, _ = run(eng, [GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True)])
    seq = p + toks["a"]
    assert seq[5:] == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]


# ------------------------------------------------------------------ oracle self-checks
def test_oracle_mechanisms():
    x = torch.arange(1.0, 9.0, dtype=torch.float64)[None]
    n = VO.group_rms(x, torch.ones(8, dtype=torch.float64), 2, 0.0)
    assert torch.allclose((n * n).view(2, 4).mean(1), torch.ones(2, dtype=torch.float64))
    assert VO.window(5, 2, 1).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [1, 0, 1, 1, 0], [1, 0, 0, 1, 1]]
    s = torch.rand(3, 4, 4, dtype=torch.float64)
    assert torch.equal(VO.mix_scores(s, torch.eye(3, dtype=torch.float64)), s)
    assert [VO.slope(h, 8) for h in (0, 7)] == [0.5, 1 / 256]
    z = torch.linspace(-4, 4, 33, dtype=torch.float64)
    assert torch.allclose(VO.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    # equal maps: the difference is (1 - weight) a, normalised and scaled
    a = torch.rand(2, 6, dtype=torch.float64)
    assert torch.allclose(VO.map_difference(a, a, 0.25, 0.4, 0.0), VO.rms(a, 0.0) * 0.6)


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
    assert json.loads(cli("make-fixture", "--family", "vedadra", "--out", d))["family"] == "vedadra"
    assert '"vedadra"' in cli("info", d)
    out = json.loads(cli("generate", "--model-dir", d, "--device", "cpu", "--tokens", "5,6,7", "-n", "4", "--ignore-eos", "--json"))
    cfg = tiny_vedadra()
    assert out["tokens"] == VO.Oracle(cfg, RandomTensors(cfg, 0)).greedy([5, 6, 7], 4)
