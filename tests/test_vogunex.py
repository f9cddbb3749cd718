"""Vogunex on the CPU path: configuration and checkpoint handling, the reference forward against an independent oracle, token
shift, windows and pooled blocks, shared weights, state and page bookkeeping, generation through the engine, replay of token
streams and the trace runner program."""
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
from ferrule_b200.models.layered_config import from_layer_list, preset_architecture, tiny_vogunex, to_layer_list
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
import vogunex_oracle as VO  # noqa: E402
from vogunex_configs import CONFIGS, FF, latent, pooled, vogunex  # noqa: E402

_memo = {}


def model(name, gain=1.6):
    if (name, gain) not in _memo:
        cfg = CONFIGS[name]
        t = RandomTensors(cfg, seed=11, dtype=torch.float32, gain=gain)
        _memo[name, gain] = (cfg, pack_weights(cfg, t), VO.Oracle(to_layer_list(cfg), t))
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
    assert detect_family(cfg.tensor_shapes()) == Family.VOGUNEX
    assert all(classify(n, Family.VOGUNEX).role != TensorRole.UNKNOWN for n in cfg.tensor_shapes())


def test_shared_weights():
    cfg, w, _ = model("all")
    assert [cfg.owner(i) for i in range(7)] == [0, 1, 0, 3, 4, 3, 6]
    assert w.layers[2] is w.layers[0] and w.layers[5] is w.layers[3] and w.layers[6] is not w.layers[1]
    assert not any(n.startswith(("l2.", "l5.")) for n in cfg.tensor_shapes())
    assert cfg.cache_runs == (0, 1, 2, 4, 6)                       # a cache plane and a state of its own for every layer
    pool = RecurrentStatePool(cfg, 2, "cpu", max_tokens=50)
    assert set(pool.state) == {3, 5} and set(pool.shift) == set(range(7)) and set(pool.pooled) == {0, 2, 4}
    assert pool.pooled[0].shape == (2, 13, cfg.plane_dim(0)) and pool.pooled[4].shape == (2, 8, cfg.plane_dim(4))
    d = to_layer_list(cfg)
    d["layers"][5]["weights_of"] = 5
    with pytest.raises(ValueError, match="weights"):
        from_layer_list(d)
    d["layers"][5]["weights_of"] = 1
    with pytest.raises(ValueError, match="sizes differ"):
        from_layer_list(d)
    # a layer that names one which itself names another: the tensors are the last one's
    d = to_layer_list(cfg)
    d["layers"].append({**d["layers"][2], "weights_of": 2})
    assert from_layer_list(d).owner(7) == 0
    assert VO.owner(d["layers"], 7) == 0
    assert cfg.first_layers(4).owner(2) == 0 and cfg.cycled(10).owner(9) == 0 and cfg.cycled(10).owner(7) == 7


def test_configuration_errors():
    good = to_layer_list(CONFIGS["all"])
    for edit, text in ((lambda d: d["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"),
                       (lambda d: d["layers"][0]["mixer"]["mask"].update(size=0), "window"),
                       (lambda d: d["layers"][0]["mixer"]["mask"].update(pool=0), "pool"),
                       (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=22), "rot.dims"),
                       (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "rot.dims"),
                       (lambda d: d["layers"][1]["mixer"].update(rot_dim=5), "rot_dim"),
                       (lambda d: d["layers"][1]["mixer"].update(q_rank=0), "q_rank"),
                       (lambda d: d["layers"][3]["mixer"].update(groups=3), "groups"),
                       (lambda d: d["layers"][3]["mixer"].update(norm_groups=5), "norm_groups"),
                       (lambda d: d["layers"][1]["mlp"]["router"].update(top=6), "router"),
                       (lambda d: d["layers"][1]["mlp"].update(kind="gated"), "feed-forward"),
                       (lambda d: d["layers"][4].update(type="delta"), "mixer type")):
        d = json.loads(json.dumps(good))
        d["layers"] = [{k: v for k, v in l.items() if k != "weights_of"} for l in d["layers"]]
        edit(d)
        with pytest.raises(ValueError, match=text):
            from_layer_list(d)
    supisun = {"architecture": "Supisun", "vocab": 8, "width": 8, "norm": {"eps": 1e-5}, "max_positions": 8, "canon": {"taps": 1},
               "layers": [{"type": "mamba1", "mixer": {"inner": 8, "state": 2, "dt_rank": 1, "conv": 2}, "mlp": None}] * 2}
    supisun["layers"][1] = {**supisun["layers"][1], "weights_of": 0}
    with pytest.raises(ValueError, match="weights of their own"):
        from_layer_list(supisun)


def test_checkpoint_directory_loads_and_damage_is_refused(tmp_path):
    cfg, w, _ = model("all")
    export_layered(cfg, RandomTensors(cfg, seed=11, gain=1.6), tmp_path / "m")
    assert architecture_of(str(tmp_path / "m")).name == "vogunex"
    got = load_layered(tmp_path / "m", dtype=torch.float32)
    assert got.cfg == cfg
    for a, b in zip(got.layers, w.layers):
        for x, y in ((a, b), (a.mixer, b.mixer)):
            for k, v in vars(y).items():
                if k != "mixer":
                    assert torch.equal(getattr(x, k), v) if isinstance(v, torch.Tensor) else getattr(x, k) == v, k
    assert load_layered(tmp_path / "m", max_layers=3).cfg.n_layers == 3
    c = json.loads((tmp_path / "m" / "config.json").read_text())
    for edit in (lambda d: d.update(width=63), lambda d: d["layers"].append(d["layers"][0]), lambda d: d.pop("norm"),
                 lambda d: d["layers"][1]["mixer"].update(heads=2), lambda d: d["layers"][6]["mlp"].update(ff=73),
                 lambda d: d["layers"][1]["mlp"]["shared"].update(ff=39), lambda d: d["layers"][2].pop("weights_of"),
                 lambda d: d["layers"][0]["mixer"].pop("mask")):
        d = json.loads(json.dumps(c))
        edit(d)
        (tmp_path / "m" / "config.json").write_text(json.dumps(d))
        with pytest.raises(CheckpointError):
            load_layered(tmp_path / "m")


def test_support_contract_knows_the_design():
    cfg = tiny_vogunex()
    plan = lambda **kw: EnginePlan.from_policies(PolicySet.from_config(cfg, parallelism=ParallelismPlan(**kw)), cfg.n_heads,
                                                 cfg.n_routed_experts, cfg.n_layers, cfg.vocab_size)
    assert plan().is_executable and plan().family == "vogunex"
    assert set(plan().policies.kv.planes) == {"latent_kv", "kv", "recurrent_state", "pooled_kv", "token_shift"}
    assert plan().policies.expert.shared == 1 and not plan(tensor_parallel=2).is_executable
    assert preset_architecture("tiny-vogunex") == "vogunex" and preset_architecture("vogunex-moe-lite") == "vogunex"


def test_planes_are_as_wide_as_their_rows():
    cfg, w, _ = model("all")
    assert [cfg.plane_dim(i) for i in (0, 1, 2, 4, 6)] == [120, 64, 120, 120, 64]      # the wider attention row serves both
    assert latent(2, 16, 8, 500, 16, 40, 9).row_dim == 576 and latent(2, 16, 8, 500, 16, 40, 9).rot_offset == 512
    assert latent(2, 16, 8, 440, 16, 72, 9).row_dim == 512 and latent(2, 16, 8, 600, 16, 72, 9).row_dim == 704
    eng = make_engine(cfg, w)
    assert [eng.runner.pool.layer(i).shape[-1] for i in range(5)] == [120, 64, 120, 120, 64]
    schema = eng.runner.kv_schema()
    assert {(p.name, p.elements_per_token, p.layer_count) for p in schema.planes} == {("latent_kv", 64, 2), ("kv", 120, 3)}
    assert schema.pages_for_tokens(9) == 2


# ------------------------------------------------------------------ forward against the oracle
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_token_by_token_match_the_oracle(name):
    eng, oracle, cfg = engine(name)
    toks = prompt(cfg, 61, 1)
    want = oracle.logits(toks)
    same(eng.replay([ReplayEntry("w", toks, list(range(61)))], ["w"])[0], want)
    for i, t in enumerate(toks):
        same(eng.replay([ReplayEntry("d", [t], [0])], ["d"] if i == 60 else [])[0], want[i:i + 1])


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
        assert (got - want.float()).abs().max() < 3e-4 * max(1.0, float(want.abs().max()))
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


def seen(m, p, t):
    """Whether the query at p sees the token at t, itself or in its block."""
    if p < t:
        return False
    if p - t < m.window:
        return True
    return bool(getattr(m, "pool", 0)) and t // m.pool * m.pool + m.pool - 1 <= p - m.window


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("page,mixer", [(4, pooled(4, 2, 16, 8, 0.5, 12, 5)), (8, pooled(2, 1, 16, 8, 0.5, 9, 8)),
                                        (8, pooled(3, 3, 16, 8, 0.5, 1, 3)), (4, pooled(2, 2, 16, 8, 0.5, 10, 1)),
                                        (8, latent(2, 8, 8, 12, 16, 4, 11)), (4, latent(2, 8, 8, 12, 16, 4, 1))],
                         ids=lambda x: f"{x.kind}{x.window}p{getattr(x, 'pool', 0)}" if hasattr(x, "kind") else str(x))
def test_a_token_is_seen_exactly_in_windows_and_blocks(decoded, page, mixer):
    """One layer whose scores are nearly equal: a changed token changes the rows that see it, and no others."""
    cfg = vogunex(50, 32, 1e-5, 1.0, (mixer, FF))
    t = RandomTensors(cfg, seed=3, dtype=torch.float32, gain=1.5)
    # without the shift: it would carry a token into the next one's key as well
    zero = lambda n: torch.zeros_like(t(n)) if n.endswith("shift") else t(n)
    w = pack_weights(cfg, zero)
    toks = prompt(cfg, 40, 5)

    def logits(seq):
        eng = make_engine(cfg, w, page=page)
        if decoded:
            return np.concatenate([eng.replay([ReplayEntry("a", [t], [0])])[0] for t in seq])
        return eng.replay([ReplayEntry("a", seq, list(range(len(seq))))])[0]

    base = logits(toks)
    for t0 in (0, 1, 2, 3, 4, 5, 7, 8, 12, 20, 30):
        seq = list(toks)
        seq[t0] = (seq[t0] + 7) % cfg.vocab_size
        changed = np.abs(logits(seq) - base).max(1) > 1e-6
        assert changed.tolist() == [seen(mixer, p, t0) for p in range(40)], t0


def test_the_shift_sees_exactly_the_token_before():
    """A window of one token: a changed token reaches the row after it through the shift alone, over a portion's edge too."""
    cfg = vogunex(50, 32, 1e-5, 1.0, (latent(2, 8, 8, 12, 16, 4, 1), None))
    w = pack_weights(cfg, RandomTensors(cfg, seed=3, dtype=torch.float32, gain=1.5))
    toks = prompt(cfg, 12, 6)

    def logits(seq, cuts):
        eng, at, out = make_engine(cfg, w), 0, []
        for n in cuts:
            out.append(eng.replay([ReplayEntry("a", seq[at:at + n], list(range(n)))])[0])
            at += n
        return np.concatenate(out)

    for cuts in ((12,), (5, 7), (1,) * 12, (2,) * 6):
        base = logits(toks, cuts)
        for t0 in (0, 4, 5, 11):
            seq = list(toks)
            seq[t0] = (seq[t0] + 9) % 50
            changed = np.abs(logits(seq, cuts) - base).max(1) > 1e-6
            assert changed.tolist() == [p in (t0, t0 + 1) for p in range(12)], (cuts, t0)


def test_mixed_batches_reuse_pages_and_slots():
    """Twelve requests of unequal length through four slots and a pool that is full most of the time: portions beside
    single tokens, requests left out of steps, every logit equal to the request's alone."""
    for seed in (0, 1):
        rnd = random.Random(seed)
        eng, oracle, cfg = engine("all", pages=12)
        todo = [(f"q{i}", prompt(cfg, rnd.randrange(1, 40), 100 + i)) for i in range(12)]
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
    """A retained session goes on from its slot; a swapped-out sequence keeps its slot (states, pooled rows) and its pages, of two
    row widths, come back."""
    eng, oracle, cfg = engine("all", cls=Engine)
    a, b = prompt(cfg, 9, 8), prompt(cfg, 4, 9)
    toks, _ = run(eng, [GenerateRequest("t0", a, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    more, _ = run(eng, [GenerateRequest("t1", b, max_new_tokens=3, ignore_eos=True, session_id="s", retain_session=True)])
    assert more["t1"] == oracle.greedy(a + toks["t0"] + b, 3)
    eng, oracle, cfg = engine("all", cls=Engine, pages=7)
    eng.cfg.auto_preempt = True
    ps = {f"r{i}": prompt(cfg, 14, 70 + i) for i in range(3)}
    toks, _ = run(eng, [GenerateRequest(r, p, max_new_tokens=30, ignore_eos=True) for r, p in ps.items()])
    assert eng.stats.auto_preemptions > 0
    for r, p in ps.items():
        assert toks[r] == oracle.greedy(p, 30), r


@pytest.mark.parametrize("name", ["attention", "scan"])
def test_long_decoding(name):
    eng, oracle, cfg = engine(name, pages=40, cls=Engine)
    p = prompt(cfg, 5, 21)
    toks, _ = run(eng, [GenerateRequest("a", p, max_new_tokens=150, ignore_eos=True)])
    seq = p + toks["a"]
    assert seq[5:] == [int(i) for i in oracle.logits(seq[:-1]).argmax(-1)[4:]]


# ------------------------------------------------------------------ oracle self-checks
def test_oracle_mechanisms():
    h = torch.arange(6.0, dtype=torch.float64).view(3, 2)
    assert VO.token_shift(h, torch.tensor([1.0, 0.5], dtype=torch.float64)).tolist() == [[0, 0.5], [0, 2], [2, 4]]
    assert VO.window(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    # blocks of two tokens behind a window of three: block 0 (tokens 0, 1) from position 4 on
    assert VO.pooled_visible(7, 3, 2).int().tolist() == [[0, 0, 0]] * 4 + [[1, 0, 0]] * 2 + [[1, 1, 0]]
    assert VO.block_means(torch.tensor([[1.0], [3.0], [5.0], [9.0], [2.0]]), 2).tolist() == [[2.0], [7.0]]
    x = torch.rand(5, 2, 10, dtype=torch.float64)
    for turn in (VO.rotate_halves, VO.rotate_pairs):
        y = turn(x, 100.0, 6)
        assert torch.allclose(y.norm(dim=-1), x.norm(dim=-1)) and torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    perm = [0, 2, 4, 1, 3, 5, 6, 7, 8, 9]
    assert torch.allclose(VO.rotate_pairs(x, 100.0, 6)[..., perm], VO.rotate_halves(x[..., perm], 100.0, 6))
    w = torch.rand(3, 4, 4, dtype=torch.float64)
    assert torch.equal(VO.mixed_weights(w, torch.eye(3, dtype=torch.float64)), w)
    assert VO.softcap(torch.tensor([1e9, 0.0, 1e-9]), 5.0).tolist() == pytest.approx([5.0, 0.0, 1e-9])
    r = VO.route(torch.tensor([[1.0, 3.0, 2.0, -1.0]], dtype=torch.float64), 2)
    assert r[0, [0, 3]].tolist() == [0, 0] and math.isclose(float(r.sum()), 1.0) and math.isclose(float(r[0, 1] / r[0, 2]), math.e)
    # a scan whose decay is one and whose inputs are units: sums of the inputs
    one = torch.ones(4, 1, 1, dtype=torch.float64)
    y = VO.scalar_decay_scan(one, one, one, one[..., 0], torch.zeros(1, dtype=torch.float64), torch.zeros(1, dtype=torch.float64))
    assert y.flatten().tolist() == [1, 2, 3, 4]
    z = torch.linspace(-30, 30, 33, dtype=torch.float64)
    assert torch.allclose(VO.softplus(z), torch.nn.functional.softplus(z, threshold=100)) and torch.allclose(VO.gelu(z), torch.nn.functional.gelu(z))


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
    assert json.loads(cli("make-fixture", "--family", "vogunex", "--out", d))["family"] == "vogunex"
    assert '"vogunex"' in cli("info", d)
    out = json.loads(cli("generate", "--model-dir", d, "--device", "cpu", "--tokens", "5,6,7", "-n", "4", "--ignore-eos", "--json"))
    cfg = tiny_vogunex()
    assert out["tokens"] == VO.Oracle(to_layer_list(cfg), RandomTensors(cfg, 0)).greedy([5, 6, 7], 4)
