
import os, torch, torch.distributed as dist
from ferrule_b200.models import config as C, weights as W, deepseek as D
from ferrule_b200.parallel.pp import PipelineParallel, stage_weights
dist.init_process_group("gloo")
rank, world = dist.get_rank(), dist.get_world_size()
cfg = C.tiny_fixture()
w = W.random_weights(cfg, device="cpu", seed=0)
page = 16
def batch(lens, new, seed):
    g = torch.Generator().manual_seed(seed)
    ids, pos, slot, rseq, lrows = [], [], [], [], []
    bt = torch.zeros(len(lens), 8, dtype=torch.int32)
    pc = 1
    for s, (n0, nn) in enumerate(zip(lens, new)):
        for j in range((n0 + nn + page - 1) // page):
            bt[s, j] = pc; pc += 1
        for j in range(nn):
            p_ = n0 + j
            ids.append(int(torch.randint(0, cfg.vocab_size, (1,), generator=g))); pos.append(p_)
            slot.append(int(bt[s, p_ // page]) * page + p_ % page); rseq.append(s)
        lrows.append(len(ids) - 1)
    t = lambda v, dt: torch.tensor(v, dtype=dt)
    return D.DeviceBatch(t(ids, torch.int32), t(pos, torch.int32), t(slot, torch.int64), t(rseq, torch.int32),
                         t(pos, torch.int32), bt, t(lrows, torch.int32), len(ids), len(lrows))
full = D.ReferenceForward(w, D.KvPool(cfg, 32, page, "cpu", dtype=torch.float32))
ws = stage_weights(w, rank, world)
stage = D.ReferenceForward(ws, D.KvPool(ws.cfg, 32, page, "cpu", dtype=torch.float32))
pp = PipelineParallel(rank, world)
ok = True
lens, new = [0, 0], [19, 7]
for step in range(3):
    b = batch(lens, new, step)
    want = full.forward(b)
    ids, vals = pp.step(stage, b, cfg.hidden, torch.float32, cuda=False)
    ok &= bool(torch.equal(ids.long(), want.argmax(-1))) and bool(torch.allclose(vals, want.max(-1).values, atol=1e-4))
    lens = [l + n for l, n in zip(lens, new)]; new = [1, 1]
# micro-batched decode: two row ranges in flight
pp2 = PipelineParallel(rank, world, microbatches=2)
b = batch(lens, [1, 1], 9)
want = full.forward(b)
ids, vals = pp2.step(stage, b, cfg.hidden, torch.float32, cuda=False)
ok &= bool(torch.equal(ids.long(), want.argmax(-1)))
print("PP_OK" if ok else "PP_BAD", rank, flush=True)
dist.destroy_process_group()
