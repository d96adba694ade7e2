"""Gidurax configurations drawn at random (layer order, every size, repeated runs, feed-forwards of either kind or none, temperatures or
none, shared experts and identities or none), each run as one batch of unequal prompts whose last tokens are decoded together, in
32-bit and in bfloat16, against the plain implementation.  IERT_TEST_RANDOM_GIDURAX=N draws N configurations instead of eight."""
import os
import random

import pytest
import torch

import test_gpu_gidurax as T
from plain import gidurax_plain as P

pytestmark = pytest.mark.gpu

COUNT = int(os.environ.get("IERT_TEST_RANDOM_GIDURAX", "8"))


def draw_mixer(rng):
    kind = rng.choice(["delta", "attention", "mamba1"])
    kv, group = rng.choice([1, 2, 3, 4]), rng.choice([1, 2, 3])
    if kind == "delta":
        return T.delta(heads=kv * group, kv_heads=kv, dim=rng.choice([16, 24, 32, 64]), vdim=rng.choice([7, 16, 24, 32, 64, 96]), conv=rng.choice([1, 2, 3, 4, 6]))
    if kind == "attention":
        dim = rng.choice([4, 8, 16, 24, 32, 48, 64, 80, 128])
        return T.attn(heads=kv * group, kv_heads=kv, dim=dim, vdim=rng.choice([dim, 8, 20, 48, 64]), scale=round(dim ** -0.5 * rng.choice([0.5, 1.0]), 4),
                      temp=rng.choice([None, (0.3, 1), (0.5, 16), (0.2, 33), (-0.1, 64)]))
    return T.scan(inner=rng.choice([24, 40, 63, 64, 128, 200]), state=rng.choice([1, 4, 8, 13, 16, 24, 32, 50]), dt_rank=rng.choice([1, 5, 8, 12, 16, 40]),
                  conv=rng.choice([1, 2, 3, 4, 5]))


def draw_mlp(rng):
    return rng.choice([None, T.dense(rng.choice([5, 24, 64, 136])), T.dense(64),
                       T.moe(ff=rng.choice([5, 8, 24, 64]), experts=rng.choice([1, 3, 6, 9]), top=1 + rng.randrange(2), identity=rng.choice([None, 1, 3]),
                             shared=rng.choice([None, 9, 32, 64]))])


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("random_gidurax"))


@pytest.mark.parametrize("case", range(COUNT))
def test_random_configuration(root, case):
    rng = random.Random(7000 + case)
    n = rng.choice([1, 2, 3, 4])
    layers = [T.layer(draw_mixer(rng), draw_mlp(rng)) for _ in range(n)]
    for l in layers:
        if l["mlp"] and l["mlp"]["kind"] == "moe":
            r = l["mlp"]["router"]
            r["top"] = min(r["top"], r["experts"] + r.get("identity", 0))
    start = rng.randrange(n)
    cfg = T.config(layers, width=rng.choice([40, 50, 64, 100, 128, 192]), vocab=rng.choice([61, 256, 500]), eps=rng.choice([1e-5, 1e-6]), embed=rng.choice([1.0, 3.0, 11.0]),
                   mult=rng.choice([1.0, 0.7, 0.3]), loop=rng.choice([None, (start, rng.randint(start + 1, n), rng.choice([1, 2, 3]))]))
    prompts = T.tokens(cfg, (1, rng.randint(2, 60), rng.randint(61, 140), rng.randint(141, 260)), seed=case)
    runs = len(P.runs(cfg))
    for dtype in ("float32", "bfloat16"):
        model, weights = T.make_model(root, cfg, 100 + case, dtype, std=0.08)
        want = [P.forward(cfg, weights, p, T.rounding(dtype)) for p in prompts]
        eng = T.engine_of(model, max_tokens=64 * 12, max_sequences=4)
        slots = [eng.open_sequence() for _ in prompts]
        tails = [min(len(p) - 1, 6 + 33 * i) for i, p in enumerate(prompts)]
        rows = [[] for _ in prompts]
        got, at = eng.step([(s, p[:len(p) - t]) for s, p, t in zip(slots, prompts, tails)], want="all"), 0
        for i, (p, t) in enumerate(zip(prompts, tails)):
            rows[i].append(got[at:at + len(p) - t])
            at += len(p) - t
        pos = [len(p) - t for p, t in zip(prompts, tails)]
        live = [i for i in range(len(prompts)) if pos[i] < len(prompts[i])]
        for i in range(len(prompts)):
            if i not in live:
                eng.close_sequence(slots[i])
        while live:
            got = eng.step([(slots[i], [prompts[i][pos[i]]]) for i in live], want="last")
            for k, i in enumerate(live):
                rows[i].append(got[k:k + 1])
                pos[i] += 1
            for i in [i for i in live if pos[i] == len(prompts[i])]:
                eng.close_sequence(slots[i])
                live.remove(i)
        eng.check_device()
        for i, p in enumerate(prompts):
            slack = max(1.0, runs / 3)
            if dtype == "bfloat16":         # how far rounding alone moves this model (a read-out near zero under a norm moves far)
                exact = P.forward(cfg, weights, p)
                noise = ((exact - want[i]).pow(2).mean(-1).sqrt() / exact.abs().max()).max().item()
                slack = max(slack, 1.5 * noise / 0.012)
            T.compare(torch.cat(rows[i]), want[i], dtype, f"case {case} ({dtype}), request {i}: {cfg}", slack=slack)
