"""Botulorn configurations drawn at random (layer order, every size, windows and kept first positions on and off the page
size, rotations on part of a head, stretched or none, value sizes unlike the key's, value mixing or not, layers without a
feed-forward, with and without the pair embedding), each run as one batch of unequal prompts whose last tokens are decoded
together, in 32-bit and in bfloat16, against the plain implementation.  IERT_TEST_RANDOM_BOTULORN=N draws N configurations
instead of eight."""
import os
import random

import pytest
import torch

import test_gpu_botulorn as T
from plain import botulorn_plain as P

pytestmark = pytest.mark.gpu

COUNT = int(os.environ.get("IERT_TEST_RANDOM_BOTULORN", "8"))


def draw_scaling(rng):
    return rng.choice([None, T.stretch(rng.choice([1.5, 4.0, 16.0]), rng.choice([30, 100, 1000]), rng.choice([32.0, 4.0]), rng.choice([1.0, 0.25]))])


def draw_mixer(rng, mixing):
    if rng.random() < 0.55:
        dim = rng.choice([4, 8, 16, 24, 32, 48, 64, 80, 128, 192])
        kv, vdim = mixing if rng.random() < 0.7 else (rng.choice([1, 2, 3, 4]), rng.choice([dim, 8, 20, 48, 64]))
        dims = rng.choice([None, dim // 4 * 2, dim // 2, dim])
        return "attention", T.attn(heads=kv * rng.choice([1, 2, 3]), kv_heads=kv, dim=dim, vdim=vdim, scale=round(dim ** -0.5 * rng.choice([0.3, 0.5, 1.0]), 4),
                                   rotation=None if dims is None else T.rot(dims // 2 * 2, rng.choice([100.0, 10000.0, 500000.0]), draw_scaling(rng)),
                                   window=rng.choice([None, 1, 7, 32, 63, 64, 65, 100, 128, 200]), keep=rng.choice([None, 0, 1, 4, 63, 64, 65, 130]),
                                   v_mix=(kv, vdim) == mixing)
    dim, rot_dim = rng.choice([4, 8, 16, 24, 32, 64]), rng.choice([0, 2, 4, 8, 16, 32])
    return "latent_attention", T.latent(heads=rng.choice([1, 2, 3, 4, 8, 17, 33]), dim=dim, rot_dim=rot_dim, vdim=rng.choice([dim, dim + rot_dim, 8, 20, 48, 64]),
                                        q_rank=rng.choice([8, 15, 32, 48]), kv_rank=rng.choice([8, 20, 32, 40, 64, 96, 128, 192]),
                                        scale=round((dim + rot_dim) ** -0.5 * rng.choice([0.5, 1.0]), 4), base=rng.choice([100.0, 10000.0]),
                                        scaling=draw_scaling(rng), window=rng.choice([None, 1, 31, 64, 65, 100, 190]))


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("random_botulorn"))


@pytest.mark.parametrize("case", range(COUNT))
def test_random_configuration(root, case):
    rng = random.Random(9000 + case)
    mixing = (rng.choice([1, 2, 3]), rng.choice([8, 20, 48, 64]))
    n = rng.choice([1, 2, 3, 4, 5])
    layers = [T.layer(*draw_mixer(rng, mixing), T.dense(rng.choice([5, 24, 64, 136])) if rng.random() < 0.8 else None) for _ in range(n)]
    cfg = T.config(layers, width=rng.choice([40, 50, 64, 100, 128, 192, 320]), vocab=rng.choice([61, 256, 500]), eps=rng.choice([1e-5, 1e-6]),
                   embed=rng.choice([1.0, 3.0, 11.0]), bigram=rng.choice([None, (1, 1, 1), (37, 5, 0), (1531, 1000003, 77)]))
    prompts = T.tokens(cfg, (1, rng.randint(2, 60), rng.randint(61, 140), rng.randint(141, 330)), seed=case)
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
        for i in range(len(prompts)):
            T.compare(torch.cat(rows[i]), want[i], dtype, f"case {case} ({dtype}), request {i}: {cfg}", slack=max(1.0, n / 2.5))
