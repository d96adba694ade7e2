"""The Botulorn design in the engine against the plain statement of its equations (`tests/plain/botulorn_plain.py`):
each mechanism alone (kernels against one function of the plain statement, and one-layer models), then whole models under
every way of cutting the work: whole prompts, tokens one by one through the cache and the state, batches of unequal
requests through slots and pages that are used again, long decoding that goes round the ring of a window several times,
short prompt steps replayed as graphs, and greedy generation through the session.  Sizes differ from test to test (also
sizes that are 1 or equal to one another), and where random weights would hide a fault the weights are made so that it
shows: one key that decides, just inside and just outside a window and among or behind the kept first positions."""
import json
import os

import pytest
import torch

from helpers import compare as compare_exactly, plain_weights, prompts_for
from plain import botulorn_plain as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def compare(got, ref, dtype, what="", slack=1.0):
    """float32: every logit within 2e-4, absolute + relative.  bfloat16: both sides round activations to bfloat16, but not
    at exactly the same places: the root-mean-square error of every row against the largest logit below 1.2 %, of the
    median row below 0.6 %."""
    if dtype == "float32":
        return compare_exactly(got, ref, dtype, what)
    got, ref = torch.as_tensor(got).float().cpu(), torch.as_tensor(ref).float().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite values"
    rows = (got - ref).pow(2).mean(-1).sqrt() / ref.abs().max()
    assert rows.max() < 0.012 * slack, f"{what}: row {int(rows.argmax())} is off by {rows.max().item():.3g} of the largest logit"
    assert len(rows) < 8 or rows.median() < 0.006 * slack, f"{what}: the median row is off by {rows.median().item():.3g}"


def stretch(factor=3.0, original=60, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rot(dims, base=900.0, scaling=None):
    out = {"base": base, "dims": dims}
    if scaling is not None:
        out["scaling"] = dict(scaling)
    return out


def attn(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.5, rotation=rot(8, scaling=stretch()), window=27, keep=3, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if rotation is not None:
        m["rot"] = dict(rotation)
    if window is not None:
        m["mask"] = {"size": window}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    return m


def latent(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=40, scale=0.3, base=700.0, scaling=stretch(2.0, 90), window=22):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot_dim:
        m["rot"] = rot(rot_dim, base, scaling)
    if window is not None:
        m["mask"] = {"size": window}
    return m


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, width=64, vocab=96, eps=1e-5, embed=3.0, bigram=(53, 17, 5)):
    e = {"scale": embed}
    if bigram is not None:
        e["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    return {"architecture": "Botulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": e,
            "layers": json.loads(json.dumps(layers))}


ALONE = {
    "attention": [layer("attention", attn())],
    "attention, equal sizes": [layer("attention", attn(heads=2, kv_heads=2, dim=16, vdim=16, rotation=rot(16), v_mix=False))],
    "attention, wide values": [layer("attention", attn(heads=3, kv_heads=1, dim=8, vdim=40, rotation=rot(2, 50.0), window=64, keep=1))],
    "attention, a window of one": [layer("attention", attn(heads=1, kv_heads=1, window=1, keep=0))],
    "attention, a window of one and a kept first": [layer("attention", attn(heads=2, kv_heads=1, window=1, keep=1))],
    "attention, more kept than the window": [layer("attention", attn(window=9, keep=70))],
    "attention, no first kept": [layer("attention", attn(window=65, keep=None))],
    "attention without a mask or a rotation": [layer("attention", attn(rotation=None, window=None))],
    "attention twice, values mixed": [layer("attention", attn()), layer("attention", attn(dim=24, rotation=rot(24)))],
    "a layer between that does not mix": [layer("attention", attn()), layer("attention", attn(kv_heads=1, vdim=8, v_mix=False)),
                                          layer("attention", attn(heads=6))],
    "latent attention": [layer("latent_attention", latent())],
    "latent attention, one head, equal sizes": [layer("latent_attention", latent(heads=1, dim=32, rot_dim=32, vdim=32, q_rank=32, kv_rank=32, window=64))],
    "latent attention, value as wide as the key": [layer("latent_attention", latent(heads=2, dim=16, rot_dim=16, vdim=32, scaling=None))],
    "latent attention without a rotated part": [layer("latent_attention", latent(rot_dim=0, window=None))],
    "latent attention, a window of one": [layer("latent_attention", latent(window=1))],
    "dense": [layer("attention", attn(), dense())],
    "latent and dense": [layer("latent_attention", latent(), dense(24))],
}

FULL = config([layer("attention", attn(), dense()),
               layer("latent_attention", latent(), dense(40)),
               layer("latent_attention", latent(heads=2, dim=8, rot_dim=4, vdim=8, q_rank=12, kv_rank=16, window=70), None),
               layer("attention", attn(heads=2, dim=32, rotation=rot(32, 5000.0, stretch(4.0, 40, 4.0, 0.5)), window=80, keep=5), dense(24)),
               layer("attention", attn(v_mix=False, window=33, keep=0), dense())])
# sizes no kernel for the tensor cores takes: everything runs the plain kernels, also in bfloat16
ODD = config([layer("latent_attention", latent(heads=3, dim=10, rot_dim=6, vdim=14, q_rank=9, kv_rank=22, window=37), dense(21)),
              layer("attention", attn(heads=3, kv_heads=3, dim=10, vdim=7, rotation=rot(6), window=29, keep=67), None),
              layer("attention", attn(heads=6, kv_heads=3, dim=14, vdim=7, rotation=rot(14, scaling=stretch()), window=None), dense(5))],
             width=50, vocab=75, eps=1e-6, embed=1.0, bigram=(7, 0, 1))
# sizes the tensor-core kernels take: tcgen05 prompt attention at head size 64, the one-token latent kernel
TENSOR = config([layer("latent_attention", latent(heads=4, dim=48, rot_dim=16, vdim=64, q_rank=48, kv_rank=64, scale=0.25, window=100), dense(136)),
                 layer("attention", attn(heads=4, kv_heads=2, dim=64, vdim=48, scale=0.3, rotation=rot(64, scaling=stretch()), window=75, keep=6), dense(136)),
                 layer("latent_attention", latent(heads=20, dim=16, rot_dim=16, vdim=32, q_rank=40, kv_rank=160, scale=0.25, window=64), dense(136)),
                 layer("attention", attn(heads=8, kv_heads=2, dim=48, vdim=48, scale=0.3, rotation=rot(32, scaling=stretch()), window=130, keep=65), dense(136))],
                width=128, vocab=160, embed=6.0, bigram=(211, 3, 11))
WIDE_HEADS = config([layer("attention", attn(heads=2, kv_heads=1, dim=128, vdim=96, scale=0.2, rotation=rot(128), window=130, keep=2), dense(64)),
                     layer("latent_attention", latent(heads=2, dim=128, rot_dim=64, vdim=128, q_rank=64, kv_rank=256, scale=0.2, window=150), None),
                     layer("attention", attn(heads=2, kv_heads=1, dim=96, vdim=96, scale=0.2, rotation=rot(40), window=None), dense(32))],
                    width=120, vocab=128, bigram=None)
WHOLE_MODELS = {"full": FULL, "odd": ODD, "tensor": TENSOR, "wide_heads": WIDE_HEADS}


def spread(tensors):
    """Mixing weights inside (0, 1), gates that differ from head to head, norm biases and hashed rows that matter."""
    n = 0
    for name in sorted(tensors):
        if name.endswith(".mix.vmix"):
            tensors[name] = torch.tensor(0.25 + 0.25 * (n % 3), dtype=tensors[name].dtype)
            n += 1
        elif name.endswith(".mix.g"):
            tensors[name] = tensors[name] * 3.0
        elif name.endswith(".b"):
            tensors[name] = tensors[name] * 3.0
        elif name == "bigram":
            tensors[name] = tensors[name] * 4.0


def make_model(root, cfg, seed, dtype, edit=spread, std=0.1):
    from safetensors.torch import load_file, save_file
    from inference_engine_rust_b200 import LoadedModel, write_random_model
    d = os.path.join(root, f"m{abs(hash((json.dumps(cfg, sort_keys=True), seed, dtype, getattr(edit, '__name__', None)))) % 10 ** 9}")
    if not os.path.isdir(d):
        write_random_model(d, cfg, seed=seed, dtype=dtype, std=std)
        if edit is not None:
            path = os.path.join(d, "model.safetensors")
            tensors = load_file(path)
            edit(tensors)
            save_file({k: v.contiguous() for k, v in tensors.items()}, path)
    return LoadedModel.load(d, dtype=dtype), plain_weights(d)


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("botulorn"))


def rounding(dtype):
    return P.bf16 if dtype == "bfloat16" else P.exact


def engine_of(model, max_tokens=64 * 16, **kw):
    return model.session(max_tokens=max_tokens, poison_cache=True, **kw).engine


def run_whole(eng, prompt):
    slot = eng.open_sequence()
    got = eng.step([(slot, prompt)], want="all")
    eng.check_device()
    eng.close_sequence(slot)
    return got


def tokens(cfg, lengths, seed=0):
    return prompts_for({"vocab_size": cfg["vocab"]}, lengths, seed=seed)


def B():
    from inference_engine_rust_b200.csrc import bindings
    return bindings


def stream():
    return torch.cuda.current_stream().cuda_stream


class Batch:
    """The device arrays of a step over sequences in `slots` that bring `q_lens` tokens behind `pos0` earlier ones."""

    def __init__(self, q_lens, pos0, slots, pad=0):
        cu = [0]
        for n in q_lens:
            cu.append(cu[-1] + n)
        seq = sum(([i] * n for i, n in enumerate(q_lens)), []) + [-1] * pad
        self.arrays = [torch.tensor(a, dtype=torch.int32, device=DEV) for a in (cu, slots, seq, pos0)]
        self.n_tokens = len(seq)
        c, s, t, p = (a.data_ptr() for a in self.arrays)
        self.view = B().BatchView(cu_q=c, slot_ids=s, tok_seq=t, pos0=p, n_seqs=len(q_lens), n_tokens=self.n_tokens)


# ---------------------------------------------------------------------------------------
# kernels against one function of the plain statement each


@pytest.mark.parametrize("width", [8, 52, 128, 130, 1000, 2048, 4096, 5120, 9000])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_two_norms_of_one_row(width, dtype):
    """Both norms of a layer in one pass, and one norm alone on gathered rows; rows with a large mean."""
    g = torch.Generator().manual_seed(width)
    x = torch.randn(7, width, generator=g) + 30.0
    w, b, w2, b2 = (torch.randn(width, generator=g) for _ in range(4))
    dt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    out, out2 = (torch.empty(7, width, dtype=dt, device=DEV) for _ in range(2))
    B().layernorm(x.to(DEV), out, w.to(DEV), b.to(DEV), 1e-5, 7, stream(), second=(w2.to(DEV), b2.to(DEV), out2))
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == "bfloat16" else dict(rtol=2e-4, atol=2e-4)
    torch.testing.assert_close(out.float().cpu(), P.layer_norm(x, w, b, 1e-5), **tol)
    torch.testing.assert_close(out2.float().cpu(), P.layer_norm(x, w2, b2, 1e-5), **tol)
    idx = torch.tensor([5, 0, 5], dtype=torch.int32, device=DEV)
    B().layernorm(x.to(DEV), out[:3], w.to(DEV), b.to(DEV), 1e-5, 3, stream(), rows_idx=idx)
    torch.testing.assert_close(out[:3].float().cpu(), P.layer_norm(x[[5, 0, 5]], w, b, 1e-5), **tol)


@pytest.mark.parametrize("table_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [24, 50, 1024, 1536, 4096, 5120])
@pytest.mark.parametrize("buckets,mul_prev,mul_cur", [(53, 17, 5), (1, 3, 4), (97, 0, 1), (65521, 2 ** 31 - 1, 2 ** 33 + 7)])
def test_pair_embedding_and_its_state(hidden, buckets, mul_prev, mul_cur, table_dtype):
    """Unequal prompts, then single tokens and a longer continuation: the token in front of a step's first one comes from
    the slot's state; a slot that starts anew does not read what the sequence before it left; padding writes no state."""
    vocab, scale = 300, 2.5
    g = torch.Generator().manual_seed(hidden + buckets)
    if buckets > 1000 and hidden > 1024:
        buckets = 8191
    table = torch.randn(vocab, hidden, generator=g).to(table_dtype)
    pairs = torch.randn(buckets + 1, hidden, generator=g).to(table_dtype)
    td, pd = table.to(DEV), pairs.to(DEV)
    last = torch.full((5, 3), 7, dtype=torch.int32, device=DEV)
    seqs = {1: torch.randint(0, vocab, (40,), generator=g).tolist(), 4: torch.randint(0, vocab, (9,), generator=g).tolist()}
    cfg = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}
    want = {s: P.embed(cfg, {"embed": table, "bigram": pairs}, t) for s, t in seqs.items()}
    pos = {1: 0, 4: 0}
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    for plan in ({1: 5, 4: 1}, {1: 1, 4: 1}, {4: 1}, {1: 8, 4: 6}, {1: 26}):
        slots = list(plan)
        bt = Batch([plan[s] for s in slots], [pos[s] for s in slots], slots, pad=2)
        ids = sum((seqs[s][pos[s]:pos[s] + plan[s]] for s in slots), []) + [0, 1]
        x = torch.full((len(ids), hidden), float("nan"), device=DEV)
        B().embed_pairs(td, pd, torch.tensor(ids, dtype=torch.int32, device=DEV), x, scale, buckets, mul_prev, mul_cur, last, bt.view,
                        err, stream())
        ref = torch.cat([want[s][pos[s]:pos[s] + plan[s]] for s in slots] + [table[:2].float() * scale])
        torch.testing.assert_close(x.cpu(), ref, rtol=1e-6, atol=1e-6)
        for s in slots:
            pos[s] += plan[s]
    assert last[1, 0] == seqs[1][-1] and last[4, 0] == seqs[4][-1]
    assert (last[:, 1:] == 7).all() and (last[[0, 2, 3], 0] == 7).all() and int(err) == 0


@pytest.mark.parametrize("D,vdim,rotary,half,heads,kv,ld_odd", [
    (16, 16, 16, True, 4, 2, False), (16, 24, 8, True, 3, 3, False), (128, 128, 128, True, 8, 2, False), (192, 64, 72, True, 2, 1, False),
    (20, 12, 12, True, 4, 2, False), (10, 6, 6, True, 2, 2, True), (32, 32, 24, False, 4, 1, False), (12, 12, 0, True, 2, 1, False)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_query_key_value_preparation(D, vdim, rotary, half, heads, kv, ld_odd, dtype):
    """Norm per head, rotation of either pairing with a factor on cosine and sine, values mixed with another layer's, at
    positions that do not start at 0; sizes that the 16-byte accesses take and sizes that they do not."""
    b = B()
    g = torch.Generator().manual_seed(D * 10 + rotary)
    T, pos0, lam, mul = 5, 37, 0.3, 1.2
    P_ = max(D, vdim) if dtype == "float32" else -(-max(D, vdim) // 16) * 16
    n = heads * D + kv * (D + vdim)
    proj = torch.randn(T, n + (3 if ld_odd else 4), generator=g)
    vf = torch.randn(T, kv * vdim + 4, generator=g)
    wq, wk = torch.randn(D, generator=g), torch.randn(D, generator=g)
    rates = torch.rand(max(rotary // 2, 1), generator=g)
    q, k, v = proj[:, :heads * D].view(T, heads, D), proj[:, heads * D:(heads + kv) * D].view(T, kv, D), proj[:, (heads + kv) * D:n].view(T, kv, vdim)

    def turned(x, w):
        x = P.rms_norm(x, w, 1e-5)
        out = x.clone()
        ang = torch.arange(pos0, pos0 + T).float()[:, None] * rates[None, :rotary // 2]
        c, s = (torch.cos(ang) * mul)[:, None], (torch.sin(ang) * mul)[:, None]
        i0 = torch.arange(rotary // 2) if half else 2 * torch.arange(rotary // 2)
        i1 = i0 + rotary // 2 if half else i0 + 1
        out[..., i0], out[..., i1] = x[..., i0] * c - x[..., i1] * s, x[..., i1] * c + x[..., i0] * s
        return out
    dt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    cache = torch.full((2, 4, kv, 64, P_), float("nan"), dtype=dt, device=DEV)
    table = torch.tensor([[-1, -1], [2, 1]], dtype=torch.int32, device=DEV)
    kvv = b.KvView(k=cache[0].data_ptr(), v=cache[1].data_ptr(), page_table=table.data_ptr(), table_width=2, ring_pages=2, page_tokens=64,
                   n_pages=4, kv_heads=kv, head_dim=P_, dtype=b.dtype_code(dt), window=0, chunk=0)
    bt = Batch([T], [pos0], [1])
    qkv = torch.full((T, (heads + 2 * kv) * P_), float("nan"), dtype=dt, device=DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    b.qkv_prep(proj.to(DEV), None, qkv, bt.view, kvv, heads, D, vdim, rates.to(DEV), rotary, b.PAIR_HALF if half else b.PAIR_INTERLEAVED,
               wq.to(DEV), wk.to(DEV), 1e-5, True, err, stream(), rot_mul=mul, v_first=vf.to(DEV)[:, :kv * vdim], lam=lam)
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == "bfloat16" else dict(rtol=2e-5, atol=2e-5)
    got = qkv.float().cpu().view(T, heads + 2 * kv, P_)
    vm = (1.0 - lam) * v + lam * vf[:, :kv * vdim].view(T, kv, vdim)
    torch.testing.assert_close(got[:, :heads, :D], turned(q, wq), **tol)
    torch.testing.assert_close(got[:, heads:heads + kv, :D], turned(k, wk), **tol)
    torch.testing.assert_close(got[:, heads + kv:, :vdim], vm, **tol)
    assert (got[:, :heads + kv, D:] == 0).all() and (got[:, heads + kv:, vdim:] == 0).all() and int(err) == 0
    stored = cache[:, 2, :, pos0:pos0 + T].float().cpu()
    assert torch.equal(stored[0].transpose(0, 1), got[:, heads:heads + kv]) and torch.equal(stored[1].transpose(0, 1), got[:, heads + kv:])


@pytest.mark.parametrize("D", [48, 64, 128, 192])
@pytest.mark.parametrize("window,keep", [(70, 5), (64, 64), (1, 1), (130, 67), (33, 0), (10, 200), (0, 9)])
def test_prompt_attention_with_kept_positions(D, window, keep):
    """The tensor-core prompt kernels and the plain one under a window with kept first positions, on packed prompts of
    unequal lengths; scores are sharp (large queries), so one key too many or too few shows."""
    b = B()
    g = torch.Generator().manual_seed(D + window)
    H, G, lens = 4, 2, [1, 300, 65, 190]
    T = sum(lens)
    qkv = torch.randn(T, (H + 2 * G) * D, generator=g)
    qkv[:, :H * D] *= 3.0
    qkv = qkv.to(torch.bfloat16)
    bt = Batch(lens, [0] * 4, [3, 1, 0, 2])
    scale = D ** -0.5
    want = torch.cat([P.masked_attention(*(x.float() for x in qkv[a:a + n].view(n, H + 2 * G, D).split([H, G, G], dim=1)), scale,
                                         P.visible(n, window or None, keep)).reshape(n, H * D)
                      for a, n in zip([0, 1, 301, 366], lens)])
    qd = qkv.to(DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.empty(T, H * D, dtype=torch.bfloat16, device=DEV)
    for legacy in (False, True):
        out.fill_(float("nan"))
        assert b.attention_prefill(qd, out, bt.view, H, G, D, window, scale, max(lens), stream(), err=err, legacy=legacy, keep=keep)
        torch.testing.assert_close(out.float().cpu(), want, rtol=2e-2, atol=2e-2)
    own = b.KvView(k=None, v=None, page_table=None, table_width=0, ring_pages=1, page_tokens=1, n_pages=0, kv_heads=G, head_dim=D,
                   dtype=b.F32, window=window, chunk=0, keep=keep)
    full = torch.empty(T, H * D, device=DEV)
    b.attention_plain(qd.float(), full, bt.view, own, H, scale, False, err, stream())
    torch.testing.assert_close(full.cpu(), want, rtol=1e-4, atol=1e-4)
    assert int(err) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(root, name, dtype):
    """One to three layers: prompts, and the same tokens partly one by one (over page borders and round the windows' rings)."""
    cfg = config(ALONE[name])
    model, weights = make_model(root, cfg, 3, dtype)
    eng = engine_of(model)
    for prompt, first in zip(tokens(cfg, (1, 2, 210), seed=1), (1, 1, 60)):
        ref = P.forward(cfg, weights, prompt, rounding(dtype))
        compare(run_whole(eng, prompt), ref, dtype, f"{name}, {len(prompt)} tokens")
        slot = eng.open_sequence()
        rows = [eng.step([(slot, prompt[:first])], want="all")] + [eng.step([(slot, [t])], want="last") for t in prompt[first:]]
        eng.check_device()
        eng.close_sequence(slot)
        compare(torch.cat(rows), ref, dtype, f"{name}, {first} tokens and {len(prompt) - first} one by one")


def test_residual_after_every_layer(root):
    model, weights = make_model(root, FULL, 5, "float32")
    eng = engine_of(model)
    prompt = tokens(FULL, (37,), seed=2)[0]
    want, got = [], []
    P.forward(FULL, weights, prompt, residuals=want)
    model.model.after_block = lambda pos, rows, ctx: got.append(rows[:ctx.n_tokens].clone())
    try:
        run_whole(eng, prompt)
    finally:
        model.model.after_block = None
    assert len(got) == len(want) == 5
    for i, (g, w) in enumerate(zip(got, want)):
        compare(g, w, "float32", f"residual after layer {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(WHOLE_MODELS))
def test_whole_prompts(root, name, dtype):
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 7, dtype)
    eng = engine_of(model)
    for prompt in tokens(cfg, (1, 3, 64, 65, 300), seed=3):
        compare(run_whole(eng, prompt), P.forward(cfg, weights, prompt, rounding(dtype)), dtype, f"{name}, {len(prompt)} tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(WHOLE_MODELS))
def test_prompt_then_tokens_one_by_one(root, name, dtype):
    """A prompt in one step, then single tokens over page borders and several times round the windows' rings; also from
    the very first token on and from a prompt of two tokens, and behind a prompt longer than every ring."""
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 8, dtype)
    eng = engine_of(model)
    for first, total in ((1, 30), (2, 75), (61, 61 + 340), (400, 470)):
        seq = tokens(cfg, (total,), seed=first)[0]
        ref = P.forward(cfg, weights, seq, rounding(dtype))
        slot = eng.open_sequence()
        rows = [eng.step([(slot, seq[:first])], want="all")]
        for t in seq[first:]:
            rows.append(eng.step([(slot, [t])], want="last"))
        eng.check_device()
        eng.close_sequence(slot)
        compare(torch.cat(rows), ref, dtype, f"{name}: {first} tokens, then {total - first} one by one")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(WHOLE_MODELS))
def test_unequal_batches_through_slots_and_pages_used_again(root, name, dtype):
    """Batches of unequal requests decoded together, the shorter ones ending earlier, in a cache so small that slots,
    pages and states are handed out again (pages poisoned when freed): every row equals the request run alone."""
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 9, dtype)
    eng = engine_of(model, max_tokens=64 * 9, max_sequences=4)
    for wave, lengths in enumerate(((1, 70, 5), (130, 2, 64, 33), (3, 280))):
        seqs = tokens(cfg, [n + d for n, d in zip(lengths, (9, 3, 14, 6))], seed=10 + wave)
        refs = [P.forward(cfg, weights, s, rounding(dtype)) for s in seqs]
        slots = [eng.open_sequence() for _ in seqs]
        got = [[] for _ in seqs]
        out = eng.step([(sl, s[:n]) for sl, s, n in zip(slots, seqs, lengths)], want=[[n - 1] for n in lengths])
        for i in range(len(seqs)):
            got[i].append(out[i:i + 1])
        done = list(lengths)
        live = list(range(len(seqs)))
        while live:
            out = eng.step([(slots[i], [seqs[i][done[i]]]) for i in live], want="last")
            for r, i in enumerate(live):
                got[i].append(out[r:r + 1])
                done[i] += 1
            for i in [i for i in live if done[i] == len(seqs[i])]:
                eng.close_sequence(slots[i])
                live.remove(i)
        eng.check_device()
        for i, (s, n) in enumerate(zip(seqs, lengths)):
            compare(torch.cat(got[i]), refs[i][n - 1:], dtype, f"{name}: wave {wave}, request {i} ({n} + {len(s) - n} tokens)")
        eng.cache.check()


def test_the_tolerances_refuse_planted_faults(root):
    """The comparison that the other tests pass is not passed by a plain statement with one fault."""
    cfg = FULL
    model, weights = make_model(root, cfg, 7, "float32")
    prompt = tokens(cfg, (120,), seed=3)[0]
    got = run_whole(engine_of(model), prompt)
    compare(got, P.forward(cfg, weights, prompt), "float32", "unplanted")

    def planted(change):
        bad = json.loads(json.dumps(cfg))
        w = dict(weights)
        change(bad, w)
        return P.forward(bad, w, prompt)

    def longer_window(bad, w):
        bad["layers"][0]["mixer"]["mask"]["size"] += 1

    def longer_latent_window(bad, w):
        bad["layers"][1]["mixer"]["mask"]["size"] += 1

    def one_kept_less(bad, w):
        bad["layers"][0]["mixer"]["mask"]["keep_first"] -= 1

    def plain_rotation(bad, w):
        del bad["layers"][3]["mixer"]["rot"]["scaling"]

    def other_ramp(bad, w):
        bad["layers"][1]["mixer"]["rot"]["scaling"]["original"] *= 4

    def less_mixing(bad, w):
        w["l3.mix.vmix"] = w["l3.mix.vmix"] * 0.9

    def no_hash(bad, w):
        bad["embedding"]["bigram"]["mul_prev"] += 1

    def first_row(bad, w):
        w["bigram"] = w["bigram"].clone()
        w["bigram"][-1] = w["bigram"][0]

    def no_gate(bad, w):
        w["l0.mix.g"] = w["l0.mix.g"] * 0.9

    def same_norm(bad, w):
        w["l0.norm2"], w["l0.norm2.b"] = w["l0.norm1"], w["l0.norm1.b"]
    for change in (longer_window, longer_latent_window, one_kept_less, plain_rotation, other_ramp, less_mixing, no_hash, first_row,
                   no_gate, same_norm):
        with pytest.raises(AssertionError):
            compare(got, planted(change), "float32", change.__name__)


def _deciding_key(root, cfg, edit, n, place, seen, dtype="float32"):
    """A prompt of `n` tokens whose last query matches the key of the token at `place` alone: a change of that token's VALUE
    must move the last row if `seen` and must not if not, in the prompt and from the cache."""
    model, weights = make_model(root, cfg, 13, dtype, edit, std=0.3)
    prompt = [min(t, 46) for t in tokens(cfg, (n,), seed=5)[0]]
    prompt[place], prompt[-1] = 48, 49
    eng = engine_of(model, max_tokens=64 * 16)
    ref = P.forward(cfg, weights, prompt, rounding(dtype))
    compare(run_whole(eng, prompt)[-1:], ref[-1:], dtype, "in a prompt")
    slot = eng.open_sequence()
    start = max(1, min(place - 2, n - 90))
    eng.step([(slot, prompt[:start])], want="none")
    for t in prompt[start:-1]:
        eng.step([(slot, [t])], want="none")
    compare(eng.step([(slot, prompt[-1:])], want="last"), ref[-1:], dtype, "from the cache")
    eng.check_device()
    eng.close_sequence(slot)
    moved = (P.forward(cfg, weights, prompt[:place] + [47] + prompt[place + 1:])[-1] - P.forward(cfg, weights, prompt)[-1]).abs().max()
    if seen:
        assert moved > 0.05, "the key does not matter in this test"
    else:
        assert moved < 1e-5, "the key is seen"


def _matched_attention(t):
    """Query head h's map is its key head's map behind a turn of the input by one place, and token 48's row is token 49's
    turned back: the query of 49 meets the key of 48 head on."""
    for n in ("l0.norm1", "l0.mix.q.norm", "l0.mix.k.norm"):
        t[n] = torch.ones_like(t[n])
    t["l0.norm1.b"] = torch.zeros_like(t["l0.norm1.b"])
    k = t["l0.mix.k"]
    t["l0.mix.q"] = torch.roll(k, 1, dims=1).repeat(2, 1).contiguous()
    t["embed"][48] = torch.roll(t["embed"][49], -1)


WINDOW, KEPT = 70, 66


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,place,seen", [
    (300, 300 - WINDOW, True), (300, 300 - WINDOW - 1, False),            # the window's far edge
    (300, KEPT - 1, True), (300, KEPT, False), (300, 0, True),            # the last kept position, the next one, the first
    (130, KEPT - 1, True), (130, KEPT, True), (138, KEPT, False),         # the window's edge just behind the kept ones
    (257, 256 - WINDOW + 1, True), (65, 0, True), (640, 640 - WINDOW, True), (640, 5, True), (640, 569, False)])
def test_a_key_at_the_edges_of_attention_decides(root, n, place, seen, dtype):
    cfg = config([layer("attention", attn(heads=2, kv_heads=1, dim=64, vdim=64, scale=1.5, rotation=None, window=WINDOW, keep=KEPT, v_mix=False))],
                 width=64, vocab=50, embed=1.0, bigram=None)
    _deciding_key(root, cfg, _matched_attention, n, place, seen, dtype)


def _matched_latent(t):
    t["l0.norm1"], t["l0.norm1.b"] = torch.ones_like(t["l0.norm1"]), torch.zeros_like(t["l0.norm1.b"])
    t["l0.mix.dkv.norm"], t["l0.mix.dq.norm"] = torch.ones_like(t["l0.mix.dkv.norm"]), torch.ones_like(t["l0.mix.dq.norm"])
    # keys = W_uk c with c the normed W_dkv h: the query's latent is W_dkv behind a turn of the input, its map W_uk
    t["l0.mix.dq"] = torch.roll(t["l0.mix.dkv"], 1, dims=1).contiguous()
    t["l0.mix.uq"] = (2.0 * t["l0.mix.uk"]).contiguous()
    t["embed"][48] = torch.roll(t["embed"][49], -1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,place,seen", [(300, 300 - 90, True), (300, 300 - 91, False), (640, 640 - 90, True), (640, 0, False),
                                          (90, 0, True), (91, 0, False)])
def test_a_key_at_the_edge_of_latent_attention_decides(root, n, place, seen, dtype):
    cfg = config([layer("latent_attention", latent(heads=2, dim=32, rot_dim=0, vdim=32, q_rank=64, kv_rank=64, scale=0.6, window=90))],
                 width=64, vocab=50, embed=1.0, bigram=None)
    _deciding_key(root, cfg, _matched_latent, n, place, seen, dtype)


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_a_far_key_decides_without_a_window(root, kind):
    if kind == "attention":
        m = attn(heads=2, kv_heads=1, dim=64, vdim=64, scale=1.5, rotation=None, window=None, v_mix=False)
    else:
        m = latent(heads=2, dim=32, rot_dim=0, vdim=32, q_rank=64, kv_rank=64, scale=0.6, window=None)
    cfg = config([layer(kind, m)], width=64, vocab=50, embed=1.0, bigram=None)
    _deciding_key(root, cfg, _matched_attention if kind == "attention" else _matched_latent, 800, 40, True)


def test_a_long_decode_goes_round_the_ring(root):
    """Hundreds of single tokens from the first one on: kept pages stay, the ring behind them is written again and again
    (also across a page that both hold), and the last rows still agree with the plain statement."""
    cfg = config([layer("attention", attn(heads=2, kv_heads=1, dim=32, vdim=32, window=100, keep=70, v_mix=False), dense(16)),
                  layer("latent_attention", latent(heads=2, dim=16, rot_dim=16, vdim=16, q_rank=16, kv_rank=32, window=65), None)], width=48, vocab=60)
    for dtype in ("float32", "bfloat16"):
        model, weights = make_model(root, cfg, 19, dtype)
        seq = tokens(cfg, (700,), seed=8)[0]
        ref = P.forward(cfg, weights, seq, rounding(dtype))
        eng = engine_of(model, max_tokens=64 * 12, max_sequences=1)
        slot = eng.open_sequence()
        rows = [eng.step([(slot, [t])], want="last") for t in seq]
        eng.check_device()
        compare(torch.cat(rows), ref, dtype, f"700 single tokens ({dtype})")
        held = [len(g.pages_of(slot)) for g in eng.cache.kv_groups]
        assert sorted(held) == [2, 4], held                        # two pages for the window of 65; two kept and two of a ring of 100


@pytest.mark.parametrize("name", sorted(WHOLE_MODELS))
def test_greedy_generation_through_the_session(root, name):
    """`generate` (the scheduler's batches, the sampler, steps fed from device memory) against greedy choices made
    from the plain implementation's logits."""
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 11, "float32")
    prompts = tokens(cfg, (1, 6, 70, 17), seed=4)
    session = model.session(max_tokens=64 * 10, max_sequences=3)
    got = session.generate(prompts, max_new_tokens=12, stop_ids=[])
    for p, g in zip(prompts, got):
        seq = list(p)
        for _ in range(12):
            logits = P.forward(cfg, weights, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if top2[0] - top2[1] < 1e-3:           # a close call proves nothing either way
                break
            seq.append(int(torch.argmax(logits)))
        n = len(seq) - len(p)
        assert g[:n] == seq[len(p):], f"{name}: prompt of {len(p)} tokens"


def test_command_line_and_presets(root, capsys):
    from inference_engine_rust_b200 import cli
    path = os.path.join(root, "cfg.json")
    with open(path, "w") as f:
        json.dump(ODD, f)
    out = os.path.join(root, "cli_model")
    assert cli.main(["random-model", "--config", path, "--seed", "2", "--out", out]) == 0
    capsys.readouterr()
    assert cli.main(["-m", out, "-n", "5", "--stop-token", "-1", "3 9 27"]) == 0
    ids = capsys.readouterr().out.split()
    assert len([t for t in ids if t.lstrip("-").isdigit()]) >= 5
    assert cli.main(["--random", "botulorn-tiny", "--seed", "1", "-n", "4", "--stop-token", "-1", "5 6"]) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(root, tmp_path, dtype):
    """bin/trace_run picks the architecture from config.json: requests whole, with their last tokens one by one, and
    as unequal batches whose shorter requests end earlier; every wanted row against the plain implementation."""
    from safetensors.torch import load_file, save_file
    from inference_engine_rust_b200 import write_random_model
    import test_gpu_trace_run as R
    cfg = TENSOR if dtype == "bfloat16" else FULL
    d = str(tmp_path / "model")
    write_random_model(d, cfg, seed=21, dtype=dtype, std=0.1)
    path = os.path.join(d, "model.safetensors")
    tensors = load_file(path)
    spread(tensors)
    save_file({k: v.contiguous() for k, v in tensors.items()}, path)
    weights = plain_weights(d)
    seqs = tokens(cfg, (90, 7, 231), seed=6)
    refs = [P.forward(cfg, weights, s, rounding(dtype)) for s in seqs]
    steps, wanted = [], []
    n = 0
    for i, s in enumerate(seqs):                       # whole; then all but five tokens and the rest one by one
        steps.append({"step": n, "entries": [{"id": f"w{i}", "tokens": s, "want": [0, len(s) - 1]}], "end": [f"w{i}"]})
        wanted.append((n, [refs[i][0], refs[i][-1]]))
        n += 1
        cut = max(1, len(s) - 5)
        steps.append({"step": n, "entries": [{"id": f"d{i}", "tokens": s[:cut], "want": []}], "end": []})
        n += 1
        for j in range(cut, len(s)):
            steps.append({"step": n, "entries": [{"id": f"d{i}", "tokens": [s[j]], "want": [0]}],
                          "end": [f"d{i}"] if j == len(s) - 1 else []})
            wanted.append((n, [refs[i][j]]))
            n += 1
    cuts = [len(s) - k for s, k in zip(seqs, (4, 2, 6))]       # together: unequal prompts, then decoded until each ends
    steps.append({"step": n, "entries": [{"id": f"t{i}", "tokens": s[:c], "want": [c - 1]} for i, (s, c) in enumerate(zip(seqs, cuts))],
                  "end": []})
    wanted.append((n, [refs[i][c - 1] for i, c in enumerate(cuts)]))
    n += 1
    pos = list(cuts)
    while any(p < len(s) for p, s in zip(pos, seqs)):
        live = [i for i, s in enumerate(seqs) if pos[i] < len(s)]
        steps.append({"step": n, "entries": [{"id": f"t{i}", "tokens": [seqs[i][pos[i]]], "want": [0]} for i in live],
                      "end": [f"t{i}" for i in live if pos[i] + 1 == len(seqs[i])]})
        wanted.append((n, [refs[i][pos[i]] for i in live]))
        for i in live:
            pos[i] += 1
        n += 1
    out = str(tmp_path / "out")
    R.replay(d, dtype, steps, out, max_tokens=64 * 9)
    for step, rows in wanted:
        compare(R.read(out, step, cfg["vocab"]), torch.stack(rows), dtype, f"step {step}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_short_prompt_steps_replayed_as_graphs(root, dtype):
    """Prompt steps of up to 512 tokens that want their last rows are captured into a CUDA graph from a shape bucket's
    second use on (padding tokens and padding sequences inside): same logits as the plain statement on every turn, with
    slots, pages and states used again in between, and the tokens after the prompt one by one."""
    cfg = WHOLE_MODELS["tensor" if dtype == "bfloat16" else "full"]
    model, weights = make_model(root, cfg, 17, dtype)
    # memory that the graphs' own buffers will be cut from holds NaN: rows of padding tokens that nobody writes show
    junk = [torch.full((16 << 20,), float("nan"), device="cuda") for _ in range(4)]
    del junk
    prompts = tokens(cfg, (3, 1, 63, 200, 140, 331), seed=8)
    want = [P.forward(cfg, weights, p + [5, 6], rounding(dtype)) for p in prompts]
    eng = engine_of(model, max_tokens=64 * 14, max_sequences=4)
    batches = [[1, 0], [3], [1, 2], [4, 0], [5], [0, 1], [3, 1], [2, 1], [5], [4]]
    for turn, batch in enumerate(batches * 2):
        slots = [eng.open_sequence() for _ in batch]
        got = eng.step([(s, prompts[i]) for s, i in zip(slots, batch)], want="last")
        more = eng.step([(s, [5]) for s in slots], want="last")
        last = eng.step([(s, [6]) for s in slots], want="last")
        eng.check_device()
        for k, i in enumerate(batch):
            n = len(prompts[i])
            compare(torch.cat([got[k:k + 1], more[k:k + 1], last[k:k + 1]]), want[i][n - 1:], dtype,
                    f"turn {turn}: a {n}-token prompt and two tokens more")
        for s in slots:
            eng.close_sequence(s)
    assert sum(1 for k in eng._graphs if isinstance(k, tuple) and k and k[0] == "prompt") >= 4, "few prompt steps were replayed"
