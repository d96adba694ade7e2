"""The Gidurax design in the engine against the plain statement of its equations (`tests/plain/gidurax_plain.py`): each mechanism
alone (kernels against one function of the plain statement, and one-layer models), then whole models under every way of cutting
the work: whole prompts, tokens one by one through the caches and states (of every pass of a repeated run), batches of unequal
requests through slots and pages that are used again, long decoding, short prompt steps replayed as graphs, and greedy generation
through the session.  Sizes differ from test to test (also sizes that are 1 or equal to one another), and where random weights would
hide a fault the weights are made so that it shows: one far key that decides, sinks that weigh as much as the keys, states that
hardly decay."""
import json
import math
import os

import pytest
import torch

from helpers import compare as compare_exactly, plain_weights, prompts_for
from plain import gidurax_plain as P

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


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=4):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attn(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.5, temp=(0.4, 9)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return "attention", m


def scan(inner=48, state=12, dt_rank=6, conv=4):
    return "mamba1", {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=5, top=2, identity=2, shared=32):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if identity is not None:
        out["router"]["identity"] = identity
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def layer(mixer, mlp=None):
    return {"type": mixer[0], "mixer": mixer[1], "mlp": mlp}


def config(layers, width=64, vocab=96, eps=1e-5, embed=3.0, mult=0.7, loop=None):
    cfg = {"architecture": "Gidurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
           "residual_mult": mult, "layers": json.loads(json.dumps(layers))}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


ALONE = {
    "attention": dict(layers=[layer(attn())]),
    "attention, equal sizes, one head": dict(layers=[layer(attn(heads=1, kv_heads=1, dim=16, vdim=16))]),
    "attention, wide values, no temperature": dict(layers=[layer(attn(heads=3, kv_heads=1, dim=8, vdim=40, temp=None))]),
    "attention, a temperature for every token": dict(layers=[layer(attn(heads=6, kv_heads=3, dim=64, vdim=64, scale=0.2, temp=(0.7, 1)))]),
    "attention, narrow values": dict(layers=[layer(attn(dim=32, vdim=8, temp=(-0.1, 64)))]),
    "delta": dict(layers=[layer(delta())]),
    "delta, equal sizes, two taps": dict(layers=[layer(delta(heads=2, kv_heads=2, dim=32, vdim=32, conv=2))]),
    "delta, one tap, one head": dict(layers=[layer(delta(heads=1, kv_heads=1, dim=8, vdim=20, conv=1))]),
    "delta, odd sizes": dict(layers=[layer(delta(heads=6, kv_heads=3, dim=10, vdim=7, conv=3))]),
    "delta, many taps, wide heads": dict(layers=[layer(delta(heads=2, kv_heads=1, dim=128, vdim=136, conv=7))]),
    "scan": dict(layers=[layer(scan())]),
    "scan, one state, one tap, rank one": dict(layers=[layer(scan(inner=40, state=1, dt_rank=1, conv=1))]),
    "scan, equal sizes": dict(layers=[layer(scan(inner=64, state=16, dt_rank=16, conv=2))]),
    "scan, odd sizes": dict(layers=[layer(scan(inner=37, state=11, dt_rank=7, conv=3))]),
    "scan, many states and taps": dict(layers=[layer(scan(inner=72, state=70, dt_rank=20, conv=9))]),
    "dense": dict(layers=[layer(attn(), dense())]),
    "experts": dict(layers=[layer(scan(), moe())]),
    "experts without a shared one or identities": dict(layers=[layer(scan(), moe(experts=3, top=1, identity=None, shared=None))]),
    "all experts chosen": dict(layers=[layer(attn(), moe(ff=7, experts=2, top=4, identity=2, shared=9))]),
    "a repeated layer": dict(layers=[layer(attn())], loop=(0, 1, 3)),
    "a repeated run in the middle": dict(layers=[layer(scan()), layer(delta(), dense()), layer(attn()), layer(scan())], loop=(1, 3, 2)),
    "a run of one pass": dict(layers=[layer(attn()), layer(scan())], loop=(1, 2, 1)),
    "no factor on the sublayers": dict(layers=[layer(delta(), dense())], mult=1.0, embed=1.0),
}

FULL = config([layer(scan(), dense()), layer(delta(), moe()), layer(attn(), dense(40)), layer(attn(heads=2, kv_heads=1, dim=32, vdim=16), moe(ff=16)),
               layer(scan(inner=56, state=20, dt_rank=9, conv=3), None), layer(delta(heads=6, kv_heads=3, dim=32, vdim=16, conv=3), moe(top=3))],
              loop=(1, 4, 2))
# sizes no kernel for the tensor cores takes: everything runs the plain kernels, also in bfloat16
ODD = config([layer(attn(heads=3, kv_heads=3, dim=10, vdim=7, temp=(0.5, 5)), dense(21)), layer(scan(inner=37, state=5, dt_rank=3, conv=2), moe(ff=9, shared=11)),
              layer(delta(heads=6, kv_heads=2, dim=14, vdim=9, conv=5), dense(13)), layer(attn(heads=6, kv_heads=2, dim=14, vdim=22, temp=None), moe(ff=5, shared=None))],
             width=50, vocab=75, eps=1e-4, embed=7.0, mult=0.9, loop=(2, 4, 3))
# sizes the tensor-core kernels take: tcgen05 prompt attention at head size 64, projections in whole runs of 64
TENSOR = config([layer(scan(inner=256, state=16, dt_rank=16), dense(256)), layer(delta(heads=4, kv_heads=4, dim=64, vdim=32), moe(ff=64, experts=6, shared=64)),
                 layer(attn(heads=8, kv_heads=2, dim=64, vdim=48, scale=0.3, temp=(0.2, 50)), dense(192)),
                 layer(attn(heads=4, kv_heads=4, dim=48, vdim=64, scale=0.3), moe(ff=64, experts=4, top=3, identity=1, shared=128))],
                width=128, vocab=160, embed=6.0, mult=0.5, loop=(0, 3, 2))
WIDE_HEADS = config([layer(attn(heads=2, kv_heads=1, dim=128, vdim=96, scale=0.2), dense(64)), layer(delta(heads=2, kv_heads=2, dim=128, vdim=128), None),
                     layer(attn(heads=2, kv_heads=1, dim=96, vdim=192, scale=0.2, temp=None), dense(32))], width=120, vocab=128, mult=1.0)
WHOLE_MODELS = {"full": FULL, "odd": ODD, "tensor": TENSOR, "wide_heads": WIDE_HEADS}


def spread(tensors):
    """Sinks about as heavy as the keys, step vectors and biases that matter, corrections that change choices, and channels and
    heads from hardly decaying to forgetting at once."""
    for name in sorted(tensors):
        t = tensors[name]
        if name.endswith(".sink"):
            tensors[name] = t * 20.0
        elif name == "loop.step":
            tensors[name] = t * 10.0
        elif name.endswith(".correction"):
            tensors[name] = t * 3.0
        elif name.endswith(".conv") or name.endswith(".conv.b") or name.endswith("shared.sg"):
            tensors[name] = t * 4.0
        elif name.endswith(".dt.b") or name.endswith(".dt_bias"):
            tensors[name] = (torch.linspace(-7.0, 1.0, t.numel()).to(t.dtype) + t)
        elif name.endswith(".A_log"):
            tensors[name] = t * 6.0


def settled(tensors):
    """`spread` for bfloat16: corrections so far apart that rounding decides no choice (the weights still follow the scores)."""
    spread(tensors)
    for i, name in enumerate(sorted(n for n in tensors if n.endswith(".correction"))):
        n = tensors[name].numel()
        tensors[name] = (torch.arange(n).add(2 * i + n - 2).remainder(n) * 1.5).to(tensors[name].dtype)


def edit_for(dtype):
    return settled if dtype == "bfloat16" else spread


def make_model(root, cfg, seed, dtype, edit=None, std=0.1):
    from safetensors.torch import load_file, save_file
    from inference_engine_rust_b200 import LoadedModel, write_random_model
    edit = edit or edit_for(dtype)
    d = os.path.join(root, f"m{abs(hash((json.dumps(cfg, sort_keys=True), seed, dtype, getattr(edit, '__name__', None)))) % 10 ** 9}")
    if not os.path.isdir(d):
        write_random_model(d, cfg, seed=seed, dtype=dtype, std=std)
        path = os.path.join(d, "model.safetensors")
        tensors = load_file(path)
        edit(tensors)
        save_file({k: v.contiguous() for k, v in tensors.items()}, path)
    return LoadedModel.load(d, dtype=dtype), plain_weights(d)


@pytest.fixture(scope="module")
def root(tmp_path_factory):
    return str(tmp_path_factory.mktemp("gidurax"))


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


@pytest.mark.parametrize("width", [8, 50, 128, 1000, 1536, 4096, 5120, 9000])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norms_on_both_sides_in_one_pass(width, dtype):
    """x += norm(y), y cleared, the next norm of the new x; and the head of a pass: x += e + step with the old rows kept."""
    b = B()
    g = torch.Generator().manual_seed(width)
    x, y, e = (torch.randn(7, width, generator=g) * s for s in (3.0, 0.4, 2.0))
    w, w2, step = (torch.randn(width, generator=g) for _ in range(3))
    dt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    tol = dict(rtol=1e-2, atol=1e-2) if dtype == "bfloat16" else dict(rtol=2e-5, atol=2e-5)
    out = torch.full((7, width), float("nan"), dtype=dt, device=DEV)
    xd, yd = x.to(DEV), y.to(DEV)
    b.add_normed(xd, yd, w.to(DEV), out, 6, 1e-5, stream(), w2=w2.to(DEV), eps2=1e-3)
    want = x[:6] + P.rms_norm(y[:6], w, 1e-5)
    torch.testing.assert_close(xd[:6].cpu(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(out[:6].float().cpu(), P.rms_norm(want, w2, 1e-3), **tol)
    assert (yd[:6] == 0).all() and torch.equal(yd[6].cpu(), y[6]) and torch.equal(xd[6].cpu(), x[6]) and out[6].isnan().all()
    for use_e in (False, True):
        xd, yd, keep = x.to(DEV), y.to(DEV), torch.zeros(7, width, device=DEV)
        b.rows_begin(xd, 7, stream(), e=e.to(DEV) if use_e else None, step=step.to(DEV), keep=keep, y=yd, out=out, w2=w2.to(DEV), eps2=1e-3)
        want = x + step + (e if use_e else 0.0)
        torch.testing.assert_close(xd.cpu(), want, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(out.float().cpu(), P.rms_norm(want, w2, 1e-3), **tol)
        assert torch.equal(keep.cpu(), x) and (yd == 0).all()
    xd = x.to(DEV)
    b.rows_begin(xd, 7, stream(), keep=keep.zero_())
    assert torch.equal(xd.cpu(), x) and torch.equal(keep.cpu(), x)


@pytest.mark.parametrize("M,N,K,F,E,odt", [
    (1, 200, 128, 40, 4, torch.bfloat16), (8, 4096, 512, 256, 15, torch.bfloat16), (16, 96, 64, 7, 5, torch.float32), (20, 320, 2048, 64, 4, torch.bfloat16),
    (70, 264, 192, 66, 3, torch.bfloat16), (200, 520, 1024, 64, 8, torch.float32), (300, 1000, 256, 100, 9, torch.bfloat16), (513, 264, 64, 24, 11, torch.bfloat16)])
def test_a_products_epilogue(M, N, K, F, E, odt):
    """Exact GELU and a factor per token and block of columns (blocks on and off the kernels' runs of 4 and 16 columns, a last
    block of another width) on the kernels for few and many tokens, with and without split K, and as a kernel of its own."""
    b = B()
    g = torch.Generator().manual_seed(M + N)
    x, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) * K ** -0.5 * 2).bfloat16()
    s = torch.rand(M, E + 1, generator=g) * (torch.rand(M, E + 1, generator=g) < 0.7)
    blk = torch.clamp(torch.arange(N) // F, max=E)
    z = x.float() @ w.float().t()
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    xd, wd, sd = x.to(DEV), w.to(DEV), s.to(DEV)
    for act in ("gelu", "none"):
        ep = b.epilogue(act, scale=sd, blocks=E, block_cols=F)
        want = (P.gelu_erf(z) if act == "gelu" else z) * s[:, blk]
        runs = [lambda o: b.gemm_tc(xd, wd, o, M, b.GEMM_STORE, err, stream(), epilogue=ep)]
        if M <= 16:
            runs.append(lambda o: b.gemm_rows(xd, wd, o, M, b.GEMM_STORE, err, stream(), epilogue=ep))
        if M > 256:
            runs.append(lambda o: b.gemm_tc(xd, wd, o, M, b.GEMM_STORE, err, stream(), force_bt=256, epilogue=ep))
        for run in runs:
            out = torch.full((M, N), float("nan"), dtype=odt, device=DEV)
            assert run(out)
            torch.testing.assert_close(out.float().cpu(), want, rtol=1e-2, atol=1e-2)
        alone = z.to(DEV)
        b.epilogue_rows(alone, M, ep, stream())
        torch.testing.assert_close(alone.cpu(), want, rtol=1e-5, atol=1e-5)
    assert int(err) == 0


@pytest.mark.parametrize("E,identity,top", [(1, 0, 1), (5, 2, 2), (6, 3, 9), (40, 0, 4), (70, 5, 8)])
@pytest.mark.parametrize("by_output", [False, True])
def test_routing_with_plain_scores(E, identity, top, by_output):
    """Weights are the chosen scores as they are; the shared expert's gate beside them; identities added to the residual."""
    b = B()
    g = torch.Generator().manual_seed(E + top)
    T, N, H = 19, E + identity, 68
    z = torch.randn(T, N + 1, generator=g) * 2
    corr = torch.randn(N, generator=g) * 0.2
    x = torch.randn(T, H, generator=g).bfloat16()
    idx, w = P.route(z[:, :N], corr, top)
    wt, wid, res = torch.zeros(T, E + 1), torch.zeros(T), torch.randn(T, H, generator=g)
    for t in range(T):
        for e, a in zip(idx[t].tolist(), w[t].tolist()):
            if e < E:
                wt[t, e] += a
            else:
                wid[t] += a
    wt[:, E] = torch.sigmoid(z[:, N])
    zd = (z.t().contiguous() if by_output else z).to(DEV)
    gw, gid, gi, gv = torch.full((T, E + 1), 9.0, device=DEV), torch.empty(T, device=DEV), torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    rd = res.to(DEV)
    b.router_grouped(zd, corr.to(DEV), T, E, N, top, 1, 1, gw, gid, gi, gv, stream(), by_output=by_output, renormalize=False, shared_gate=True,
                     x=x.to(DEV), residual=rd)
    torch.testing.assert_close(gw.cpu(), wt, rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(gid.cpu(), wid, rtol=1e-5, atol=1e-6)
    torch.testing.assert_close(rd.cpu(), res + wid[:, None] * x.float(), rtol=1e-5, atol=1e-5)
    assert torch.equal(gi.cpu().long(), idx)


@pytest.mark.parametrize("C,N,K", [(36, 1, 4), (128, 16, 4), (300, 12, 3), (37, 11, 2), (64, 33, 1), (8, 64, 6), (40, 130, 16), (24, 256, 4), (96, 24, 5)])
@pytest.mark.parametrize("lanes", [None, 4, 8, 16, 32])
def test_selective_convolution_and_scan(monkeypatch, C, N, K, lanes):
    """Both kernels over unequal prompts with padding between, then single tokens, in slots that other sequences used before;
    every number of lanes per channel; states that hardly decay and states that forget at once."""
    if lanes is not None:
        monkeypatch.setenv("IERT_SCAN_LANES", str(lanes))
    b = B()
    g = torch.Generator().manual_seed(C + N)
    lens = {2: 77, 0: 3, 3: 33}
    ld, P_ = 2 * C + 4, N * 2 + 8
    A = -torch.exp(torch.randn(C, N, generator=g))
    D, cb, db = torch.randn(C, generator=g), torch.randn(C, generator=g), torch.linspace(-8, 2, C)
    taps = torch.randn(C, K, generator=g)
    xz = {s: torch.randn(n, ld, generator=g) for s, n in lens.items()}
    bc = {s: torch.randn(n, P_, generator=g) for s, n in lens.items()}
    raw = {s: torch.randn(n, C, generator=g) for s, n in lens.items()}
    for dtype in (torch.float32, torch.bfloat16):
        rnd = P.bf16 if dtype == torch.bfloat16 else P.exact
        want_u = {s: rnd(P.silu(P.short_conv(rnd(xz[s][:, :C]), taps, cb))) for s in lens}
        want = {}
        for s in lens:
            y, S = P.selective_scan(want_u[s], P.softplus(raw[s] + db), A, rnd(bc[s][:, :N]), rnd(bc[s][:, N:2 * N]), D)
            want[s] = (y * P.silu(rnd(xz[s][:, C:2 * C])), S)
        state = torch.full((4, C * N + K * C), float("nan"), device=DEV)
        A2 = (A * (math.log2(math.e) if dtype == torch.bfloat16 else 1.0)).to(DEV)
        for s in lens:
            state[s].zero_()
        pos = {s: 0 for s in lens}
        for plan, pad in (({2: 70, 0: 1, 3: 33}, 5), ({0: 1, 2: 1}, 0), ({2: 1, 0: 1}, 0), ({2: 1}, 0)):
            slots = list(plan)
            one = all(pos[s] > 0 and plan[s] == 1 for s in slots)
            bt = Batch([plan[s] for s in slots], [pos[s] for s in slots], slots, pad=pad)

            def rows(src, width):
                return torch.cat([src[s][pos[s]:pos[s] + plan[s]] for s in slots] + [torch.full((pad, width), float("nan"))]).to(DEV)
            xd, pd, dd = rows(xz, ld).to(dtype), rows(bc, P_).to(dtype), rows(raw, C)
            u, out = (torch.full((bt.n_tokens, C), float("nan"), dtype=dtype, device=DEV) for _ in range(2))
            b.selective_conv(xd, taps.t().contiguous().to(DEV), cb.to(DEV), state, C * N, u, C, K, bt.view, stream())
            b.selective_scan(u, dd, db.to(DEV), pd, xd[:, C:], A2, D.to(DEV), state, 0, out, C, N, one, bt.view, stream())
            at = 0
            tol = dict(rtol=2e-2, atol=4e-2) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=1e-4)
            for s in slots:
                n = plan[s]
                ref = want[s][0][pos[s]:pos[s] + n]
                torch.testing.assert_close(u[at:at + n].float().cpu(), want_u[s][pos[s]:pos[s] + n], rtol=1e-2 if dtype == torch.bfloat16 else 1e-5, atol=1e-2 if dtype == torch.bfloat16 else 1e-5)
                got = out[at:at + n].float().cpu()
                scale = ref.abs().max()
                torch.testing.assert_close(got / scale, ref / scale, **tol)
                at += n
                pos[s] += n
            assert out[at:].isnan().all()
        assert state[1].isnan().all()
        for s in (0, 3):
            if pos[s] == lens[s]:
                S = state[s, :C * N].view(C, N).cpu()
                torch.testing.assert_close(S / want[s][1].abs().max(), want[s][1] / want[s][1].abs().max(), rtol=2e-2 if dtype == torch.bfloat16 else 1e-4, atol=2e-3 if dtype == torch.bfloat16 else 1e-5)


@pytest.mark.parametrize("D", [48, 64, 128, 192])
@pytest.mark.parametrize("softness", [1.0, 4.0])
def test_prompt_attention_with_sinks(D, softness):
    """The tensor-core prompt kernels and the plain one with a sink per head, from negligible to dominant, on packed prompts."""
    b = B()
    g = torch.Generator().manual_seed(D)
    H, G, lens = 4, 2, [1, 300, 65, 190]
    T = sum(lens)
    qkv = torch.randn(T, (H + 2 * G) * D, generator=g)
    qkv[:, :H * D] *= softness
    qkv = qkv.to(torch.bfloat16)
    bt = Batch(lens, [0] * 4, [3, 1, 0, 2])
    scale, sink = D ** -0.5, torch.tensor([-20.0, 0.0, 3.0, 9.0])
    want = torch.cat([P.sink_attention(*(x.float() for x in qkv[a:a + n].view(n, H + 2 * G, D).split([H, G, G], dim=1)), scale, sink).reshape(n, H * D)
                      for a, n in zip([0, 1, 301, 366], lens)])
    qd, sd = qkv.to(DEV), sink.to(DEV)
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    for legacy in (False, True):
        out = torch.full((T, H * D), float("nan"), dtype=torch.bfloat16, device=DEV)
        assert b.attention_prefill(qd, out, bt.view, H, G, D, 0, scale, max(lens), stream(), err=err, legacy=legacy, sink=sd)
        torch.testing.assert_close(out.float().cpu(), want, rtol=2e-2, atol=2e-2)
    own = b.KvView(k=None, v=None, page_table=None, table_width=0, ring_pages=1, page_tokens=1, n_pages=0, kv_heads=G, head_dim=D, dtype=b.F32, window=0, chunk=0, keep=0)
    full = torch.empty(T, H * D, device=DEV)
    b.attention_plain(qd.float(), full, bt.view, own, H, scale, False, err, stream(), sink=sd)
    torch.testing.assert_close(full.cpu(), want, rtol=1e-4, atol=1e-4)
    assert int(err) == 0


@pytest.mark.parametrize("dim,vdim,every", [(64, 64, 64), (16, 24, 7), (10, 6, 1), (128, 96, 100)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_query_temperature(dim, vdim, every, dtype):
    """Positions around every step of the logarithm, far ones too; keys and values are left as they are."""
    b = B()
    g = torch.Generator().manual_seed(dim)
    H, G, coef = 3, 1, 0.6
    D = max(dim, vdim) if dtype == "float32" else -(-max(dim, vdim) // 16) * 16
    dt = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    wq, wk = torch.rand(dim, generator=g) + 0.5, torch.rand(dim, generator=g) + 0.5
    for pos0 in (0, every - 1, 7 * every - 3 if every > 3 else 20, 100000):
        T = 6
        n = (H + G) * dim + G * vdim
        proj = torch.randn(T, n + (-n % 4), generator=g)
        cache = torch.zeros(2, 1, G, 64, D, dtype=dt, device=DEV)
        table = torch.zeros(1, 1, dtype=torch.int32, device=DEV)
        kvv = b.KvView(k=cache[0].data_ptr(), v=cache[1].data_ptr(), page_table=table.data_ptr(), table_width=1, ring_pages=1, page_tokens=64,
                       n_pages=1, kv_heads=G, head_dim=D, dtype=b.dtype_code(dt), window=0, chunk=0)
        bt = Batch([T], [pos0], [0])
        qkv = torch.full((T, (H + 2 * G) * D), float("nan"), dtype=dt, device=DEV)
        err = torch.zeros(1, dtype=torch.int32, device=DEV)
        b.qkv_prep(proj.to(DEV), None, qkv, bt.view, kvv, H, dim, vdim, None, 0, b.PAIR_HALF, wq.to(DEV), wk.to(DEV), 1e-5, False, err, stream(),
                   temp_coef=coef, temp_every=float(every))
        got = qkv.float().cpu().view(T, H + 2 * G, D)
        f = P.temperature(torch.arange(pos0, pos0 + T), coef, every)[:, None, None]
        tol = dict(rtol=1e-2, atol=1e-2) if dtype == "bfloat16" else dict(rtol=2e-5, atol=2e-5)
        torch.testing.assert_close(got[:, :H, :dim], P.rms_norm(proj[:, :H * dim].view(T, H, dim), wq, 1e-5) * f, **tol)
        torch.testing.assert_close(got[:, H:H + G, :dim], P.rms_norm(proj[:, H * dim:(H + G) * dim].view(T, G, dim), wk, 1e-5), **tol)
        torch.testing.assert_close(got[:, H + G:, :vdim], proj[:, (H + G) * dim:n].view(T, G, vdim), **tol)


# ---------------------------------------------------------------------------------------
# models


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(root, name, dtype):
    """One to four layers: prompts, and the same tokens partly one by one (over page borders)."""
    cfg = config(**ALONE[name])
    model, weights = make_model(root, cfg, 3, dtype)
    eng = engine_of(model)
    for prompt, first in zip(tokens(cfg, (1, 2, 150), seed=1), (1, 1, 50)):
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
    assert len(got) == len(want) == 9
    for i, (g, w) in enumerate(zip(got, want)):
        compare(g, w, "float32", f"residual after layer run {i}")


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
    """A prompt in one step, then single tokens over page borders; also from the very first token on and from a prompt of two."""
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 8, dtype)
    eng = engine_of(model)
    for first, total in ((1, 30), (2, 75), (61, 61 + 80), (300, 340)):
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
    prompt = tokens(cfg, (90,), seed=3)[0]
    got = run_whole(engine_of(model), prompt)
    compare(got, P.forward(cfg, weights, prompt), "float32", "unplanted")

    def planted(change):
        bad = json.loads(json.dumps(cfg))
        w = dict(weights)
        change(bad, w)
        return P.forward(bad, w, prompt)

    def scaled(name, f):
        def change(bad, w):
            w[name] = w[name] * f
        change.__name__ = f"{name} times {f}"
        return change

    def no_temperature(bad, w):
        del bad["layers"][2]["mixer"]["q_temp"]

    def later_temperature(bad, w):
        bad["layers"][2]["mixer"]["q_temp"]["every"] += 1

    def one_pass_less(bad, w):
        bad["loop"]["times"] -= 1

    def steps_in_the_other_order(bad, w):
        w["loop.step"] = w["loop.step"].flip(0)

    def no_identities(bad, w):
        w["l1.mlp.router"] = w["l1.mlp.router"].clone()
        w["l1.mlp.router"][5:] = 0.0

    def same_norms(bad, w):
        w["l0.norm1b"] = w["l0.norm1"]

    def no_sink(bad, w):
        w["l2.mix.sink"] = w["l2.mix.sink"] - 50.0
    for change in (no_temperature, later_temperature, one_pass_less, steps_in_the_other_order, no_identities, same_norms, no_sink,
                   scaled("l1.mix.k.conv", 0.9), scaled("l1.mix.dt_bias", 0.9), scaled("l0.mix.dt.b", 0.9), scaled("l0.mix.A_log", 0.9),
                   scaled("l0.mix.D", 0.9), scaled("l1.mlp.correction", 0.5), scaled("l1.mlp.shared.sg", 0.5), scaled("l1.mix.b", 0.9)):
        with pytest.raises(AssertionError):
            compare(got, planted(change), "float32", change.__name__)


def _matched(t):
    """Query head h's map is its key head's map behind a turn of the input by one place, and token 48's row is token 49's
    turned back: the query of 49 meets the key of 48 head on.  The sinks are weak beside that score and strong beside the others."""
    for n in ("l0.norm1", "l0.mix.q.norm", "l0.mix.k.norm"):
        t[n] = torch.ones_like(t[n])
    t["l0.mix.q"] = torch.roll(t["l0.mix.k"], 1, dims=1).repeat(2, 1).contiguous()
    t["l0.mix.sink"] = torch.full_like(t["l0.mix.sink"], 20.0)
    t["embed"][48] = torch.roll(t["embed"][49], -1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,place", [(65, 0), (66, 1), (129, 63), (129, 64), (200, 127), (200, 128), (800, 3), (800, 447), (800, 798)])
def test_one_far_key_decides(root, n, place, dtype):
    """First tokens, page borders and far keys, in a prompt and from the cache; the token at `place` matters to the last row."""
    cfg = config([layer(attn(heads=2, kv_heads=1, dim=64, vdim=64, scale=0.6, temp=(0.1, 50)))], width=64, vocab=50, embed=1.0)
    model, weights = make_model(root, cfg, 13, dtype, _matched, std=0.3)
    prompt = [min(t, 46) for t in tokens(cfg, (n,), seed=5)[0]]
    prompt[place], prompt[-1] = 48, 49
    eng = engine_of(model)
    ref = P.forward(cfg, weights, prompt, rounding(dtype))
    compare(run_whole(eng, prompt)[-1:], ref[-1:], dtype, "in a prompt")
    slot = eng.open_sequence()
    start = max(1, min(place - 2, n - 90))
    eng.step([(slot, prompt[:start])], want="none")
    for t in prompt[start:-1]:
        eng.step([(slot, [t])], want="none")
    compare(eng.step([(slot, prompt[-1:])], want="last"), ref[-1:], dtype, "from the cache")
    eng.check_device()
    moved = (P.forward(cfg, weights, prompt[:place] + [47] + prompt[place + 1:])[-1] - P.forward(cfg, weights, prompt)[-1]).abs().max()
    assert moved > 0.05, "the key does not matter in this test"


def _remembering(t):
    """States that hardly decay."""
    for n in t:
        if n.endswith("dt.b") or n.endswith("dt_bias"):
            t[n] = torch.full_like(t[n], -9.0)
        elif n.endswith(".A_log"):
            t[n] = torch.full_like(t[n], -2.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["delta", "scan"])
def test_a_state_carries_the_first_token_far(root, kind, dtype):
    """Hundreds of tokens later the first one still moves the logits, in prompts of several chunks and after single tokens."""
    cfg = config([layer(delta(heads=2, kv_heads=1, dim=32, vdim=32) if kind == "delta" else scan(inner=64, state=16, dt_rank=4))],
                 width=48, vocab=60, embed=1.0)
    model, weights = make_model(root, cfg, 23, dtype, _remembering, std=0.3)
    seq = tokens(cfg, (420,), seed=4)[0]
    ref = P.forward(cfg, weights, seq, rounding(dtype))
    moved = (P.forward(cfg, weights, [(seq[0] + 7) % 60] + seq[1:])[-1] - P.forward(cfg, weights, seq)[-1]).abs().max()
    assert moved > 2e-3, f"the first token is forgotten in this test ({moved})"
    eng = engine_of(model)
    compare(run_whole(eng, seq), ref, dtype, "in a prompt")
    slot = eng.open_sequence()
    rows = [eng.step([(slot, seq[:250])], want="all")] + [eng.step([(slot, [t])], want="last") for t in seq[250:]]
    eng.check_device()
    compare(torch.cat(rows), ref, dtype, "250 tokens and 170 one by one")


def test_a_long_decode(root):
    """Hundreds of single tokens from the first one on, through every pass's own cache and state."""
    cfg = config([layer(attn(heads=2, kv_heads=1, dim=32, vdim=32), dense(16)), layer(scan(inner=32, state=8, dt_rank=4), None),
                  layer(delta(heads=2, kv_heads=2, dim=16, vdim=16), moe(ff=8, shared=8))], width=48, vocab=60, loop=(0, 2, 2))
    for dtype in ("float32", "bfloat16"):
        model, weights = make_model(root, cfg, 19, dtype)
        seq = tokens(cfg, (600,), seed=8)[0]
        ref = P.forward(cfg, weights, seq, rounding(dtype))
        eng = engine_of(model, max_tokens=64 * 12, max_sequences=1)
        slot = eng.open_sequence()
        rows = [eng.step([(slot, [t])], want="last") for t in seq]
        eng.check_device()
        compare(torch.cat(rows), ref, dtype, f"600 single tokens ({dtype})")


@pytest.mark.parametrize("name", sorted(WHOLE_MODELS))
def test_greedy_generation_through_the_session(root, name):
    """`generate` (the scheduler's batches, the sampler, steps fed from device memory) against greedy choices made
    from the plain implementation's logits."""
    cfg = WHOLE_MODELS[name]
    model, weights = make_model(root, cfg, 11, "float32")
    prompts = tokens(cfg, (1, 6, 70, 17), seed=4)
    got = model.session(max_tokens=64 * 10, max_sequences=3).generate(prompts, max_new_tokens=12, stop_ids=[])
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
    assert cli.main(["--random", "gidurax-tiny", "--seed", "1", "-n", "4", "--stop-token", "-1", "5 6"]) == 0


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
    edit_for(dtype)(tensors)
    save_file({k: v.contiguous() for k, v in tensors.items()}, path)
    weights = plain_weights(d)
    seqs = tokens(cfg, (90, 7, 231), seed=6)
    refs = [P.forward(cfg, weights, s, rounding(dtype)) for s in seqs]
    steps, wanted, n = [], [], 0
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
