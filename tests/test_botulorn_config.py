"""The Botulorn configuration on the CPU: keys read and defaults, refusals that name the key, the spec it builds (tensor
names, parts and their constants, which layer's values are mixed into which), the random folder, a cache or state entry
per layer and for the pair embedding, pages of kept first positions, stretched rotations, and the plain statement's pieces
against hand-worked numbers."""
import json
import math

import pytest
import torch

from inference_engine_rust_b200.cache import Cache, KVRequest, StateRequest
from inference_engine_rust_b200.config import ConfigError, PartSpec, config_from_dict, preset, spec_of
from inference_engine_rust_b200.engine.model import Model
from inference_engine_rust_b200.parts.base import Runtime
from inference_engine_rust_b200.parts.rope import RotaryEncoding, yarn_rates
from plain import botulorn_plain as P

STRETCH = {"factor": 5.0, "original": 100, "fast": 16.0, "slow": 2.0}
ATT = {"heads": 6, "kv_heads": 2, "dim": 16, "vdim": 20, "scale": 0.3, "mask": {"size": 70, "keep_first": 3}, "v_mix": True,
       "rot": {"base": 1000.0, "dims": 8, "scaling": STRETCH}}
LAT = {"heads": 5, "dim": 12, "rot_dim": 4, "vdim": 22, "q_rank": 14, "kv_rank": 24, "scale": 0.25, "mask": {"size": 33},
       "rot": {"base": 500.0, "dims": 4}}
MLP = {"kind": "dense", "ff": 28}


def cfg(**top):
    layers = [{"type": "attention", "mixer": dict(ATT, v_mix=False, vdim=8), "mlp": MLP},
              {"type": "attention", "mixer": ATT, "mlp": None},
              {"type": "latent_attention", "mixer": LAT, "mlp": MLP},
              {"type": "attention", "mixer": dict(ATT, heads=2, dim=18), "mlp": MLP}]
    d = {"architecture": "Botulorn", "vocab": 90, "width": 56, "norm": {"eps": 1e-6},
         "embedding": {"scale": 5.0, "bigram": {"buckets": 41, "mul_prev": 3, "mul_cur": 8}}, "layers": json.loads(json.dumps(layers))}
    d.update(top)
    return d


def model_of(raw):
    return Model(spec_of(config_from_dict(raw)), Runtime(dtype=torch.float32, device="cpu"))


def test_spec_of_a_configuration():
    c = config_from_dict(cfg())
    spec = spec_of(c)
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3] and spec.embedding_scale == 5.0
    assert spec.lm_head_name == "head" and spec.head.kind == "linear" and spec.final_norm.kind == "layernorm"
    assert all(l.block.kind == "two_norms" and l.norm.kind == "layernorm" and l.norm["eps"] == 1e-6 for l in spec.layers)
    a = spec.layers[1].mixer
    assert a.kind == "gated_attention" and (a["window"], a["keep"], a["v_dim"], a["gate"], a["qk_norm"]) == (70, 3, 20, "head", "head")
    assert a["position"]["pairing"] == "half" and a["position"]["rotary_dim"] == 8 and a["position"]["yarn"]["factor"] == 5.0
    assert [l.mixer.get("v_mix") for l in spec.layers] == [None, "source", None, "mix"]
    m = spec.layers[2].mixer
    assert m.kind == "latent_attention" and (m["q_rank"], m["rot_dim"], m["window"], m["gate"], m["sink"]) == (14, 4, 33, None, False)
    assert m["position"]["yarn"] is None and spec.layers[1].ffn is None
    f = spec.layers[0].ffn
    assert f.kind == "swiglu" and f["activation"] == "gelu_tanh" and f["intermediate_size"] == 28
    (part, prefix), = spec.inputs
    assert part.kind == "pair_embedding" and prefix == "" and (part["buckets"], part["mul_prev"], part["mul_cur"]) == (41, 3, 8)
    model = model_of(cfg())
    shapes = {k: tuple(v.shape) for k, v in model.expected_tensors().items()}
    names = ({"embed", "bigram", "head", "final.norm", "final.norm.b"} | {f"l{i}.norm1{b}" for i in range(4) for b in ("", ".b")}
             | {f"l{i}.norm2{b}" for i in (0, 2, 3) for b in ("", ".b")} | {f"l{i}.mlp.{n}" for i in (0, 2, 3) for n in ("gate", "up", "down")}
             | {f"l{i}.mix.{n}" for i in (0, 1, 3) for n in ("q", "k", "v", "q.norm", "k.norm", "g", "o")} | {"l1.mix.vmix", "l3.mix.vmix"}
             | {f"l2.mix.{n}" for n in ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o")})
    assert set(shapes) == names
    assert shapes["bigram"] == (42, 56) and shapes["l1.mix.vmix"] == () and shapes["l1.mix.g"] == (6, 56) and shapes["l1.mix.v"] == (40, 56)
    assert shapes["l1.mix.o"] == (56, 120) and shapes["l1.mix.q.norm"] == (16,) and shapes["l3.mix.q"] == (36, 56)
    assert shapes["l2.mix.dq"] == (14, 56) and shapes["l2.mix.uq"] == (80, 14) and shapes["l2.mix.dkv"] == (28, 56)
    assert shapes["l2.mix.uk"] == (60, 24) and shapes["l2.mix.uv"] == (110, 24) and shapes["l2.mix.o"] == (56, 110)
    reqs = model.cache_requests()
    assert sorted(reqs) == [-1, 0, 1, 2, 3] and reqs[-1] == StateRequest((1,), torch.int32)
    assert reqs[1] == KVRequest(2, 20, 70, keep=3) and reqs[2] == KVRequest(1, 28, 33, values=False)
    assert config_from_dict(c.to_dict()) == c and model.graph_safe()


def test_defaults():
    raw = cfg()
    del raw["embedding"]
    for key in ("mask", "rot", "v_mix"):
        del raw["layers"][1]["mixer"][key]
    del raw["layers"][1]["mixer"]["vdim"], raw["layers"][0]["mixer"]["mask"]["keep_first"], raw["layers"][2]["mixer"]["mask"]
    c = config_from_dict(raw)
    assert c.embedding_scale == 1.0 and c.bigram is None
    spec = spec_of(c)
    assert spec.inputs == () and spec.layers[1].mixer["window"] is None and spec.layers[1].mixer["v_dim"] == 16
    assert spec.layers[1].mixer["position"]["rotary_dim"] == 0 and spec.layers[0].mixer["keep"] == 0
    assert [l.mixer.get("v_mix") for l in spec.layers] == [None, None, None, "source"]
    reqs = model_of(raw).cache_requests()
    assert sorted(reqs) == [0, 1, 2, 3] and reqs[1].reach is None and reqs[2].reach is None
    assert config_from_dict(c.to_dict()) == c


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"), (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 1, "type"), "mlstm", "type"),
    (("layers", 0, "mixer", "mask", "size"), 0, "size"), (("layers", 0, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"), (("norm",), None, "eps"), (("layers", 0, "mixer", "scale"), None, "scale"),
    (("layers", 0, "mlp", "ff"), None, "ff"), (("layers", 2, "mixer", "rot", "dims"), 2, "rot_dim"), (("layers", 2, "mixer", "rot_dim"), 3, "rot_dim"),
    (("layers", 2, "mixer", "kv_rank"), None, "kv_rank"), (("layers", 2, "mixer", "q_rank"), 0, "q_rank"), (("layers", 2, "mixer", "rot"), None, "rot"),
    (("layers", 0, "mixer", "v_mix"), 1, "v_mix"), (("layers", 3, "mixer", "vdim"), 8, "v_mix"), (("layers", 3, "mixer", "kv_heads"), 1, "v_mix"),
    (("layers", 1, "mixer", "rot", "scaling", "slow"), None, "slow"), (("layers", 1, "mixer", "rot", "base"), 1.0, "base"),
    (("embedding", "bigram", "buckets"), 0, "buckets"), (("embedding", "bigram", "mul_cur"), None, "mul_cur"),
])
def test_refusals_name_the_key(path, value, word):
    raw = cfg()
    at = raw
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        config_from_dict(raw)
    assert word in str(e.value)


def test_presets_and_random_folder(tmp_path):
    from inference_engine_rust_b200 import write_random_model
    from inference_engine_rust_b200.weights import TensorSource
    for name in ("botulorn-tiny", "botulorn-7b-sizes", "botulorn-12b-sizes"):
        spec_of(config_from_dict(preset(name)))
    d = str(tmp_path / "m")
    write_random_model(d, preset("botulorn-tiny"), seed=3, dtype="bfloat16")
    src = TensorSource(d)
    assert {"head", "bigram", "l1.mix.vmix", "l0.mix.dq.norm", "l3.norm2.b"} <= set(src.names())
    assert tuple(src.describe("l2.mix.vmix")[1]) == () and src.get("l2.mix.vmix").dtype == torch.bfloat16


def test_pages_of_kept_first_positions():
    """A ring of two pages behind two kept ones: whatever a sequence's length, it holds at most four pages, all of which go
    back when it ends; a table that needs no ring keeps none apart."""
    req = KVRequest(1, 4, 100, keep=70)
    c = Cache({0: req, 1: KVRequest(1, 4, 100)}, max_tokens=64 * 40, max_seq_len=64 * 20, max_sequences=3, dtype=torch.float32, device="cpu")
    g, plain = c.kv_groups
    assert (g.keep_pages, g.ring_pages, g.ring_capacity) == (2, 4, 128) and (plain.keep_pages, plain.ring_pages) == (0, 2)
    slot = c.open_sequence()
    held = []
    for n in (1, 64, 65, 129, 200, 256, 257, 900, 1280):
        c.reserve(slot, n)
        c.seq_lens[slot] = n
        held.append(len(g.pages_of(slot)))
    assert held == [1, 1, 2, 3, 4, 4, 4, 4, 4]
    assert c.kv_bytes_read([slot]) == (170 + 100) * 2 * 4 * 4
    c.check()
    c.close_sequence(slot)
    c.check()
    assert not g.pages.held()
    short = Cache({0: req}, max_tokens=64 * 3, max_seq_len=64 * 3, max_sequences=1, dtype=torch.float32, device="cpu").kv_groups[0]
    assert (short.keep_pages, short.ring_pages) == (0, 3)


def test_stretched_rotations():
    for dims, base, s in ((8, 1000.0, STRETCH), (32, 50000.0, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
                          (2, 10.0, {"factor": 2.0, "original": 4, "fast": 1.0, "slow": 1.0})):
        want, m = P.turn_rates({"dims": dims, "base": base, "scaling": s})
        rates, mul = yarn_rates(base, dims, **s)
        assert torch.allclose(rates, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and mul == m
    # 16 turns in 100 positions at pair 8 ln(100 / (32 pi)) / (2 ln 1000) < 0, two turns at pair 1.2: pair 0 keeps its rate, pair 1
    # lies half way, the pairs from 2 on are divided by 5
    rates, mul = yarn_rates(1000.0, 8, **STRETCH)
    f = [1000.0 ** (-i / 4) for i in range(4)]
    want = [f[0], f[1] * (0.5 + 0.1), f[2] / 5, f[3] / 5]
    assert torch.allclose(rates, torch.tensor(want, dtype=torch.float64), rtol=1e-12) and abs(mul - (1 + 0.1 * math.log(5.0))) < 1e-12
    part = RotaryEncoding(PartSpec("rope", {"theta": 1000.0, "rotary_dim": 8, "pairing": "half", "yarn": STRETCH}), 16,
                          Runtime(dtype=torch.float32, device="cpu"))
    assert part.rotary_constants() is None and part.scaled_rotary_constants()[3] == mul
    with pytest.raises(ValueError):
        RotaryEncoding(PartSpec("rope", {"theta": 10.0, "rotary_dim": 2, "yarn": STRETCH, "freq_factors": [1.0]}), 4,
                       Runtime(dtype=torch.float32, device="cpu"))


def test_the_plain_pieces_by_hand():
    # two pairs (0, 2) and (1, 3) turn, the rest of the head passes; factor 1 without scaling
    v = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0, 6.0]]]).repeat(3, 1, 1)
    got = P.rotate(v, {"dims": 4, "base": 100.0})
    for p in range(3):
        a0, a1 = p * 1.0, p * 0.1
        want = [math.cos(a0), -2 * math.sin(a1), math.sin(a0), 2 * math.cos(a1), 5.0, 6.0]
        assert torch.allclose(got[p, 0], torch.tensor(want), atol=1e-6)
    # a window of 3 and one kept first position
    sees = P.visible(7, 3, 1)
    assert [j for j in range(7) if sees[5, j]] == [0, 3, 4, 5] and [j for j in range(7) if sees[1, j]] == [0, 1]
    assert P.visible(4, None).tolist() == torch.ones(4, 4).tril().bool().tolist()
    # the hashed rows: the first token takes the last row
    assert P.pair_rows([4, 9, 2], 10, 3, 8) == [10, (12 + 72) % 10, (27 + 16) % 10]
    x = torch.tensor([[1.0, 3.0]])
    assert torch.allclose(P.layer_norm(x, torch.tensor([2.0, 1.0]), torch.tensor([0.5, 0.0]), 0.0), torch.tensor([[-1.5, 1.0]]))
    assert torch.allclose(P.rms_norm(x, torch.ones(2), 0.0), x / math.sqrt(5.0))
    assert abs(float(P.gelu_tanh(torch.tensor(1.0))) - 0.841192) < 1e-5
    # value mixing and the gate: one head of one number that sees itself alone
    one = torch.ones(1, 1)
    w = {"q": one, "k": one, "v": torch.tensor([[3.0]]), "q.norm": torch.ones(1), "k.norm": torch.ones(1), "vmix": torch.tensor(0.25),
         "g": torch.zeros(1, 1), "o": torch.tensor([[2.0]])}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0}
    y, first = P.attention(one, w, m, 1e-6)
    assert float(first) == 3.0 and abs(float(y) - 3.0) < 1e-6
    y, first = P.attention(one, w, m, 1e-6, v_first=torch.full((1, 1, 1), 7.0))
    assert float(first) == 3.0 and abs(float(y) - (0.75 * 3 + 0.25 * 7)) < 1e-6
