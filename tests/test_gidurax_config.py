"""The Gidurax configuration on the CPU: keys read and defaults, refusals that name the key, the spec it builds (tensor names,
parts and their constants, the schedule with its passes), the random folder, a cache or state entry per run of a layer, and the
plain statement's pieces against hand-worked numbers."""
import json
import math

import pytest
import torch

from inference_engine_rust_b200.cache import KVRequest, StateRequest
from inference_engine_rust_b200.config import ConfigError, ModelSpec, ScheduleEntry, config_from_dict, preset, spec_of
from inference_engine_rust_b200.engine.model import Model
from inference_engine_rust_b200.parts.base import Runtime
from plain import gidurax_plain as P

DELTA = {"heads": 6, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 3}
ATT = {"heads": 6, "kv_heads": 3, "dim": 10, "vdim": 14, "scale": 0.4, "q_temp": {"coef": 0.3, "every": 7}}
SCAN = {"inner": 44, "state": 9, "dt_rank": 5, "conv": 5}
DENSE = {"kind": "dense", "ff": 30}
MOE = {"kind": "moe", "expert": {"ff": 11}, "router": {"experts": 5, "identity": 2, "top": 3}, "shared": {"ff": 13}}


def cfg(**top):
    layers = [{"type": "attention", "mixer": ATT, "mlp": DENSE}, {"type": "delta", "mixer": DELTA, "mlp": MOE},
              {"type": "mamba1", "mixer": SCAN, "mlp": None}, {"type": "mamba1", "mixer": SCAN, "mlp": DENSE}]
    d = {"architecture": "Gidurax", "vocab": 90, "width": 52, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0}, "residual_mult": 0.6,
         "loop": {"start": 1, "stop": 3, "times": 3}, "layers": json.loads(json.dumps(layers))}
    d.update(top)
    return d


def model_of(raw):
    return Model(spec_of(config_from_dict(raw)), Runtime(dtype=torch.float32, device="cpu"))


def test_spec_of_a_configuration():
    c = config_from_dict(cfg())
    spec = spec_of(c)
    assert [(e.layer, e.pass_start) for e in spec.schedule] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    assert spec.embedding_scale == 3.0 and spec.lm_head_name == "head" and spec.final_norm["eps"] == 1e-5
    assert spec.passes[0].kind == "step_vectors" and spec.passes[0]["times"] == 3 and spec.passes[1] == "loop."
    assert all(l.block.kind == "sandwich_norm" and l.block["factor"] == 0.6 for l in spec.layers)
    a = spec.layers[0].mixer
    assert a.kind == "gated_attention" and a["sink"] and not a["bias"] and not a["gate"] and a["qk_norm"] == "head" and a["window"] is None
    assert a["q_temp"] == {"coef": 0.3, "every": 7.0} and (a["head_dim"], a["v_dim"], a["scale"]) == (10, 14, 0.4)
    assert a["position"]["rotary_dim"] == 0
    assert spec.layers[1].mixer.kind == "gated_delta" and spec.layers[1].mixer["conv"] == 3 and spec.layers[1].mixer["eps"] == 1e-5
    assert spec.layers[2].mixer.kind == "selective_scan" and spec.layers[2].ffn is None and "ffn_out" not in spec.layers[2].extra_norms
    f = spec.layers[1].ffn
    assert f.kind == "ungated_moe" and (f["experts"], f["identity"], f["top"], f["expert_ff"], f["shared_ff"]) == (5, 2, 3, 11, 13)
    assert f["renormalize"] is False and spec.layers[0].ffn.kind == "mlp"
    model = model_of(cfg())
    shapes = {k: tuple(v.shape) for k, v in model.expected_tensors().items()}
    names = ({"embed", "head", "final.norm", "loop.step"} | {f"l{i}.norm{n}" for i in range(4) for n in ("1", "1b")}
             | {f"l{i}.norm{n}" for i in (0, 1, 3) for n in ("2", "2b")} | {f"l{i}.mlp.{n}" for i in (0, 3) for n in ("up", "down")}
             | {f"l1.mlp.e{e}.{n}" for e in range(5) for n in ("up", "down")}
             | {"l1.mlp.router", "l1.mlp.correction", "l1.mlp.shared.up", "l1.mlp.shared.down", "l1.mlp.shared.sg"}
             | {f"l0.mix.{n}" for n in ("q", "k", "v", "q.norm", "k.norm", "sink", "o")}
             | {f"l1.mix.{n}" for n in ("q", "k", "v", "q.conv", "k.conv", "v.conv", "b", "a", "A_log", "dt_bias", "norm", "g", "o")}
             | {f"l{i}.mix.{n}" for i in (2, 3) for n in ("in", "conv", "conv.b", "x", "dt", "dt.b", "A_log", "D", "o")})
    assert set(shapes) == names
    assert shapes["loop.step"] == (3, 52) and shapes["l0.mix.sink"] == (6,) and shapes["l0.mix.v"] == (42, 52) and shapes["l0.mix.o"] == (52, 84)
    assert shapes["l1.mix.q.conv"] == (24, 3) and shapes["l1.mix.v"] == (120, 52) and shapes["l1.mix.norm"] == (20,)
    assert shapes["l2.mix.in"] == (88, 52) and shapes["l2.mix.x"] == (23, 44) and shapes["l2.mix.dt"] == (44, 5) and shapes["l2.mix.A_log"] == (44, 9)
    assert shapes["l1.mlp.router"] == (7, 52) and shapes["l1.mlp.correction"] == (7,) and shapes["l1.mlp.shared.sg"] == (1, 52)
    reqs = model.cache_requests()
    assert sorted(reqs) == list(range(8))                              # every pass of a layer has storage of its own
    assert reqs[0] == KVRequest(3, 14) and reqs[1] == reqs[3] == reqs[5] == StateRequest((6 * 12 * 20 + 3 * (2 * 24 + 120),))
    assert reqs[2] == reqs[4] == StateRequest((44 * 9 + 5 * 44,))
    assert config_from_dict(c.to_dict()) == c and model.graph_safe()


def test_defaults():
    raw = cfg()
    for key in ("embedding", "residual_mult", "loop"):
        del raw[key]
    del raw["layers"][0]["mixer"]["q_temp"], raw["layers"][0]["mixer"]["vdim"], raw["layers"][1]["mixer"]["kv_heads"]
    del raw["layers"][1]["mlp"]["shared"], raw["layers"][1]["mlp"]["router"]["identity"]
    c = config_from_dict(raw)
    spec = spec_of(c)
    assert spec.embedding_scale == 1.0 and spec.layers[0].block["factor"] == 1.0 and spec.passes is None
    assert [(e.layer, e.pass_start) for e in spec.schedule] == [(i, None) for i in range(4)]
    assert spec.layers[0].mixer["q_temp"] is None and spec.layers[0].mixer["v_dim"] == 10 and spec.layers[1].mixer["kv_heads"] == 6
    names = model_of(raw).expected_tensors()
    assert "loop.step" not in names and "l1.mlp.shared.sg" not in names and names["l1.mlp.router"].shape == (5, 52)
    assert config_from_dict(c.to_dict()) == c


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "mlstm", "type"), (("layers", 0, "mixer"), None, "mixer"), (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 0, "mixer", "scale"), None, "scale"), (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
    (("layers", 0, "mixer", "q_temp", "coef"), None, "coef"), (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 2, "mixer", "conv"), 17, "conv"), (("layers", 2, "mixer", "state"), 257, "state"), (("layers", 2, "mixer", "dt_rank"), None, "dt_rank"),
    (("layers", 0, "mlp", "kind"), "gated", "kind"), (("layers", 0, "mlp", "ff"), 0, "ff"), (("layers", 1, "mlp", "expert"), None, "ff"),
    (("layers", 1, "mlp", "router", "top"), 8, "top"), (("layers", 1, "mlp", "router", "identity"), -1, "identity"),
    (("layers", 1, "mlp", "shared", "ff"), None, "ff"), (("loop", "stop"), 5, "loop"), (("loop", "start"), 3, "loop"),
    (("loop", "times"), 0, "times"), (("norm",), None, "eps"), (("layers",), [], "layers"), (("vocab",), None, "vocab"), (("residual_mult",), "x", "residual_mult"),
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


def test_a_pass_needs_a_part_for_it():
    spec = spec_of(config_from_dict(cfg()))
    kw = {f: getattr(spec, f) for f in spec.__dataclass_fields__}
    with pytest.raises(ValueError, match="starts a pass"):
        ModelSpec(**{**kw, "passes": None}).validate()
    with pytest.raises(ValueError, match="streams"):
        ModelSpec(**{**kw, "residual_streams": 2}).validate()
    ModelSpec(**{**kw, "passes": None, "schedule": (ScheduleEntry(0),)}).validate()


def test_presets_and_random_folder(tmp_path):
    from inference_engine_rust_b200 import write_random_model
    from inference_engine_rust_b200.weights import TensorSource
    for name in ("gidurax-tiny", "gidurax-7b-sizes", "gidurax-12b-sizes"):
        spec_of(config_from_dict(preset(name)))
    d = str(tmp_path / "m")
    write_random_model(d, preset("gidurax-tiny"), seed=3, dtype="bfloat16")
    model = model_of(preset("gidurax-tiny"))
    model.load(TensorSource.open(d) if hasattr(TensorSource, "open") else TensorSource(d))
    assert model.loaded and model.passes.step.shape == (3, 80)


def test_plain_pieces_by_hand():
    x = torch.tensor([[1.0], [2.0], [4.0]])
    u = P.short_conv(x, torch.tensor([[10.0, 1.0]]), torch.tensor([0.5]))              # the last tap is the current token's
    assert u[:, 0].tolist() == [1.5, 12.5, 24.5]
    t = P.temperature(torch.tensor([0, 6, 7, 13, 20]), 2.0, 7)
    assert torch.allclose(t, torch.tensor([1.0, 1 + 2 * math.log(2), 1 + 2 * math.log(2), 1 + 2 * math.log(3), 1 + 2 * math.log(4)]))
    # one key of score 0 beside a sink of log 3: the value comes through with weight 1/4
    a = P.sink_attention(torch.zeros(1, 1, 2), torch.zeros(1, 1, 2), torch.full((1, 1, 1), 8.0), 1.0, torch.tensor([math.log(3.0)]))
    assert torch.allclose(a, torch.full((1, 1, 1), 2.0))
    o, S = P.delta_rule(torch.tensor([[1.0, 0.0], [0.0, 2.0]]), torch.tensor([[1.0, 0.0], [1.0, 1.0]]), torch.tensor([[3.0], [5.0]]),
                        torch.tensor([1.0, 0.5]), torch.tensor([0.7, 0.5]))
    # S = (3, 0); decayed (1.5, 0), u = 0.5 (5 - 1.5) = 1.75, S = (3.25, 1.75)
    assert torch.allclose(o[:, 0], torch.tensor([3.0, 3.5])) and torch.allclose(S[:, 0], torch.tensor([3.25, 1.75]))
    y, S = P.selective_scan(torch.tensor([[2.0], [1.0]]), torch.tensor([[0.5], [1.0]]), torch.tensor([[-math.log(2.0), 0.0]]),
                            torch.tensor([[1.0, 3.0], [2.0, 0.0]]), torch.tensor([[1.0, 1.0], [1.0, 2.0]]), torch.tensor([10.0]))
    # S = (1, 3), y = 4 + 20; then (1/2 + 2, 3), y = 2.5 + 6 + 10
    assert torch.allclose(y[:, 0], torch.tensor([24.0, 18.5])) and torch.allclose(S[0], torch.tensor([2.5, 3.0]))
    idx, w = P.route(torch.log(torch.tensor([[0.5, 0.2, 0.3]])), torch.tensor([-1.0, 0.0, 0.0]), 2)
    assert idx.tolist() == [[2, 1]] and torch.allclose(w, torch.tensor([[0.3, 0.2]]))
    assert torch.allclose(P.gelu_erf(torch.tensor([1.0])), torch.tensor([0.8413447]), atol=1e-6)
    order = P.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}})
    assert order == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
