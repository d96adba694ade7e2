"""Typed configuration of the Gidurax decoder, read from the keys of its own config.json, and its
`ModelSpec` builder.

A Gidurax model is a list of layers with an RMS norm on both sides of each sublayer (x <- x + m N1b(mixer(N1(x))), then
x <- x + m N2b(ff(N2(x))), m one factor of the whole model).  A layer's mixer is one of three: a gated delta rule with short
convolutions; grouped-query attention without positions, with a weighted RMS norm on every head of q and k, a query
temperature that grows with the logarithm of the position, a learned sink per head and a value size of its own; or a selective
scan (Mamba).  The feed-forward is absent, dense without a gate (exact GELU) or a mixture of such experts: one softmax over all
router outputs, the choice on score + correction, the chosen scores themselves as weights, last outputs that return their
input, and a shared expert behind a sigmoid gate.  A run of layers may be executed several times in a row with the same
weights, each pass with a cache or state of its own; a vector per pass, and from the second pass on the embedded rows, are added
to the residual in front of it.  The output head has a matrix of its own.  Every size and every constant that can differ
between models comes from config.json:

    architecture   "Gidurax"
    vocab, width, norm.eps
    embedding      {scale (optional, 1)} (optional)
    residual_mult  (optional, 1)
    loop           (optional) {start, stop, times}: layers start .. stop-1 run `times` times in a row
    layers[i]      {"type": "delta" | "attention" | "mamba1", "mixer": {...}, "mlp": {...} | null}
      delta          heads, kv_heads (optional, = heads), dim, vdim (optional, = dim), conv
      attention      heads, kv_heads (optional, = heads), dim, vdim (optional, = dim), scale, q_temp {coef, every} (optional)
      mamba1         inner, state, dt_rank, conv
      mlp            {"kind": "dense", "ff"}
                     {"kind": "moe", "expert": {ff}, "router": {experts, top, identity (optional)}, "shared": {ff} (optional)}
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .registry import ConfigError, register_architecture
from .specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Gidurax"
MOST_TAPS, MOST_STATE, MOST_TOP = 16, 256, 32


def _number(where: str, raw: Any, key: str, typ, positive: bool = True):
    if not isinstance(raw, Mapping) or key not in raw or raw[key] is None:
        raise ConfigError(f"config.json: {where}: required key {key!r} is missing")
    v = raw[key]
    if isinstance(v, bool) or not isinstance(v, (int, float) if typ is float else int):
        raise ConfigError(f"config.json: {where}.{key} must be {'a number' if typ is float else 'an integer'}, got {v!r}")
    v = typ(v)
    if not math.isfinite(v) or (positive and not v > 0):
        raise ConfigError(f"config.json: {where}.{key} must be {'positive and ' if positive else ''}finite, got {v!r}")
    return v


def _optional(where: str, raw: Any, key: str, typ, default, positive: bool = True):
    if not isinstance(raw, Mapping) or raw.get(key) is None:
        return default
    return _number(where, raw, key, typ, positive)


def _whole(where: str, raw: Any, key: str, default: Optional[int] = None) -> int:
    v = _number(where, raw, key, int, positive=False) if default is None else _optional(where, raw, key, int, default, positive=False)
    if v < 0:
        raise ConfigError(f"config.json: {where}.{key} must not be negative, got {v}")
    return v


def _at_most(where: str, key: str, v: int, most: int) -> int:
    if v > most:
        raise ConfigError(f"config.json: {where}.{key} {v}: at most {most} is supported")
    return v


def _heads(where: str, raw: Mapping[str, Any]) -> Dict[str, int]:
    heads, dim = _number(where, raw, "heads", int), _number(where, raw, "dim", int)
    kv_heads = _optional(where, raw, "kv_heads", int, heads)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": _optional(where, raw, "vdim", int, dim)}


def _delta(where: str, raw: Mapping[str, Any]) -> Dict[str, Any]:
    return {**_heads(where, raw), "conv": _number(where, raw, "conv", int)}


def _attention(where: str, raw: Mapping[str, Any]) -> Dict[str, Any]:
    out: Dict[str, Any] = {**_heads(where, raw), "scale": _number(where, raw, "scale", float)}
    t = raw.get("q_temp")
    out["q_temp"] = None if t is None else {"coef": _number(where + ".q_temp", t, "coef", float, positive=False),
                                            "every": _number(where + ".q_temp", t, "every", float)}
    return out


def _mamba1(where: str, raw: Mapping[str, Any]) -> Dict[str, Any]:
    out = {key: _number(where, raw, key, int) for key in ("inner", "state", "dt_rank", "conv")}
    _at_most(where, "conv", out["conv"], MOST_TAPS)
    _at_most(where, "state", out["state"], MOST_STATE)
    return out


_MIXERS = {"delta": _delta, "attention": _attention, "mamba1": _mamba1}


def _mlp(where: str, raw: Any) -> Optional[Dict[str, Any]]:
    if raw is None:
        return None
    if not isinstance(raw, Mapping) or raw.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where}.kind must be 'dense' or 'moe' (or mlp null), got "
                          f"{raw.get('kind') if isinstance(raw, Mapping) else raw!r}")
    if raw["kind"] == "dense":
        return {"kind": "dense", "ff": _number(where, raw, "ff", int)}
    r = raw.get("router")
    experts, top = _number(where + ".router", r, "experts", int), _number(where + ".router", r, "top", int)
    identity = _whole(where + ".router", r, "identity", 0)
    if top > experts + identity:
        raise ConfigError(f"config.json: {where}.router: top {top} exceeds the {experts + identity} outputs (experts + identity)")
    _at_most(where + ".router", "top", top, MOST_TOP)
    s = raw.get("shared")
    return {"kind": "moe", "expert": {"ff": _number(where + ".expert", raw.get("expert"), "ff", int)},
            "router": {"experts": experts, "top": top, "identity": identity},
            "shared": None if s is None else {"ff": _number(where + ".shared", s, "ff", int)}}


@dataclass(frozen=True)
class GiduraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    residual_mult: float
    loop: Optional[Mapping[str, int]]
    layers: Tuple[Mapping[str, Any], ...]       # validated copies of config.json's entries
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "GiduraxConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(lr, Mapping) or lr.get("type") not in _MIXERS:
                raise ConfigError(f"config.json: {where}.type must be one of {tuple(_MIXERS)}, got "
                                  f"{lr.get('type') if isinstance(lr, Mapping) else lr!r}")
            if not isinstance(lr.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where}: required key 'mixer' is missing")
            layers.append({"type": lr["type"], "mixer": _MIXERS[lr["type"]](where + ".mixer", lr["mixer"]),
                           "mlp": _mlp(where + ".mlp", lr.get("mlp"))})
        loop = raw.get("loop")
        if loop is not None:
            loop = {"start": _whole("loop", loop, "start"), "stop": _whole("loop", loop, "stop"), "times": _number("loop", loop, "times", int)}
            if not loop["start"] < loop["stop"] <= len(layers):
                raise ConfigError(f"config.json: loop: start {loop['start']} .. stop {loop['stop']} is no run of the "
                                  f"{len(layers)} layers")
        return cls(vocab=_number("top level", raw, "vocab", int), width=_number("top level", raw, "width", int),
                   eps=_number("norm", raw.get("norm"), "eps", float),
                   embedding_scale=_optional("embedding", raw.get("embedding"), "scale", float, 1.0, positive=False),
                   residual_mult=_optional("top level", raw, "residual_mult", float, 1.0, positive=False), loop=loop,
                   layers=tuple(layers))

    def schedule(self) -> Tuple[ScheduleEntry, ...]:
        """The layers in the order in which they run, the starts of the loop's passes marked."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        a, b, times = self.loop["start"], self.loop["stop"], self.loop["times"]
        passes = [ScheduleEntry(i, pass_start=t if i == a else None) for t in range(times) for i in range(a, b)]
        return (*(ScheduleEntry(i) for i in range(a)), *passes, *(ScheduleEntry(i) for i in range(b, n)))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                             "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult,
                             "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            d["loop"] = dict(self.loop)
        return d


def _mixer_spec(cfg: GiduraxConfig, kind: str, m: Mapping[str, Any]) -> PartSpec:
    common = {"hidden_size": cfg.width, "eps": cfg.eps}
    if kind == "delta":
        return PartSpec("gated_delta", {**common, **m})
    if kind == "mamba1":
        return PartSpec("selective_scan", {"hidden_size": cfg.width, **m})
    return PartSpec("gated_attention", {
        **common, "heads": m["heads"], "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"], "scale": m["scale"],
        "bias": False, "qk_norm": "head", "gate": False, "window": None, "sink": True, "q_temp": m["q_temp"],
        "position": PartSpec("rope", {"theta": 10000.0, "rotary_dim": 0, "pairing": "half"})})        # nothing is rotated


def _ffn_spec(cfg: GiduraxConfig, mlp: Optional[Mapping[str, Any]]) -> Optional[PartSpec]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("mlp", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu"})
    r, s = mlp["router"], mlp["shared"]
    return PartSpec("ungated_moe", {
        "hidden_size": cfg.width, "experts": r["experts"], "identity": r["identity"], "top": r["top"], "expert_ff": mlp["expert"]["ff"],
        "shared_ff": None if s is None else s["ff"], "activation": "gelu", "renormalize": False})


def build_spec(cfg: GiduraxConfig) -> ModelSpec:
    """Tensor names: `embed`, `head`, `final.norm`, `loop.step` (with a loop), `l<i>.{norm1,norm1b}`, `l<i>.{norm2,norm2b}` (with a
    feed-forward), `l<i>.mix.*` (delta: q, k, v with .conv, b, a, A_log, dt_bias, norm, g, o; attention: q, k, v, q.norm, k.norm, sink, o;
    mamba1: in, conv, conv.b, x, dt, dt.b, A_log, D, o), `l<i>.mlp.{up,down}` or `l<i>.mlp.e<j>.{up,down}` with `l<i>.mlp.router`,
    `l<i>.mlp.correction` and `l<i>.mlp.shared.{up,down,sg}`; i is the layer's place in config.json."""
    norm = PartSpec("rmsnorm", {"eps": cfg.eps})
    block = PartSpec("sandwich_norm", {"factor": cfg.residual_mult})
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        extra = {"mixer_out": (norm, p + "norm1b")}
        if layer["mlp"] is not None:
            extra["ffn_out"] = (norm, p + "norm2b")
        layers.append(LayerSpec(block=block, norm=norm, mixer=_mixer_spec(cfg, layer["type"], layer["mixer"]),
                                ffn=_ffn_spec(cfg, layer["mlp"]), mixer_prefix=p + "mix.", ffn_prefix=p + "mlp.",
                                mixer_norm_name=p + "norm1", ffn_norm_name=p + "norm2", extra_norms=extra))
    passes = None if cfg.loop is None else (PartSpec("step_vectors", {"times": cfg.loop["times"]}), "loop.")
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers), schedule=cfg.schedule(),
        final_norm=norm, embedding_name="embed", final_norm_name="final.norm", lm_head_name="head",
        embedding_scale=cfg.embedding_scale, max_position=1 << 30, bos_token_id=None, eos_token_id=None, passes=passes)


register_architecture(ARCHITECTURE, GiduraxConfig, build_spec)
