"""Typed configuration of the Botulorn decoder, read from the keys of its own config.json, and its
`ModelSpec` builder.

A Botulorn model is a list of layers whose two sublayers read the same residual, each through a LayerNorm of its own:
x <- x + (mixer(norm1(x)) + ff(norm2(x))).  The embedded row is the token's row times a factor plus a row of a second
table, chosen by a hash of the token and the one in front of it.  A layer's mixer is one of two: grouped-query attention
with a weighted RMS norm on every head of q and k, rotation of halves on the first `rot.dims` numbers of a head, a
sliding window behind which the first positions of a sequence stay visible, values mixed with those of the first layer
that mixes values, a value size of its own and a sigmoid gate per head; or latent attention with a query latent, a rotated
key part that all heads share and a sliding window.  Rotations may be stretched (YaRN).  The feed-forward is absent or
dense, gated by the tanh form of GELU; the output head has a matrix of its own.  Every size and every constant that can
differ between models comes from config.json:

    architecture   "Botulorn"
    vocab, width, norm.eps
    embedding      {scale (optional, 1), bigram {buckets, mul_prev, mul_cur} (optional)}
    layers[i]      {"type": "attention" | "latent_attention", "mixer": {...}, "mlp": {"kind": "dense", ff} | null}
      attention         heads, kv_heads, dim, vdim (optional, = dim), scale, mask {size, keep_first (optional, 0)} (optional),
                        rot (optional), v_mix (optional, false)
      latent_attention  heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask {size} (optional), rot (rot.dims = rot_dim)
      rot               {base, dims, scaling {factor, original, fast, slow} (optional)}
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .registry import ConfigError, register_architecture
from .specs import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

ARCHITECTURE = "Botulorn"
LAYER_TYPES = ("attention", "latent_attention")


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


def _rot(where: str, raw: Mapping[str, Any], most: int) -> Optional[Dict[str, Any]]:
    rot = raw.get("rot")
    if rot is None:
        return None
    where = where + ".rot"
    dims = _whole(where, rot, "dims")
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims {dims} must be even and at most {most}")
    out: Dict[str, Any] = {"base": _number(where, rot, "base", float), "dims": dims}
    s = rot.get("scaling")
    if s is not None:
        where += ".scaling"
        out["scaling"] = {key: _number(where, s, key, float) for key in ("factor", "original", "fast", "slow")}
        if out["base"] == 1.0:
            raise ConfigError(f"config.json: {where} needs a rot.base other than 1")
    return out


def _mask(where: str, raw: Mapping[str, Any], keeps: bool) -> Optional[Dict[str, Any]]:
    m = raw.get("mask")
    if m is None:
        return None
    out = {"size": _number(where + ".mask", m, "size", int)}
    if keeps:
        out["keep_first"] = _whole(where + ".mask", m, "keep_first", 0)
    return out


def _attention(where: str, raw: Mapping[str, Any]) -> Dict[str, Any]:
    heads, kv_heads = _number(where, raw, "heads", int), _number(where, raw, "kv_heads", int)
    dim = _number(where, raw, "dim", int)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads {heads} is not a multiple of kv_heads {kv_heads}")
    v_mix = raw.get("v_mix")
    if v_mix is not None and not isinstance(v_mix, bool):
        raise ConfigError(f"config.json: {where}.v_mix must be true or false, got {v_mix!r}")
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": _optional(where, raw, "vdim", int, dim),
            "scale": _number(where, raw, "scale", float), "rot": _rot(where, raw, dim), "mask": _mask(where, raw, True),
            "v_mix": bool(v_mix)}


def _latent(where: str, raw: Mapping[str, Any]) -> Dict[str, Any]:
    out: Dict[str, Any] = {key: _number(where, raw, key, int) for key in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
    out["rot_dim"] = _whole(where, raw, "rot_dim")
    out["scale"] = _number(where, raw, "scale", float)
    if out["rot_dim"] % 2:
        raise ConfigError(f"config.json: {where}.rot_dim {out['rot_dim']} must be even")
    rot = _rot(where, raw, 1 << 30)            # its size is judged against rot_dim below
    if out["rot_dim"]:
        if rot is None:
            raise ConfigError(f"config.json: {where}: required key 'rot' is missing")
        if rot["dims"] != out["rot_dim"]:
            raise ConfigError(f"config.json: {where}.rot.dims {rot['dims']} must equal rot_dim {out['rot_dim']}")
    out["rot"] = rot if out["rot_dim"] else None
    out["mask"] = _mask(where, raw, False)
    return out


_MIXERS = {"attention": _attention, "latent_attention": _latent}


def _mlp(where: str, raw: Any) -> Optional[Dict[str, Any]]:
    if raw is None:
        return None
    if not isinstance(raw, Mapping) or raw.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}.kind must be 'dense' (or mlp null), got "
                          f"{raw.get('kind') if isinstance(raw, Mapping) else raw!r}")
    return {"kind": "dense", "ff": _number(where, raw, "ff", int)}


@dataclass(frozen=True)
class BotulornConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    bigram: Optional[Mapping[str, int]]
    layers: Tuple[Mapping[str, Any], ...]       # validated copies of config.json's entries
    architecture: str = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "BotulornConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(lr, Mapping) or lr.get("type") not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type must be one of {LAYER_TYPES}, got "
                                  f"{lr.get('type') if isinstance(lr, Mapping) else lr!r}")
            if not isinstance(lr.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where}: required key 'mixer' is missing")
            layers.append({"type": lr["type"], "mixer": _MIXERS[lr["type"]](where + ".mixer", lr["mixer"]),
                           "mlp": _mlp(where + ".mlp", lr.get("mlp"))})
        mixing = [(i, l["mixer"]) for i, l in enumerate(layers) if l["mixer"].get("v_mix")]
        for i, m in mixing[1:]:
            first, m0 = mixing[0]
            if (m["kv_heads"], m["vdim"]) != (m0["kv_heads"], m0["vdim"]):
                raise ConfigError(f"config.json: layers[{i}].mixer.v_mix: its values ({m['kv_heads']} heads of {m['vdim']}) cannot be "
                                  f"mixed with those of layers[{first}] ({m0['kv_heads']} heads of {m0['vdim']})")
        e = raw.get("embedding")
        b = e.get("bigram") if isinstance(e, Mapping) else None
        bigram = None
        if b is not None:
            bigram = {"buckets": _number("embedding.bigram", b, "buckets", int),
                      "mul_prev": _whole("embedding.bigram", b, "mul_prev"), "mul_cur": _whole("embedding.bigram", b, "mul_cur")}
        return cls(vocab=_number("top level", raw, "vocab", int), width=_number("top level", raw, "width", int),
                   eps=_number("norm", raw.get("norm"), "eps", float),
                   embedding_scale=_optional("embedding", e, "scale", float, 1.0, positive=False), bigram=bigram,
                   layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        embedding: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            embedding["bigram"] = dict(self.bigram)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": embedding, "layers": copy.deepcopy(list(self.layers))}


def _position(rot: Optional[Mapping[str, Any]]) -> PartSpec:
    rot = rot or {"base": 10000.0, "dims": 0}
    return PartSpec("rope", {"theta": rot["base"], "rotary_dim": rot["dims"], "pairing": "half", "yarn": rot.get("scaling")})


def _mixer_spec(cfg: BotulornConfig, kind: str, m: Mapping[str, Any], v_mix: Optional[str]) -> PartSpec:
    common = {"hidden_size": cfg.width, "eps": cfg.eps, "heads": m["heads"], "scale": m["scale"], "position": _position(m["rot"]),
              "window": (m["mask"] or {}).get("size")}
    if kind == "attention":
        return PartSpec("gated_attention", {
            **common, "kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"], "keep": (m["mask"] or {}).get("keep_first", 0),
            "bias": False, "qk_norm": "head", "gate": "head", "v_mix": v_mix})
    return PartSpec("latent_attention", {
        **common, "dim": m["dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "rot_dim": m["rot_dim"],
        "sink": False, "gate": None})


def _ffn_spec(cfg: BotulornConfig, mlp: Optional[Mapping[str, Any]]) -> Optional[PartSpec]:
    if mlp is None:
        return None
    return PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": mlp["ff"], "activation": "gelu_tanh",
                               "tensor_names": ("gate", "up", "down")})


def build_spec(cfg: BotulornConfig) -> ModelSpec:
    """Tensor names: `embed`, `bigram`, `head`, `final.norm`(`.b`), `l<i>.norm1`(`.b`), `l<i>.norm2`(`.b`, with a feed-forward),
    `l<i>.mix.*` (attention: q, k, v, q.norm, k.norm, g, o, with value mixing vmix; latent attention: dq, dq.norm, uq, dkv,
    dkv.norm, uk, uv, o), `l<i>.mlp.{gate,up,down}`; i is the layer's place in config.json."""
    norm = PartSpec("layernorm", {"eps": cfg.eps})
    block = PartSpec("two_norms", {})
    layers, seen_source = [], False
    for i, layer in enumerate(cfg.layers):
        p, v_mix = f"l{i}.", None
        if layer["mixer"].get("v_mix"):
            v_mix = "mix" if seen_source else "source"
            seen_source = True
        layers.append(LayerSpec(block=block, norm=norm, mixer=_mixer_spec(cfg, layer["type"], layer["mixer"], v_mix),
                                ffn=_ffn_spec(cfg, layer["mlp"]), mixer_prefix=p + "mix.", ffn_prefix=p + "mlp.",
                                mixer_norm_name=p + "norm1", ffn_norm_name=p + "norm2"))
    inputs = ()
    if cfg.bigram is not None:
        inputs = ((PartSpec("pair_embedding", {**cfg.bigram, "tensor_name": "bigram"}), ""),)
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm, embedding_name="embed",
        final_norm_name="final.norm", lm_head_name="head", embedding_scale=cfg.embedding_scale, max_position=1 << 30,
        bos_token_id=None, eos_token_id=None, inputs=inputs)


register_architecture(ARCHITECTURE, BotulornConfig, build_spec)
