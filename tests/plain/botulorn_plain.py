"""Plain, slow statement of the Botulorn decoder: whole sequences, no cache, no batching, one
function per mechanism, CPU float32.  It shares no code with the package under test.

Notation: x is the [tokens, width] residual of one sequence, W matrices are [out, in] and are
applied as x W^T, t and j run over tokens in order, positions count from 0.  `rnd` is where an
engine that stores activations in bfloat16 rounds them (identity for the 32-bit statement).

A layer:   x <- x + (mixer(N1(x)) + ff(N2(x)))        (both norms read the same x; ff may be absent)
N(x) = (x - mean) / sqrt(var + eps) * w + b.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, Mapping, Optional

import torch

Tensor = torch.Tensor
Round = Callable[[Tensor], Tensor]


def exact(t: Tensor) -> Tensor:
    return t


def bf16(t: Tensor) -> Tensor:
    return t.to(torch.bfloat16).to(torch.float32)


def lin(h: Tensor, w: Tensor) -> Tensor:
    return h.float() @ w.float().t()


# ---------------------------------------------------------------------------------------
# norms


def layer_norm(x: Tensor, w: Tensor, b: Tensor, eps: float) -> Tensor:
    x = x.float()
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w.float() + b.float()


def rms_norm(y: Tensor, w: Tensor, eps: float) -> Tensor:
    y = y.float()
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * w.float()


# ---------------------------------------------------------------------------------------
# the embedding


def pair_rows(tokens, buckets: int, mul_prev: int, mul_cur: int):
    """The row of the pair table that each token adds: a hash of the token and the one in front of it; a
    sequence's first token has none in front and takes the row behind the hashed ones."""
    rows = []
    for t, tok in enumerate(tokens):
        rows.append(buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tok) * mul_cur) % buckets)
    return rows


def embed(cfg: Mapping, weights: Mapping[str, Tensor], tokens) -> Tensor:
    e = cfg.get("embedding") or {}
    x = weights["embed"].float()[torch.as_tensor(tokens, dtype=torch.long)] * e.get("scale", 1.0)
    if e.get("bigram"):
        b = e["bigram"]
        x = x + weights["bigram"].float()[pair_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]
    return x


# ---------------------------------------------------------------------------------------
# rotations: v [tokens, heads, dim]; the first `dims` numbers of a head turn, the rest pass


def turn_rates(rot: Mapping):
    """(radians per position of every pair, the factor on cosine and sine).  Stretched rotations: pairs that make
    at least `fast` turns within `original` positions keep their rate, pairs that make at most `slow` turns have it
    divided by `factor`, and the rates of the pairs between are mixed linearly in the pair's number."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def pair_with_turns(n):
        return dims * math.log(s["original"] / (2.0 * math.pi * n)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_with_turns(s["fast"])), 0)
    hi = min(math.ceil(pair_with_turns(s["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(v: Tensor, rot: Optional[Mapping], first_position: int = 0) -> Tensor:
    """Number i turns together with number i + dims/2."""
    out = v.clone().float()
    half = rot["dims"] // 2 if rot else 0
    if half == 0:
        return out
    rates, m = turn_rates(rot)
    pos = torch.arange(first_position, first_position + v.shape[0], dtype=torch.float32)
    ang = pos[:, None] * torch.tensor(rates, dtype=torch.float64).float()[None, :]
    c, s = (torch.cos(ang) * m)[:, None, :], (torch.sin(ang) * m)[:, None, :]
    a, b = v[..., :half].float(), v[..., half:2 * half].float()
    out[..., :half] = a * c - b * s
    out[..., half:2 * half] = b * c + a * s
    return out


# ---------------------------------------------------------------------------------------
# softmax attention under a visibility rule


def visible(T: int, size: Optional[int], keep_first: int = 0) -> Tensor:
    """[T, T] booleans: row t sees column j if j is not ahead and lies among the last `size` positions (t included)
    or among the first `keep_first` of the sequence."""
    t, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = (t - j < size) if size else torch.ones(T, T, dtype=torch.bool)
    return (j <= t) & (near | (j < keep_first))


def masked_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, sees: Tensor) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H/G); softmax over what a
    token sees.  Returns [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2])
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h].float() @ k[:, g].float().t()) * scale
        out[:, h] = torch.softmax(s.masked_fill(~sees, -math.inf), dim=-1) @ v[:, g].float()
    return out


def attention(h: Tensor, w: Mapping[str, Tensor], m: Mapping, eps: float, rnd: Round = exact, v_first: Optional[Tensor] = None):
    """Returns (the mixer's result, the values as projected [T, G, dv]).  `v_first`: the first value-mixing layer's
    projected values, which this layer's own are mixed with."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w["q"]).view(T, H, d), w["q.norm"], eps)
    k = rms_norm(lin(h, w["k"]).view(T, G, d), w["k.norm"], eps)
    v = projected = lin(h, w["v"]).view(T, G, dv)
    if v_first is not None:
        lam = float(w["vmix"])
        v = (1.0 - lam) * v + lam * v_first
    q, k = rnd(rotate(q, m.get("rot"))), rnd(rotate(k, m.get("rot")))
    mask = m.get("mask") or {}
    o = rnd(masked_attention(q, k, rnd(v), m["scale"], visible(T, mask.get("size"), mask.get("keep_first") or 0)))
    gate = torch.sigmoid(lin(h, w["g"]))                                                # [T, H]
    return lin(rnd((o * gate[:, :, None]).reshape(T, H * dv)), w["o"]), projected


def latent_attention(h: Tensor, w: Mapping[str, Tensor], m: Mapping, eps: float, rnd: Round = exact) -> Tensor:
    """Queries through a low-rank row of their own; keys and values grow out of one short row c per token; beside it
    one rotated key part that all heads share."""
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rnd(rms_norm(lin(h, w["dq"]), w["dq.norm"], eps))
    q = lin(cq, w["uq"]).view(T, H, d + r)
    down = lin(h, w["dkv"])
    c = rnd(rms_norm(down[:, :rank], w["dkv.norm"], eps))
    k_rot = rotate(down[:, None, rank:], m.get("rot"))                                  # [T, 1, r]
    q = torch.cat([q[..., :d], rotate(q[..., d:], m.get("rot"))], dim=-1)
    k = torch.cat([lin(c, w["uk"]).view(T, H, d), k_rot.expand(T, H, r)], dim=-1)
    v = lin(c, w["uv"]).view(T, H, dv)
    o = masked_attention(rnd(q), rnd(k), rnd(v), m["scale"], visible(T, (m.get("mask") or {}).get("size")))
    return lin(rnd(o.reshape(T, H * dv)), w["o"])


# ---------------------------------------------------------------------------------------
# feed-forward


def gelu_tanh(z: Tensor) -> Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h: Tensor, w: Mapping[str, Tensor], rnd: Round = exact) -> Tensor:
    return lin(rnd(gelu_tanh(lin(h, w["gate"])) * lin(h, w["up"])), w["down"])


# ---------------------------------------------------------------------------------------
# the model


def sub(weights: Mapping[str, Tensor], prefix: str) -> Dict[str, Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg: Mapping, weights: Mapping[str, Tensor], tokens, rnd: Round = exact, residuals: Optional[list] = None) -> Tensor:
    """Logits [tokens, vocab] of one sequence.  `residuals`, if a list, receives x after every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(cfg, weights, tokens)
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rnd(layer_norm(x, weights[p + "norm1"], weights[p + "norm1.b"], eps))
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, projected = attention(h, sub(weights, p + "mix."), m, eps, rnd, v_first if mixes else None)
            if mixes and v_first is None:
                v_first = projected
        else:
            y = latent_attention(h, sub(weights, p + "mix."), m, eps, rnd)
        if layer.get("mlp") is not None:
            h = rnd(layer_norm(x, weights[p + "norm2"], weights[p + "norm2.b"], eps))
            y = y + dense_ff(h, sub(weights, p + "mlp."), rnd)
        x = x + y
        if residuals is not None:
            residuals.append(x.clone())
    hn = rnd(layer_norm(x, weights["final.norm"], weights["final.norm.b"], eps))
    return lin(hn, weights["head"])
