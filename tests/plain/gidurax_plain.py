"""Plain, slow statement of the Gidurax decoder: whole sequences, no cache, no batching, one
function per mechanism, CPU float32.  It shares no code with the package under test.

Notation: x is the [tokens, width] residual of one sequence, W matrices are [out, in] and are
applied as x W^T, t and j run over tokens in order, positions count from 0.  `rnd` is where an
engine that stores activations in bfloat16 rounds them (identity for the 32-bit statement).

A layer norms every sublayer on both sides, m being one factor of the whole model:
    x <- x + m N1b(mixer(N1(x)));   x <- x + m N2b(ff(N2(x)))
A run of layers [start, stop) is executed `times` times in a row with the same weights; pass t
starts with x <- x + step[t], and every pass but the first with x <- x + e before that, e being
the embedded rows.
"""
from __future__ import annotations

import math
from typing import Callable, Dict, List, Mapping, Optional, Tuple

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
# small pieces


def rms_norm(y: Tensor, w: Tensor, eps: float) -> Tensor:
    """y / sqrt(mean(y^2) + eps) * w over the last axis; the weight multiplies plainly."""
    y = y.float()
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * w.float()


def silu(z: Tensor) -> Tensor:
    return z * torch.sigmoid(z)


def softplus(z: Tensor) -> Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def gelu_erf(z: Tensor) -> Tensor:
    return z * 0.5 * (1.0 + torch.erf(z / math.sqrt(2.0)))


def unit(y: Tensor) -> Tensor:
    """y / sqrt(sum y^2 + 1e-6) over the last axis."""
    return y / torch.sqrt((y * y).sum(-1, keepdim=True) + 1e-6)


def short_conv(x: Tensor, taps: Tensor, bias: Optional[Tensor] = None) -> Tensor:
    """u[t, c] = b[c] + sum_j taps[c, K-1-j] x[t-j, c], zeros in front of the sequence."""
    T, C = x.shape
    K = taps.shape[1]
    out = torch.zeros(T, C) if bias is None else bias.float().expand(T, C).clone()
    for j in range(min(K, T)):
        out[j:] += x[:T - j].float() * taps[:, K - 1 - j].float()
    return out


# ---------------------------------------------------------------------------------------
# mixer: gated delta rule


def delta_rule(q: Tensor, k: Tensor, v: Tensor, beta: Tensor, decay: Tensor, S: Optional[Tensor] = None) -> Tuple[Tensor, Tensor]:
    """One head: q, k [T, d], v [T, dv], beta and decay [T].  S (d x dv) is decayed, corrected towards
    v at k, then read at q.  Returns (o [T, dv], the last S)."""
    S = torch.zeros(q.shape[1], v.shape[1]) if S is None else S.clone()
    out = torch.zeros(q.shape[0], v.shape[1])
    for t in range(q.shape[0]):
        S = decay[t] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.t() @ q[t]
    return out, S


def delta_mixer(h: Tensor, w: Mapping[str, Tensor], m: Mapping, eps: float, rnd: Round = exact) -> Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name):
        return silu(short_conv(rnd(lin(h, w[name])), w[name + ".conv"]))
    q = unit(branch("q").view(T, G, d)) * d ** -0.5
    k = unit(branch("k").view(T, G, d))
    v = branch("v").view(T, H, dv)
    beta = torch.sigmoid(lin(h, w["b"]))
    decay = torch.exp(-torch.exp(w["A_log"].float()) * softplus(lin(h, w["a"]) + w["dt_bias"].float()))
    o = torch.zeros(T, H, dv)
    for i in range(H):
        g = i // (H // G)
        o[:, i], _ = delta_rule(q[:, g], k[:, g], v[:, i], beta[:, i], decay[:, i])
    o = rms_norm(o, w["norm"], eps).reshape(T, H * dv) * silu(rnd(lin(h, w["g"])))
    return lin(rnd(o), w["o"])


# ---------------------------------------------------------------------------------------
# mixer: attention


def temperature(positions: Tensor, coef: float, every: float) -> Tensor:
    """1 + coef ln(floor((p + 1) / every) + 1)."""
    return 1.0 + coef * torch.log(torch.floor((positions.double() + 1.0) / every) + 1.0).float()


def sink_attention(q: Tensor, k: Tensor, v: Tensor, scale: float, sink: Tensor) -> Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H/G); token t sees tokens
    j <= t; the softmax's denominator also holds exp(sink[h]).  Returns [T, H, dv]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2])
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t()) * scale
        s = torch.where(mask, s, torch.full_like(s, -math.inf))
        s = torch.cat([s, sink[h].float().expand(T, 1)], dim=1)
        out[:, h] = torch.softmax(s, dim=1)[:, :T] @ v[:, g]
    return out


def attention_mixer(h: Tensor, w: Mapping[str, Tensor], m: Mapping, eps: float, rnd: Round = exact, first_position: int = 0) -> Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(h, w["q"]).view(T, H, d), w["q.norm"], eps)
    k = rms_norm(lin(h, w["k"]).view(T, G, d), w["k.norm"], eps)
    v = rnd(lin(h, w["v"])).view(T, G, dv)
    qt = m.get("q_temp")
    if qt is not None:
        q = q * temperature(torch.arange(first_position, first_position + T), qt["coef"], qt["every"])[:, None, None]
    a = sink_attention(rnd(q), rnd(k), v, m["scale"], w["sink"])
    return lin(rnd(a.reshape(T, H * dv)), w["o"])


# ---------------------------------------------------------------------------------------
# mixer: selective scan


def selective_scan(x: Tensor, dt: Tensor, A: Tensor, Bv: Tensor, Cv: Tensor, D: Tensor, S: Optional[Tensor] = None) -> Tuple[Tensor, Tensor]:
    """x, dt [T, C], A [C, N], Bv, Cv [T, N], D [C].  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;
    y_c = sum_n S[c, n] C_n + D_c x_c.  Returns (y [T, C], the last S)."""
    S = torch.zeros_like(A) if S is None else S.clone()
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * Bv[t][None, :]
        out[t] = S @ Cv[t] + D * x[t]
    return out, S


def scan_mixer(h: Tensor, w: Mapping[str, Tensor], m: Mapping, eps: float, rnd: Round = exact) -> Tensor:
    C, R, N = m["inner"], m["dt_rank"], m["state"]
    xz = rnd(lin(h, w["in"]))
    x, z = xz[:, :C], xz[:, C:]
    x = rnd(silu(short_conv(x, w["conv"], w["conv.b"])))
    p = lin(x, w["x"])
    dt = softplus(lin(rnd(p[:, :R]), w["dt"]) + w["dt.b"].float())
    y, _ = selective_scan(x, dt, -torch.exp(w["A_log"].float()), p[:, R:R + N], p[:, R + N:], w["D"].float())
    return lin(rnd(y * silu(z)), w["o"])


# ---------------------------------------------------------------------------------------
# feed-forwards


def plain_ff(h: Tensor, up: Tensor, down: Tensor, rnd: Round = exact) -> Tensor:
    return lin(rnd(gelu_erf(lin(h, up))), down)


def route(z: Tensor, correction: Tensor, top: int) -> Tuple[Tensor, Tensor]:
    """z [T, N]: s = softmax(z); the `top` largest s + correction are chosen (the lower index wins a tie), weighted by
    their s as they are.  Returns (indices [T, top], weights [T, top])."""
    s = torch.softmax(z.float(), dim=-1)
    c = s + correction.float()
    idx = torch.stack([torch.tensor(sorted(range(z.shape[1]), key=lambda e: (-float(c[t, e]), e))[:top]) for t in range(z.shape[0])])
    return idx, torch.gather(s, 1, idx)


def moe_ff(h: Tensor, w: Mapping[str, Tensor], mlp: Mapping, rnd: Round = exact) -> Tensor:
    """Experts 0 .. experts-1 have tensors; the later router outputs stand for experts that return their input."""
    r = mlp["router"]
    E = r["experts"]
    idx, wt = route(lin(h, w["router"]), w["correction"], r["top"])
    out = torch.zeros(h.shape[0], h.shape[1])
    for e in range(w["router"].shape[0]):
        share = torch.where(idx == e, wt, torch.zeros_like(wt)).sum(1)
        on = torch.nonzero(share)[:, 0]
        if len(on) == 0:
            continue
        y = h[on].float() if e >= E else plain_ff(h[on], w[f"e{e}.up"], w[f"e{e}.down"], rnd)
        out[on] += share[on][:, None] * y
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(lin(h, w["shared.sg"])) * plain_ff(h, w["shared.up"], w["shared.down"], rnd)
    return out


# ---------------------------------------------------------------------------------------
# the model


MIXERS = {"delta": delta_mixer, "attention": attention_mixer, "mamba1": scan_mixer}


def sub(weights: Mapping[str, Tensor], prefix: str) -> Dict[str, Tensor]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def runs(cfg: Mapping) -> List[Tuple[int, Optional[int]]]:
    """(layer, the number of the pass that starts here or None) in the order in which layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    out = [(i, None) for i in range(a)]
    for t in range(times):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(cfg: Mapping, weights: Mapping[str, Tensor], tokens, rnd: Round = exact, residuals: Optional[list] = None) -> Tensor:
    """Logits [tokens, vocab] of one sequence.  `residuals`, if a list, receives x after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    tok = torch.as_tensor(tokens, dtype=torch.long)
    e = weights["embed"].float()[tok] * (cfg.get("embedding") or {}).get("scale", 1.0)
    x = e.clone()
    for i, start in runs(cfg):
        if start is not None:
            x = x + (e if start > 0 else 0.0) + weights["loop.step"][start].float()
        layer, p = cfg["layers"][i], f"l{i}."
        y = MIXERS[layer["type"]](rnd(rms_norm(x, weights[p + "norm1"], eps)), sub(weights, p + "mix."), layer["mixer"], eps, rnd)
        x = x + m * rms_norm(y, weights[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, w = rnd(rms_norm(x, weights[p + "norm2"], eps)), sub(weights, p + "mlp.")
            y = plain_ff(h, w["up"], w["down"], rnd) if mlp["kind"] == "dense" else moe_ff(h, w, mlp, rnd)
            x = x + m * rms_norm(y, weights[p + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x.clone())
    return lin(rnd(rms_norm(x, weights["final.norm"], eps)), weights["head"])
