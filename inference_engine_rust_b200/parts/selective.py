"""A selective scan (Mamba: Gu and Dao, "Mamba: Linear-Time Sequence Modeling with Selective State Spaces").  With h the
mixer's input, C = `inner` channels, N = `state` numbers kept per channel, R = `dt_rank`:

    [x | z] = W_in h
    u = silu(conv(x))                a causal convolution per channel over `conv` taps (the last tap is the current token's),
                                     with a bias, zeros before the sequence's start
    [d | B | C] = W_x u              R, N and N numbers
    dt = softplus(W_dt d + b_dt)     one per channel;  A = -exp(A_log)
    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n;   y_c = sum_n S[c, n] C_n + D_c u_c
    result = W_o (y * silu(z))

State per sequence (fp32, zero at the start, carried from step to step): S and the convolution's last inputs.  Tensors: in
[2C, hidden], conv [C, taps], conv.b [C], x [R + 2N, C], dt [C, R], dt.b [C], A_log [C, N], D [C], o [hidden, C].

The products run in the run's dtype, W_dt's with fp32 outputs; bias, softplus and everything after are fp32 arithmetic in the
kernels of `csrc/selective_scan.cu`."""
from __future__ import annotations

import math
from typing import Dict, Mapping

import torch

from ..cache import StateRequest
from ..csrc import bindings as B
from ..weights.loader import TensorSpec
from .base import Mixer, Runtime, StepContext, register_part
from .linear import Linear
from .recurrent import _f32


class SelectiveScan(Mixer):
    graph_safe = True

    def __init__(self, spec, rt: Runtime):
        self.rt = rt
        self.hidden_size = int(spec["hidden_size"])
        self.C, self.N, self.R, self.taps = int(spec["inner"]), int(spec["state"]), int(spec["dt_rank"]), int(spec["conv"])
        if not 1 <= self.taps <= 16:
            raise ValueError(f"conv must be between 1 and 16 taps, got {self.taps}")
        if not 1 <= self.N <= 256:
            raise ValueError(f"state must be between 1 and 256, got {self.N}")
        self.s_floats = self.C * self.N
        # W_x's rows as the kernels want them: d padded to whole runs of 8 (16 bytes), then B and C, the whole to runs of 8
        self.R_pad = -(-self.R // 8) * 8
        self.p_width = -(-(self.R_pad + 2 * self.N) // 8) * 8

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        h, C, N, R = self.hidden_size, self.C, self.N, self.R
        return {"in": TensorSpec((2 * C, h)), "conv": TensorSpec((C, self.taps)), "conv.b": TensorSpec((C,)),
                "x": TensorSpec((R + 2 * N, C)), "dt": TensorSpec((C, R)), "dt.b": TensorSpec((C,)),
                "A_log": TensorSpec((C, N)), "D": TensorSpec((C,), "ones_plus_normal"), "o": TensorSpec((h, C))}

    def load(self, t: Mapping[str, torch.Tensor]) -> None:
        dt, R, N = self.rt.dtype, self.R, self.N
        self.proj = Linear(t["in"], self.rt)
        wx = torch.zeros((self.p_width, self.C), dtype=dt, device=t["x"].device)
        wx[:R] = t["x"][:R].to(dt)
        wx[self.R_pad:self.R_pad + 2 * N] = t["x"][R:].to(dt)
        self.x = Linear(wx, self.rt, narrow=True)
        wdt = torch.zeros((self.C, self.R_pad), dtype=dt, device=t["dt"].device)
        wdt[:, :R] = t["dt"].to(dt)
        self.dt = Linear(wdt, self.rt)
        self.dt_b = _f32(t["dt.b"])
        self.taps_t = _f32(t["conv"].to(torch.float32).t())
        self.conv_b, self.D = _f32(t["conv.b"]), _f32(t["D"])
        # bfloat16 runs form a decay by one exponential to the base 2
        self.A2 = _f32(-torch.exp(t["A_log"].to(torch.float32)) * (math.log2(math.e) if dt == torch.bfloat16 else 1.0))
        self.o = Linear(t["o"], self.rt)

    def cache_request(self) -> StateRequest:
        return StateRequest((self.s_floats + self.taps * self.C,), torch.float32)

    def weight_bytes(self) -> int:
        return (self.proj.nbytes() + self.x.nbytes() + self.dt.nbytes() + self.o.nbytes()
                + 4 * (self.A2.numel() + self.taps_t.numel()))

    def forward(self, xn, residual, ctx: StepContext, cache_view, writes_cache: bool) -> None:
        rt, ws, T, C = self.rt, self.rt.workspace, ctx.n_tokens, self.C
        state = cache_view.state
        xz = ws.take("scan.xz", (T, 2 * C), rt.dtype)
        self.proj.apply(xn, xz, T, ctx.stream)
        u = ws.take("scan.u", (T, C), rt.dtype)
        B.selective_conv(xz, self.taps_t, self.conv_b, state, self.s_floats, u, C, self.taps, ctx.batch, ctx.stream)
        p = ws.take("scan.p", (T, self.p_width), rt.dtype)
        self.x.apply(u, p, T, ctx.stream)
        dt = ws.take("scan.dt", (T, C), torch.float32)
        self.dt.apply(p[:, :self.R_pad], dt, T, ctx.stream)
        out = ws.take("scan.out", (T, C), rt.dtype)
        B.selective_scan(u, dt, self.dt_b, p[:, self.R_pad:], xz[:, C:], self.A2, self.D, state, 0, out, C, self.N, ctx.kind == "decode",
                         ctx.batch, ctx.stream)
        self.o.apply(out, residual, T, ctx.stream, add_residual=True, ctx=ctx)


register_part("mixer", "selective_scan", SelectiveScan)
