"""Mamba-2's mixer (state-space duality) with a fixed-size state per request.

With h the mixer's input, H heads of size V, state size N, G groups of heads that share B and C, a causal convolution of `taps` taps
per channel (the last column of its weight is the current token's, zeros before a request's first token):
    [z | x | B | C | dt'] = W_in h                                                  H V, H V, G N, G N and H rows
    [x | B | C] <- silu(conv([x | B | C]) + bias),   dt = softplus(dt' + dt_bias)
    S <- exp(-exp(A_log_h) dt) S + dt B x^T,   y = S^T C + D_h x                    S [N, V] per head; head h reads group h / (H / G)
    out = W_o (rms_norm(y * silu(z)) * w)                                           over `norm_groups` equal parts of the columns
S starts at zero and lives in float32 in the request's state slot together with the last taps - 1 rows that entered the convolution;
the projection's sums and everything behind them are float32 in both precisions (csrc/recurrent.cu).  The state after a token does not
depend on how tokens were cut into steps.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Mixer, StateNeed, register_mixer
from .linear import Linear


class Mamba2(Mixer):
    graph_safe = True

    def __init__(self, width: int, heads: int, vdim: int, state: int, groups: int, taps: int, norm_groups: int, eps: float, prefix: str,
                 proj: str = "in", conv: str = "conv", conv_bias: str = "conv.b", dt_bias: str = "dt_bias", a_log: str = "A_log", skip: str = "D",
                 norm: str = "norm", o: str = "o"):
        if heads % groups:
            raise ValueError(f"{prefix}: heads must be a multiple of groups")
        if (heads * vdim) % norm_groups:
            raise ValueError(f"{prefix}: {heads * vdim} columns do not divide into {norm_groups} groups of the norm")
        if not (1 <= state <= 256):
            raise ValueError(f"{prefix}: state size {state}: the recurrence kernel takes 1 to 256")
        if not (1 <= taps <= 64):
            raise ValueError(f"{prefix}: the convolution takes 1 to 64 taps")
        self.width, self.H, self.V, self.N, self.G, self.taps = width, heads, vdim, state, groups, taps
        self.norm_groups, self.eps, self.prefix = norm_groups, float(eps), prefix
        self.inner, self.channels = heads * vdim, heads * vdim + 2 * groups * state
        self.rows = self.inner + self.channels + heads
        self.names = {k: prefix + v for k, v in dict(proj=proj, conv=conv, conv_b=conv_bias, dt_bias=dt_bias, a_log=a_log, skip=skip, norm=norm, o=o).items()}
        self.proj = self.out = None

    def state_need(self):
        return StateNeed((kernels.ssd_state_floats(self.H, self.G, self.N, self.V, self.taps),), torch.float32)

    def tensors(self):
        n, H = self.names, self.H
        return {n["proj"]: TensorSpec((self.rows, self.width)), n["conv"]: TensorSpec((self.channels, self.taps), "vector", "normal"),
                n["conv_b"]: TensorSpec((self.channels,), "vector", "zeros"), n["dt_bias"]: TensorSpec((H,), "vector", "zeros"),
                n["a_log"]: TensorSpec((H,), "vector", "zeros"), n["skip"]: TensorSpec((H,), "vector", "ones_jitter"),
                n["norm"]: TensorSpec((self.inner,), "vector", "ones_jitter"), n["o"]: TensorSpec((self.width, self.inner))}

    def bind(self, tensors, rt):
        n = self.names
        f32 = lambda name: tensors[name].to(torch.float32).contiguous()
        self.proj = Linear(tensors[n["proj"]]).prepare(rt)
        self.out = Linear(tensors[n["o"]]).prepare(rt)
        self.conv_w, self.conv_b, self.dt_bias, self.skip, self.norm_w = (f32(n[k]) for k in ("conv", "conv_b", "dt_bias", "skip", "norm"))
        self.neg_a = (-torch.exp(f32(n["a_log"]))).contiguous()

    def weight_bytes(self):
        return self.proj.nbytes() + self.out.nbytes() + self.conv_w.numel() * 4

    def forward(self, ctx, h, x, lay):
        n, inner, H = h.shape[0], self.inner, self.H
        # the projection leaves its product in float32: what enters the convolution and the recurrence is rounded once, at the
        # product's input, and the convolution's tail holds exactly what the rows held
        proj = ctx.buf("ssd_proj", (n, -(-self.rows // 8) * 8), torch.float32)[:, :self.rows]
        self.proj.forward(h, proj)
        xbc = ctx.buf("ssd_xbc", (n, self.channels), torch.float32)
        coef = ctx.buf("ssd_coef", (n, 2 * H), torch.float32)
        y = ctx.buf("ssd_y", (n, inner), torch.float32)
        kernels.ssd(proj, inner, inner + self.channels, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, self.skip, lay.state, ctx.tok_seg,
                    ctx.seg_start, ctx.seg_len, ctx.seg_slot, xbc, coef, y, ctx.n_seg, H, self.G, self.N, self.V, self.taps)
        out = ctx.buf("ssd_out", (n, inner), ctx.act_dtype)
        kernels.silu_gate_norm(y, proj, 0, self.norm_w, out, self.norm_groups, self.eps)
        ctx.set_pending(x, self.out.forward(out, x, accumulate=True, defer=True))


register_mixer("mamba2", Mamba2)
