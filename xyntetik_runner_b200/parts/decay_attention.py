"""Linear attention with decays as a mixer with a fixed-size state per request.

With h the mixer's input, H heads, key size D and value size V:
    q = f(W_q h),  k = f(W_k h),  v = f(W_v h)                                laid out head by head; f SiLU, or nothing
    S <- diag(a) S + k v^T,   o = c S^T q                                     S [D, V] per head, c a constant
    y = W_o (norm(o) * g(W_g h)) * out_scale                                  g the sigmoid, or SiLU
Two mixers, which differ in the decays a:

* ``DecayLinearAttention``: a constant per head ("lightning attention", "retention").
* ``KeyDecayLinearAttention``: a number per key channel and token ("gated linear attention"),
  a = sigmoid(z)^(1/tau), z = W_a2 (W_a1 h) + b, through a narrow middle whose size the checkpoint gives.

`norm`: "row" is one RMS norm over all heads together with a weight of H V values; "head" one per head with one weight of V values for
all heads; "unit" one per head without a weight.  S starts at zero and lives in float32 in the request's state slot.  The projections
leave their product in float32; the activations, the decays, the recurrence, the norm and the gate are float32 in both precisions
(csrc/recurrent.cu).  The state after a token does not depend on how tokens were cut into steps.
"""
from __future__ import annotations

from typing import Sequence

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Mixer, StateNeed, register_mixer
from .linear import Linear


class _LinearAttention(Mixer):
    """Everything but the decays and the walk."""
    graph_safe = True

    def __init__(self, width: int, heads: int, dim: int, vdim: int, eps: float, prefix: str, out_scale: float = 1.0, q: str = "q",
                 k: str = "k", v: str = "v", g: str = "g", o: str = "o", norm: str = "row", norm_name: str = "norm", gate: str = "sigmoid",
                 read_scale: float = 1.0):
        if dim > 256:
            raise ValueError(f"{prefix}: key size {dim}: the recurrence kernel takes up to 256")
        if norm not in ("row", "head", "unit") or gate not in ("sigmoid", "silu") or (norm == "row" and gate != "sigmoid"):
            raise ValueError(f"{prefix}: norm is 'row' (with a sigmoid gate), 'head' or 'unit', gate 'sigmoid' or 'silu'")
        self.width, self.H, self.D, self.V = width, heads, dim, vdim
        self.eps, self.prefix, self.out_scale, self.read_scale = float(eps), prefix, float(out_scale), float(read_scale)
        self.norm, self.gate = norm, gate
        self.names = {a: prefix + b for a, b in dict(q=q, k=k, v=v, g=g, o=o, norm=norm_name).items()}
        self.proj = self.out = self.norm_w = None

    def state_need(self):
        return StateNeed((self.H * self.D * self.V,), torch.float32)

    def projected(self):
        """Names of the matrices that make up the projection, in the order of its columns."""
        return [self.names[a] for a in ("q", "k", "v", "g")]

    def tensors(self):
        n, H, D, V, W = self.names, self.H, self.D, self.V, self.width
        t = {n["q"]: TensorSpec((H * D, W)), n["k"]: TensorSpec((H * D, W)), n["v"]: TensorSpec((H * V, W)),
             n["g"]: TensorSpec((H * V, W)), n["o"]: TensorSpec((W, H * V))}
        if self.norm != "unit":
            t[n["norm"]] = TensorSpec((H * V if self.norm == "row" else V,), "vector", "ones_jitter")
        return t

    def bind(self, tensors, rt):
        ws = [tensors.pop(name) for name in self.projected()]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.to(torch.float32) for w in ws]
        self.proj = Linear(torch.cat(ws, dim=0)).prepare(rt)
        del ws
        self.out = Linear(tensors[self.names["o"]]).prepare(rt)
        if self.norm != "unit":
            self.norm_w = tensors[self.names["norm"]].to(torch.float32).contiguous()

    def weight_bytes(self):
        return self.proj.nbytes() + self.out.nbytes()

    def walk(self, ctx, proj, cols, lay, o) -> None:
        raise NotImplementedError

    def forward(self, ctx, h, x, lay):
        n, H, D, V = h.shape[0], self.H, self.D, self.V
        total = self.proj.n_out
        proj = ctx.buf("decay_proj", (n, -(-total // 8) * 8), torch.float32)[:, :total]
        self.proj.forward(h, proj)
        o = ctx.buf("decay_o", (n, H * V), torch.float32)
        self.walk(ctx, proj, (0, H * D, 2 * H * D), lay, o)
        y = ctx.buf("decay_out", (n, H * V), ctx.act_dtype)
        g = 2 * H * D + H * V
        if self.norm == "row":
            kernels.row_norm_gate(o, proj, g, self.norm_w, y, self.eps)
        else:
            kernels.head_norm_gate(o, proj, g, self.norm_w, y, H, V, self.eps, silu=self.gate == "silu")
        ctx.set_pending(x, self.out.forward(y, x, accumulate=True, defer=True, alpha=self.out_scale))


class DecayLinearAttention(_LinearAttention):
    def __init__(self, width: int, heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float, prefix: str,
                 activation: str = "silu", **options):
        super().__init__(width, heads, dim, vdim, eps, prefix, **options)
        if len(decay) != heads:
            raise ValueError(f"{prefix}: {len(decay)} decays for {heads} heads")
        if activation not in ("silu", "none"):
            raise ValueError(f"{prefix}: activation is 'silu' or 'none'")
        self.decay_values, self.silu, self.decay = [float(d) for d in decay], activation == "silu", None

    def bind(self, tensors, rt):
        super().bind(tensors, rt)
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=rt.device)

    def walk(self, ctx, proj, cols, lay, o):
        kernels.decay_attention(proj, cols, self.decay, lay.state, ctx.seg_start, ctx.seg_len, ctx.seg_slot, o, ctx.n_seg, self.H, self.D,
                                self.V, silu=self.silu, read_scale=self.read_scale)


class KeyDecayLinearAttention(_LinearAttention):
    def __init__(self, width: int, heads: int, dim: int, vdim: int, tau: float, eps: float, prefix: str, a1: str = "a1", a2: str = "a2",
                 bias_suffix: str = ".b", norm: str = "head", gate: str = "silu", **options):
        super().__init__(width, heads, dim, vdim, eps, prefix, norm=norm, gate=gate, **options)
        if not tau > 0:
            raise ValueError(f"{prefix}: tau {tau}")
        self.tau, self.inner = float(tau), None
        self.names.update(a1=prefix + a1, a2=prefix + a2, a2b=prefix + a2 + bias_suffix)
        self.a2_t = self.a2_b = None

    def projected(self):
        # the decays' narrow middle rides in the same product, behind the gate
        return super().projected() + [self.names["a1"]]

    def tensors(self):
        n, C = self.names, self.H * self.D
        t = super().tensors()
        # (the size of the middle comes from the checkpoint; random weights take 16)
        t.update({n["a1"]: TensorSpec((16, self.width), any_rows=True), n["a2"]: TensorSpec((C, 16), any_cols=True),
                  n["a2b"]: TensorSpec((C,), "vector", "zeros")})
        return t

    def bind(self, tensors, rt):
        n = self.names
        self.inner = tensors[n["a1"]].shape[0]
        a2 = tensors[n["a2"]].to(torch.float32)
        if a2.shape[1] != self.inner:
            raise ValueError(f"{n['a2']} is {list(a2.shape)}, but {n['a1']} has {self.inner} rows")
        super().bind(tensors, rt)
        self.a2_t = a2.t().contiguous()
        self.a2_b = tensors[n["a2b"]].to(torch.float32).contiguous()

    def weight_bytes(self):
        return super().weight_bytes() + (self.a2_t.numel() + self.a2_b.numel()) * 4

    def walk(self, ctx, proj, cols, lay, o):
        H, D, V = self.H, self.D, self.V
        decays = ctx.buf("decay_keys", (proj.shape[0], H * D), torch.float32)
        kernels.key_decay_attention(proj, cols + (2 * H * D + 2 * H * V,), self.inner, self.a2_t, self.a2_b, self.tau, decays, lay.state,
                                    ctx.seg_start, ctx.seg_len, ctx.seg_slot, o, ctx.n_seg, H, D, V, read_scale=self.read_scale)


register_mixer("decay_linear_attention", DecayLinearAttention)
register_mixer("key_decay_linear_attention", KeyDecayLinearAttention)
