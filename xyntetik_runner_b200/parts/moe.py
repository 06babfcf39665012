"""Routed experts with an optional shared expert.

    z = W_router h (float32);  the `top` experts with the largest z;  weights = softmax over the chosen z alone
    out = out_scale * (sum_j weight_j * expert_{e_j}(h)  (+ shared(h), or sigmoid(w_sg h) shared(h)))
    expert(h) = W_down gate_act(W_gate h, W_up h), no biases; or with `gate` None  W_down act(W_up h)
The softmax over the chosen z is also what the chosen scores of a softmax over all experts, divided by their sum, come to.
`shared_gate` names the one-row matrix w_sg: its row rides in the router's product, and the shared expert (an ungated ``MLP``) leaves
its product, or the partial sums of it, to the kernel that adds the experts' outputs.  That kernel is left to the next norm where
nothing else adds to the stream behind it (``PendingExperts``): the sum, the stream and the norm are then one pass.
With ``scoring="softmax_all"`` the scores are s = softmax(z) over all outputs of the router, which may have `identity` outputs
more than there are experts: these identity experts take part in the choice like the others, their output is h itself, and
they have no tensors.  The choice goes by s + correction; `groups=(count, keep)` splits the outputs into `count` equal groups of
neighbours of which only the `keep` with the largest s + correction can be chosen from; the weights are s * `scale`, not
renormalised.  With ``scoring="sigmoid"`` the scores are s = sigmoid(z); the `top` largest s + correction are chosen (`correction`: a tensor of
one number per expert, or None) and the weights are the chosen experts' s, not renormalised.
The activation is one of ``kernels.ACTIVATIONS`` (with its `limit` where it has one).  Experts' matrices are kept as
[experts, rows, columns] arrays; the (token, choice) pairs are put in the order of their experts on the device and every
expert multiplies the rows that chose it (csrc/moe.cu), so no step waits for the host.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import FeedForward, register_feed_forward
from .feed_forward import GatedFeedForward, MLP, _act_id
from . import linear_tc
from .linear import Linear


class PendingExperts:
    """The weighted sum of a step's expert outputs (and of the shared expert's), still to be added into x: by ``finish``, or by the
    norm that follows, in one pass with it."""

    def __init__(self, x: torch.Tensor, args: tuple, options: dict, slab=None):
        self.x, self.args, self.options, self.slab = x, args, options, slab

    def _release(self) -> None:
        if self.slab is not None:
            self.slab.release()

    def finish(self) -> None:
        kernels.moe_combine(self.x, *self.args, **self.options)
        self._release()

    def finish_norm(self, x, w, out, eps, w2=None, out2=None) -> None:
        if w2 is not None:
            self.finish()
            kernels.rmsnorm(x, w, out, eps, None, w2, out2)
            return
        kernels.moe_combine(self.x, *self.args, norm_w=w, out=out, eps=eps, **self.options)
        self._release()


class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, width: int, experts: int, top: int, inner: int, prefix: str, activation: str = "silu",
                 limit: float = 0.0, shared: Optional[FeedForward] = None, router: str = "router",
                 expert: str = "e{}.", gate: Optional[str] = "gate", up: str = "up", down: str = "down", scoring: str = "softmax",
                 correction: Optional[str] = None, identity: int = 0, groups: tuple = (1, 1), scale: float = 1.0,
                 shared_gate: Optional[str] = None, out_scale: float = 1.0):
        if scoring not in ("softmax", "softmax_all", "sigmoid"):
            raise ValueError(f"{prefix}: scoring is 'softmax' (over the chosen logits), 'softmax_all' or 'sigmoid'")
        if correction is not None and scoring == "softmax":
            raise ValueError(f"{prefix}: a correction of the choice goes with sigmoid scores or those of a softmax over all outputs")
        if scoring != "softmax_all" and (identity or tuple(groups) != (1, 1) or float(scale) != 1.0):
            raise ValueError(f"{prefix}: identity experts, groups and a factor on the weights go with scoring='softmax_all'")
        count, keep = (int(g) for g in groups)
        outputs = experts + int(identity)
        if count < 1 or outputs % count or not (1 <= keep <= count):
            raise ValueError(f"{prefix}: {outputs} outputs of the router in {count} groups of which {keep} are kept")
        if not (1 <= top <= keep * (outputs // count)):
            raise ValueError(f"{prefix}: top {top} of {keep * (outputs // count)} experts that can be chosen")
        if shared_gate is not None and (not isinstance(shared, MLP) or scoring == "softmax_all"):
            raise ValueError(f"{prefix}: a gated shared expert is an ungated feed-forward, and goes with a choice that reads strided rows")
        if shared is not None and shared_gate is None and float(out_scale) != 1.0:
            raise ValueError(f"{prefix}: a shared expert that adds into the stream itself goes without a factor on the output")
        if gate is None and activation == "swish_clamp":
            raise ValueError(f"{prefix}: swish_clamp is an activation of gated experts")
        self.width, self.E, self.top, self.inner, self.prefix = width, experts, top, inner, prefix
        self.act, self.limit, self.shared = _act_id(activation), float(limit), shared
        self.router_name = prefix + router
        self.outputs, self.groups, self.scale, self.softmax_all = outputs, (count, keep), float(scale), scoring == "softmax_all"
        self.sigmoid, self.correction_name, self.correction = scoring == "sigmoid", None if correction is None else prefix + correction, None
        self.gated, self.out_scale = gate is not None, float(out_scale)
        self.shared_gate_name = None if shared_gate is None else prefix + shared_gate
        # an expert's matrices: (gate, up, down), or (up, down)
        kinds = ((gate,) if self.gated else ()) + (up, down)
        self.expert_names = [tuple(prefix + expert.format(e) + s for s in kinds) for e in range(experts)]
        self.router = self.w_gate_up = self.w_down = None
        self.tensor_cores, self._nbytes = False, 0

    def tensors(self):
        t = {self.router_name: TensorSpec((self.outputs, self.width))}
        if self.correction_name is not None:
            t[self.correction_name] = TensorSpec((self.outputs,), "vector", "zeros")
        if self.shared_gate_name is not None:
            t[self.shared_gate_name] = TensorSpec((1, self.width))
        for names in self.expert_names:
            for first in names[:-1]:
                t[first] = TensorSpec((self.inner, self.width))
            t[names[-1]] = TensorSpec((self.width, self.inner))
        if self.shared is not None:
            t.update(self.shared.tensors())
        return t

    def bind(self, tensors, rt):
        router = tensors[self.router_name]
        if self.shared_gate_name is not None:
            sg = tensors[self.shared_gate_name]
            both = router.dtype if router.dtype == sg.dtype else torch.float32
            router = torch.cat([router.to(both), sg.to(both)], dim=0)
        self.router = Linear(router).prepare(rt)
        if self.correction_name is not None:
            self.correction = tensors[self.correction_name].to(torch.float32).contiguous()
        ws = [tensors.pop(n) for names in self.expert_names for n in names]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.to(torch.float32) for w in ws]
        # [E][2F][width]: an expert's gate rows, then its up rows ([E][F][width] without a gate); [E][width][F]
        m = len(ws) // self.E
        gate_up = torch.stack([torch.cat(ws[m * e:m * e + m - 1], dim=0) for e in range(self.E)]).contiguous()
        down = torch.stack([ws[m * e + m - 1] for e in range(self.E)]).contiguous()
        del ws
        self._nbytes = (gate_up.numel() + down.numel()) * down.element_size()
        # bfloat16 serving: the tensor-core product over rows sorted by expert, on matrices re-laid tile by tile
        self.tensor_cores = (linear_tc.ENABLED and rt.act_dtype == torch.bfloat16 and down.dtype == torch.bfloat16 and down.is_cuda
                             and self.width % 8 == 0 and self.inner % 8 == 0)
        if self.tensor_cores:
            self.w_gate_up = kernels.pack_weight_groups(gate_up, halves=2 if self.gated else 1)
            self.w_down = kernels.pack_weight_groups(down)
        else:
            self.w_gate_up, self.w_down = gate_up, down
        if self.shared is not None:
            self.shared.bind(tensors, rt)

    def weight_bytes(self):
        # a step reads the router, the shared expert, and at most all experts
        return self.router.nbytes() + self._nbytes + (self.shared.weight_bytes() if self.shared is not None else 0)

    @staticmethod
    def _row_tile(pairs: int, experts: int) -> int:
        """Rows per tile of the tensor-core product: about what an expert gets when the choices spread evenly."""
        avg = pairs / experts
        return 16 if avg <= 16 else (32 if avg <= 32 else (64 if avg <= 64 else 128))

    def forward(self, ctx, h, x):
        n, top, E = h.shape[0], self.top, self.E
        pairs = n * top
        zs = ctx.buf("moe_logits", (n, self.router.n_out), torch.float32)
        self.router.forward(h, zs)
        z = zs if self.router.n_out == self.outputs else zs[:, :self.outputs]        # (a shared expert's gate is one column more)
        ids = ctx.buf("moe_ids", (n, top), torch.int32)
        wts = ctx.buf("moe_weights", (n, top), torch.float32)
        if self.softmax_all:
            kernels.route_groups(z, ids, wts, top, self.correction, *self.groups, self.scale)
        elif self.sigmoid:
            kernels.route_topk(z, ids, wts, top, sigmoid_scores=True, correction=self.correction)
        else:
            kernels.route_topk(z, ids, wts, top)
        align = self._row_tile(pairs, E) if self.tensor_cores else kernels.moe_tile_rows()
        max_tiles = kernels.moe_max_tiles(pairs, E, align)
        rows = max_tiles * align
        row_src = ctx.buf("moe_row_src", (rows,), torch.int32)
        pair_row = ctx.buf("moe_pair_row", (pairs,), torch.int32)
        tile_group = ctx.buf("moe_tile_group", (max_tiles,), torch.int32)
        kernels.moe_plan(ids, row_src, pair_row, tile_group, E, align)
        y = ctx.buf("moe_act", (rows, self.inner), ctx.act_dtype)
        zz = ctx.buf("moe_out", (rows, self.width), torch.float32)
        if self.tensor_cores:
            xs = ctx.buf("moe_rows", (rows, self.width), ctx.act_dtype)
            kernels.moe_gather(h, xs, row_src, tile_group, top, align)
            kernels.gemm_tc_grouped(xs, self.w_gate_up, y, tile_group, align, self.inner, kernels.EPI_GATED if self.gated else kernels.EPI_STORE,
                                    self.act, self.limit)
            kernels.gemm_tc_grouped(y, self.w_down, zz, tile_group, align, self.width)
        else:
            kernels.moe_gemm(h, self.w_gate_up, y, row_src, tile_group, top, self.gated, self.act, self.limit, gather=True)
            kernels.moe_gemm(y, self.w_down, zz, row_src, tile_group, top, False)
        options, slab = dict(h=h if self.outputs > E else None, scale=self.out_scale), None
        if self.shared_gate_name is not None:
            rows = ctx.buf("moe_shared", (n, self.width), torch.float32)
            slab = self.shared.product(ctx, h, rows)
            options.update(shared=rows if slab is None else slab.partial, splits=1 if slab is None else slab.splits, gate=zs[:, self.outputs])
        ctx.set_pending(x, PendingExperts(x, (zz, wts, pair_row, top), options, slab))
        if self.shared is not None and self.shared_gate_name is None:
            ctx.materialize(x)
            self.shared.forward(ctx, h, x)


register_feed_forward("routed_experts", RoutedExperts)
