"""The Lilalorn decoder as a list of parts chosen from its configuration.

Fixed by the design: pre-norm layers with two residual additions and weighted RMS norms; rotations pair element i with i + dims/2; no
biases but the decays'; retention without activations on queries, keys and values, keys times dim^(-1/2), heads divided by their root
mean square and a SiLU gate; gated linear attention with queries times dim^(-1/2), one norm weight for all heads and a SiLU gate;
experts of two matrices with the square of relu between them, chosen by a softmax over all experts and weighted by the chosen scores
over their sum; a shared expert of the same form under a sigmoid of one number per token.  Both scalings by dim^(-1/2) are taken on
the read-outs, which is the same.  Everything else -- sizes, the order and kinds of the layers, which layers share tensors, the
rotation, scales, decays, tau, multipliers -- comes from the configuration, the decays' inner size from the tensor's shape.
Tensor names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""
from __future__ import annotations

from ..config.lilalorn import NAME, GatedLinearConfig, LilalornConfig, ParallelConfig
from ..config.llama import RopeScaling
from ..config.registry import register_architecture
from ..engine.model import ModelPlan, ScheduleEntry
from ..parts import (MLP, DecayLinearAttention, Embedding, GQAAttention, Head, KeyDecayLinearAttention, NoPosition, PreNormBlock, RMSNorm, Rope,
                     RoutedExperts, SideBySide)

# no position table limits a request's length: the rotation takes any position and the recurrences have none
MAX_POSITIONS = 1 << 30


def _softmax_side(W, m, prefix, out_scale):
    sc = m.rot.scaling
    scaling = None if sc is None else RopeScaling(rope_type="llama3", factor=sc.factor, low_freq_factor=sc.low, high_freq_factor=sc.high,
                                                  original_max_position_embeddings=sc.original)
    position = Rope(m.dim, m.rot.base, rotary_dim=m.rot.dims, scaling=scaling) if m.rot.dims else NoPosition()
    return GQAAttention(W, m.heads, m.kv_heads, m.dim, position=position, prefix=prefix, scale=m.scale, q="q", k="k", v="v", o="o",
                        weight_suffix="", value_dim=m.vdim, exact_angles=True, out_scale=out_scale)


def _mixer(W, m, eps, prefix, mult):
    """The mixer, with the stream's multiplier in its output scale."""
    if isinstance(m, ParallelConfig):
        r = m.right
        return SideBySide(_softmax_side(W, m.left, prefix + "left.", m.left_scale * mult),
                          DecayLinearAttention(W, r.heads, r.dim, r.vdim, r.decay, eps, prefix=prefix + "right.", activation="none", norm="unit",
                                               gate="silu", read_scale=r.dim ** -0.5, out_scale=m.right_scale * mult))
    if isinstance(m, GatedLinearConfig):
        return KeyDecayLinearAttention(W, m.heads, m.dim, m.vdim, m.tau, eps, prefix=prefix, read_scale=m.dim ** -0.5, out_scale=mult)
    raise ValueError(f"{prefix}: unknown mixer configuration {type(m).__name__}")


def build_lilalorn(cfg: LilalornConfig) -> ModelPlan:
    W, eps, mult = cfg.width, cfg.norm_eps, cfg.residual_mult
    blocks, at = [], {}
    for i, lay in enumerate(cfg.layers):
        if cfg.owner(i) != i:
            continue
        p, f = f"l{i}.", lay.mlp
        norm1, mixer = RMSNorm(W, eps, p + "norm1"), _mixer(W, lay.mixer, eps, p + "mix.", mult)
        at[i] = len(blocks)
        if f is None:
            blocks.append(PreNormBlock(norm1, mixer, spare_norm=p + "norm2"))
            continue
        shared = None if f.shared_ff is None else MLP(W, f.shared_ff, p + "mlp.shared.", "relu2", up="up", down="down")
        ff = RoutedExperts(W, f.experts, f.top, f.ff, p + "mlp.", activation="relu2", gate=None, shared=shared,
                           shared_gate=None if shared is None else "shared.sg", out_scale=mult)
        blocks.append(PreNormBlock(norm1, mixer, RMSNorm(W, eps, p + "norm2"), ff))
    # a layer that uses another one's tensors runs that block again, with a cache entry and a state of its own
    schedule = [ScheduleEntry(layer=at[cfg.owner(i)]) for i in range(len(cfg.layers))]
    return ModelPlan(embedding=Embedding(cfg.vocab, W, "embed"), blocks=blocks, schedule=schedule, final_norm=RMSNorm(W, eps, "final.norm"),
                     head=Head(cfg.vocab, W, name="head", scale=cfg.logit_scale), width=W, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS)


register_architecture(NAME, LilalornConfig.from_dict, build_lilalorn, replace=True)
