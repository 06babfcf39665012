"""The Semesun decoder as a list of parts chosen from its configuration.

Fixed by the design: pre-norm layers with two residual additions and weighted RMS norms; attention with a weighted norm on every
query and key head, no rotation and no biases on the projections; the dense feed-forward's square of relu; experts gated as
g sigmoid(1.702 g) (u + 1) on clamped g and u; router scores by a softmax over all outputs, the choice by score plus correction.
Everything else -- sizes, the order and kinds of the layers, windows, kept tokens, scales, the bias's reach, groups, the clamp, the
weights' factor -- comes from the configuration, the number of distance buckets from the table's shape.
Tensor names: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.semesun import NAME, AttentionConfig, DenseConfig, ExpertsConfig, MambaConfig, SemesunConfig
from ..engine.model import ModelPlan, ScheduleEntry
from ..parts import MLP, Embedding, GQAAttention, Head, Mamba2, NoPosition, PreNormBlock, RMSNorm, RoutedExperts

# no position table limits a request's length: positions enter as distances only, and the recurrence has none
MAX_POSITIONS = 1 << 30


def build_semesun(cfg: SemesunConfig) -> ModelPlan:
    W, eps = cfg.width, cfg.norm_eps
    blocks, schedule, shares = [], [], "first"
    for i, lay in enumerate(cfg.layers):
        p = f"l{i}."
        m = lay.mixer
        if isinstance(m, AttentionConfig):
            mixer = GQAAttention(W, m.heads, m.kv_heads, m.dim, position=NoPosition(), prefix=p + "mix.", window=m.window, scale=m.scale,
                                 q="q", k="k", v="v", o="o", weight_suffix="", value_dim=m.vdim, qk_norm=True, norm_eps=eps,
                                 keep_first=m.keep_first, distance_bias=None if m.bias_max is None else ("rel", m.bias_max),
                                 value_share=shares if m.v_mix else None, v_mix="vmix")
            if m.v_mix:
                shares = "mix"            # the first mixing layer leaves its values, every later one mixes them in
        elif isinstance(m, MambaConfig):
            mixer = Mamba2(W, m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups, eps, prefix=p + "mix.")
        else:
            raise ValueError(f"layer {i}: unknown mixer configuration {type(m).__name__}")
        norm1 = RMSNorm(W, eps, p + "norm1")
        if lay.mlp is None:
            blocks.append(PreNormBlock(norm1, mixer, spare_norm=p + "norm2"))
        else:
            if isinstance(lay.mlp, DenseConfig):
                ff = MLP(W, lay.mlp.ff, p + "mlp.", "relu2", up="up", down="down")
            elif isinstance(lay.mlp, ExpertsConfig):
                f = lay.mlp
                ff = RoutedExperts(W, f.experts, f.top, f.ff, p + "mlp.", activation="swish_clamp", limit=f.limit, scoring="softmax_all",
                                   correction="correction", identity=f.identity, groups=(f.group_count, f.group_keep), scale=f.scale)
            else:
                raise ValueError(f"layer {i}: unknown feed-forward configuration {type(lay.mlp).__name__}")
            blocks.append(PreNormBlock(norm1, mixer, RMSNorm(W, eps, p + "norm2"), ff))
        schedule.append(ScheduleEntry(layer=i))
    return ModelPlan(embedding=Embedding(cfg.vocab, W, "embed"), blocks=blocks, schedule=schedule, final_norm=RMSNorm(W, eps, "final.norm"),
                     head=Head(cfg.vocab, W, name="head"), width=W, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS)


register_architecture(NAME, SemesunConfig.from_dict, build_semesun, replace=True)
