"""A plain, slow implementation of the Lilalorn decoder: one function per mechanism, whole sequences, no cache.

Everything is computed on the CPU in one dtype (float64 by default) from a configuration dict and a dict of tensors
by name.  It shares no code with the engine: the tests compare the engine's logits with it.

Notation.  x: residual stream [T, width]; h: what a sublayer reads; S: a matrix memory [key channels, value channels] per head.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ---- softmax attention -----------------------------------------------------------------------------------------------
def frequencies(dims: int, base: float, scaling: Optional[dict], dtype) -> torch.Tensor:
    """Turns per position of every pair, in radians: base^(-2i/dims), long wavelengths slowed by `factor`, those between
    original/high and original/low blended."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            turns = scaling["original"] * f / (2.0 * math.pi)           # how often the pair turns over the original length
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=dtype)


def rotate(v: torch.Tensor, positions: torch.Tensor, dims: int, freq: torch.Tensor) -> torch.Tensor:
    """v [T, heads, D]: of the first `dims` elements, i and i + dims/2 are a pair turned by p * freq[i]."""
    if dims == 0:
        return v
    half = dims // 2
    ang = positions.to(v.dtype)[:, None, None] * freq[None, None, :]
    c, s = torch.cos(ang), torch.sin(ang)
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * c - b * s, b * c + a * s, v[..., dims:]], dim=-1)


def softmax_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, V = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    pos = torch.arange(T)
    q, k, v = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, G, D), (h @ w["v"].T).view(T, G, V)
    rot = m.get("rot")
    if rot:
        freq = frequencies(rot["dims"], rot["base"], rot.get("scaling"), h.dtype)
        q, k = rotate(q, pos, rot["dims"], freq), rotate(k, pos, rot["dims"], freq)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(pos[None, None, :] > pos[None, :, None], float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v)
    return o.reshape(T, H * V) @ w["o"].T


# ---- linear attention with decays ------------------------------------------------------------------------------------
def decayed_reads(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """S_t = diag(decay_t) S_(t-1) + k_t v_t^T from zero, o_t = S_t^T q_t.  q, k, decay [T, H, D], v [T, H, V] -> [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(dim=1))
    return torch.stack(out)


def retention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    """A constant decay per head; keys times dim^(-1/2); heads divided by their root mean square; a SiLU gate."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, H, D) * D ** -0.5, (h @ w["v"].T).view(T, H, V)
    decay = torch.tensor(m["decay"], dtype=h.dtype)[None, :, None].expand(T, H, D)
    o = unit_rms(decayed_reads(q, k, v, decay), eps).reshape(T, H * V)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def key_channel_decay(h: torch.Tensor, w: Dict[str, torch.Tensor], tau: float) -> torch.Tensor:
    """A decay per key channel from the token: sigmoid(z)^(1/tau), z a product through a narrow middle plus a bias."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def gated_linear_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, D) * D ** -0.5, (h @ w["k"].T).view(T, H, D), (h @ w["v"].T).view(T, H, V)
    o = decayed_reads(q, k, v, key_channel_decay(h, w, m["tau"]).view(T, H, D))
    o = rms_norm(o, w["norm"], eps).reshape(T, H * V)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    left = softmax_attention(h, _sub(w, "left."), m["left"])
    right = retention(h, _sub(w, "right."), m["right"], eps)
    return m.get("left_scale", 1.0) * left + m.get("right_scale", 1.0) * right


# ---- feed-forward ----------------------------------------------------------------------------------------------------
def relu2_ff(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (torch.relu(h @ up.T) ** 2) @ down.T


def router_scores(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return torch.softmax(h @ w["router"].T, dim=-1)


def routed_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    """The `top` experts with the largest scores, weighted by their scores over their sum, and a shared expert under a gate."""
    s = router_scores(h, w)
    chosen = torch.topk(s, f["router"]["top"], dim=-1).indices
    weight = torch.gather(s, 1, chosen)
    weight = weight / (weight.sum(dim=-1, keepdim=True) + 1e-20)
    out = torch.zeros(h.shape[0], w["e0.down"].shape[0], dtype=h.dtype)
    for e in range(f["router"]["experts"]):
        for t, j in (chosen == e).nonzero().tolist():
            out[t] += weight[t, j] * relu2_ff(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if f.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * relu2_ff(h, w["shared.up"], w["shared.down"])
    return out


# ---- the model -------------------------------------------------------------------------------------------------------
def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def sublayer_input(x: torch.Tensor) -> torch.Tensor:
    """What a sublayer reads: the norm's output itself.  (A test replaces this to see what a rounding here does.)"""
    return x


def owner(layers, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def layer(x: torch.Tensor, tensors: Dict[str, torch.Tensor], p: str, lay: dict, mult: float, eps: float) -> torch.Tensor:
    """x + mult mixer(norm1(x)), then the same with the feed-forward; `p` the prefix of the tensors it uses."""
    mix = {"gla": gated_linear_attention, "parallel": parallel_mixer}[lay["type"]]
    h = sublayer_input(rms_norm(x, tensors[p + "norm1"], eps))
    x = x + mult * mix(h, _sub(tensors, p + "mix."), lay["mixer"], eps)
    f = lay.get("mlp")
    if f:
        h = sublayer_input(rms_norm(x, tensors[p + "norm2"], eps))
        x = x + mult * routed_ff(h, _sub(tensors, p + "mlp."), f)
    return x


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: Optional[List] = None):
    """Logits [T, vocab] of one sequence.  `layers_out` receives the stream after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    x = t["embed"][torch.tensor(list(tokens))]
    for i, lay in enumerate(config["layers"]):
        own = owner(config["layers"], i)
        x = layer(x, t, f"l{own}.", config["layers"][own], mult, eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T * config.get("logit_scale", 1.0)
