"""A plain, slow implementation of the Semesun decoder: one function per mechanism, whole sequences, no cache.

Everything is computed on the CPU in one dtype (float64 by default) from a configuration dict and a dict of tensors
by name.  It shares no code with the engine: the tests compare the engine's logits with it.

Notation.  x: residual stream [T, width]; h: what a sublayer reads; i a query's position, j a key's (both from 0).
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


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# ---- attention -------------------------------------------------------------------------------------------------------
def bucket(distance: int, rows: int, bias_max: float) -> int:
    """Row of the bias table for a distance: the distance itself below rows/2, then logarithmic steps up to `bias_max`."""
    half = rows // 2
    if distance < half:
        return distance
    # (the nudge: a distance right on a step takes it, whatever the logarithms round to)
    return min(rows - 1, half + math.floor(math.log(distance / half) / math.log(bias_max / half) * (rows - half) + 1e-9))


def visible(T: int, mask: Optional[dict]) -> torch.Tensor:
    """[T, T] booleans: a causal window of mask.size positions, and the first mask.keep_first positions of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    if not mask:
        return j <= i
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def distance_bias(T: int, rel: torch.Tensor, bias_max: float) -> torch.Tensor:
    """[heads, T, T]: rel[bucket(i - j), head] below and on the diagonal, zero above."""
    rows = torch.tensor([bucket(n, rel.shape[0], bias_max) for n in range(T)])
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    b = rel[rows[(i - j).clamp(min=0)]]
    return torch.where((j <= i)[..., None], b, torch.zeros((), dtype=rel.dtype)).permute(2, 0, 1)


def mixed_values(v: torch.Tensor, first: Optional[torch.Tensor], lam) -> torch.Tensor:
    """(1 - lambda) v + lambda (the values that the first mixing layer computed for the same token)."""
    return v if first is None else (1.0 - lam) * v + lam * first


def attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, shared: dict) -> torch.Tensor:
    """`shared` carries the first mixing layer's values from layer to layer of one forward pass."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((h @ w["q"].T).view(T, H, D), w["q.norm"], eps)
    k = rms_norm((h @ w["k"].T).view(T, G, D), w["k.norm"], eps)
    v = (h @ w["v"].T).view(T, G, V)
    if m.get("v_mix"):
        if "v_first" not in shared:
            shared["v_first"] = v
        else:
            v = mixed_values(v, shared["v_first"].view(T, G, V), w["vmix"])
    rep = H // G
    k, v = k.repeat_interleave(rep, dim=1), v.repeat_interleave(rep, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] + distance_bias(T, w["rel"], m["bias_max"])
    s = s.masked_fill(~visible(T, m.get("mask"))[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v).reshape(T, H * V) @ w["o"].T


# ---- state-space duality ---------------------------------------------------------------------------------------------
def causal_conv(z: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """z [T, C], taps [C, K]: out[t] = bias + sum_j taps[:, K-1-j] z[t-j], zeros before the start."""
    T, K = z.shape[0], taps.shape[1]
    out = bias.expand(T, -1).clone()
    for j in range(min(K, T)):
        out[j:] += taps[:, K - 1 - j] * (z[:T - j] if j else z)
    return out


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """silu(z) first, then every one of `groups` equal parts divided by its own root mean square, then the weight."""
    g = y * silu(z)
    return unit_rms(g.view(g.shape[0], groups, -1), eps).reshape(g.shape) * weight


def mamba2(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float, shared: dict) -> torch.Tensor:
    T = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, G * N, G * N], dim=-1)
    x, B, C = x.view(T, H, V), B.view(T, G, N), C.view(T, G, N)
    dt = softplus(dt + w["dt_bias"])
    a = torch.exp(-torch.exp(w["A_log"]) * dt)
    S = torch.zeros(H, N, V, dtype=h.dtype)
    ys = []
    for t in range(T):
        b, c = B[t].repeat_interleave(H // G, dim=0), C[t].repeat_interleave(H // G, dim=0)
        S = a[t][:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        ys.append((torch.einsum("hnv,hn->hv", S, c) + w["D"][:, None] * x[t]).reshape(-1))
    return gated_group_norm(torch.stack(ys), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


# ---- feed-forwards ---------------------------------------------------------------------------------------------------
def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def expert_ff(h: torch.Tensor, gate, up, down, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def choice_scores(h: torch.Tensor, w: Dict[str, torch.Tensor], r: dict):
    """(scores s, what the choice goes by: s plus the correction, minus infinity outside the best groups)."""
    s = torch.softmax(h @ w["router"].T, dim=-1)
    c = s + w["correction"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    per = c.shape[1] // g["count"]
    best = torch.topk(c.view(-1, g["count"], per).max(dim=-1).values, g["keep"], dim=-1).indices
    allowed = torch.zeros(c.shape[0], g["count"], dtype=torch.bool).scatter_(1, best, True).repeat_interleave(per, dim=1)
    return s, c.masked_fill(~allowed, float("-inf"))


def routing(h: torch.Tensor, w: Dict[str, torch.Tensor], r: dict):
    """(chosen outputs of the router [T, top], their weights)."""
    s, c = choice_scores(h, w, r)
    chosen = torch.topk(c, r["top"], dim=-1).indices
    return chosen, torch.gather(s, 1, chosen) * r.get("scale", 1.0)


def routed_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], f: dict) -> torch.Tensor:
    r = f["router"]
    chosen, weight = routing(h, w, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t].tolist(), weight[t]):
            y = h[t] if e >= r["experts"] else expert_ff(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"], f["expert"]["limit"])
            out[t] += c * y
    return out


# ---- the model -------------------------------------------------------------------------------------------------------
def _sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def sublayer_input(h: torch.Tensor) -> torch.Tensor:
    """What a sublayer reads behind its norm.  (A test replaces this to see what a rounding here does.)"""
    return h


def layer(x: torch.Tensor, tensors: Dict[str, torch.Tensor], i: int, lay: dict, eps: float, shared: dict) -> torch.Tensor:
    mix = {"attention": attention, "mamba2": mamba2}[lay["type"]]
    x = x + mix(sublayer_input(rms_norm(x, tensors[f"l{i}.norm1"], eps)), _sub(tensors, f"l{i}.mix."), lay["mixer"], eps, shared)
    f = lay.get("mlp")
    if f:
        ff = dense_ff if f["kind"] == "dense" else routed_ff
        x = x + ff(sublayer_input(rms_norm(x, tensors[f"l{i}.norm2"], eps)), _sub(tensors, f"l{i}.mlp."), f)
    return x


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: Optional[List] = None):
    """Logits [T, vocab] of one sequence.  `layers_out` receives the stream after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][torch.tensor(list(tokens))]
    shared = {}
    for i, lay in enumerate(config["layers"]):
        x = layer(x, t, i, lay, eps, shared)
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T
