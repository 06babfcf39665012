"""Small Lilalorn configurations with random weights for the tests, as config.json + model.safetensors folders.

The sizes are awkward on purpose: widths that are no multiple of 8, one head, key sizes that differ from value sizes (and one that
equals it) and are no multiple of 16, as many key heads as heads and fewer, rotations over part of a head, the whole head and none of
it, with and without a frequency scaling whose three ranges all occur, decays from fast to none, narrow middles of one row and many,
roots of several degrees (and of one), routers of which all or few outputs are chosen, shared experts as wide as the others, wider,
narrower and absent, layers without a feed-forward, layers that use another layer's tensors (one through another, one ahead of it),
models of one kind of layer alone.
"""
import copy
import json
import os

import numpy as np
import torch


def softmax_side(heads, kv_heads, dim, vdim, scale, rot_dims, base=10000.0, scaling=None):
    """scaling: (factor, low, high, original), or None."""
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rot}


def retention_side(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def gla(heads, dim, vdim, tau, rank):
    """`rank`: rows of the decays' narrow middle (a size that only the tensors' shapes give)."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "_rank": rank}


def moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        d["shared"] = {"ff": shared}
    return d


def layer(mixer, mlp):
    d = dict(mixer)
    d["mlp"] = mlp
    return d


def again(lay, j):
    """A layer that uses the tensors of layer j (an equal one)."""
    d = copy.deepcopy(lay)
    d["weights_of"] = j
    return d


def model(vocab, width, eps, layers, mult=1.0, logit_scale=1.0):
    return {"architecture": "Lilalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale,
            "layers": layers}


_P = layer(parallel(softmax_side(4, 2, 24, 16, 0.21, 16, 5000.0, (6.0, 1.0, 5.0, 40)), retention_side(3, 10, 12, (0.9, 0.99, 0.6)), 0.8, 1.3), moe(7, 3, 24, 40))
_G = layer(gla(3, 20, 14, 7.0, 5), moe(6, 2, 16, 16))
_G1 = layer(gla(1, 9, 30, 1.0, 1), moe(4, 4, 12, 12))

CONFIGS = {
    # both mixers; tensors used again by a later layer, through a layer that does so itself, and with another layer in between
    "mix": model(211, 96, 1e-5, [
        _P, _G,
        layer(parallel(softmax_side(6, 2, 12, 16, 0.3, 12), retention_side(2, 24, 8, (1.0, 0.97)), -0.5, 0.7), moe(6, 1, 16, 8)),
        again(_G, 1), layer(gla(2, 16, 16, 3.0, 12), None), again(_P, 0), again(_G, 3)], 0.6, 1.7),
    # a width that is no multiple of 8; one head; gated linear attention first; a layer ahead of the one whose tensors it uses; no shared
    # expert; no rotation; no multipliers
    "odd": model(131, 68, 1e-6, [
        again(_G1, 2),
        layer(parallel(softmax_side(1, 1, 18, 6, 0.2, 18, 300.0, (3.0, 0.5, 2.0, 24)), retention_side(1, 5, 7, (0.95,)), 1.1, 0.4), moe(3, 2, 20)),
        _G1,
        layer(parallel(softmax_side(5, 5, 10, 10, 0.4, 0), retention_side(2, 33, 6, (0.8, 0.999)), 0.9, 1.2), None)]),
    # sizes that the tensor-core kernels take (heads of 64 and 128, pages of 64)
    "tc": model(160, 128, 1e-5, [
        layer(parallel(softmax_side(4, 2, 64, 64, 0.12, 64, 100000.0, (8.0, 1.0, 4.0, 128)), retention_side(2, 64, 64, (0.97, 0.99)), 0.7, 0.9), moe(8, 2, 64, 96)),
        layer(gla(2, 64, 128, 16.0, 16), moe(12, 3, 32, 32)),
        layer(parallel(softmax_side(16, 2, 64, 48, 0.15, 32, 20000.0), retention_side(4, 32, 48, (0.9, 0.95, 0.98, 0.995)), 1.2, 0.8), moe(4, 4, 64, 128)),
        layer(gla(1, 130, 72, 10.0, 24), moe(8, 1, 40, 64)),
        layer(parallel(softmax_side(2, 1, 128, 128, 0.09, 64), retention_side(1, 128, 128, (0.985,)), 0.6, 1.1), None)], 0.45, 0.5),
    # gated linear attention alone (no keys are cached at all)
    "rec": model(90, 64, 1e-5, [layer(gla(4, 16, 16, 12.0, 7), moe(5, 2, 24, 24)), layer(gla(2, 40, 24, 5.0, 70), None)], 0.9, 1.2),
}
# (drawn so that no head's read-out at a request's first token nearly cancels: its unit norm would turn float32 rounding into 1e-4)
SEEDS = {"mix": 64, "odd": 60, "tc": 61, "rec": 66}


def clean(cfg):
    """The configuration as config.json has it (without the notes that only the tensors' shapes need)."""
    d = dict(cfg)
    d["layers"] = [{k: v for k, v in lay.items() if not k.startswith("_")} for lay in cfg["layers"]]
    return d


def shapes(cfg):
    """Tensor names and shapes of a configuration."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "final.norm": (W,), "head": (cfg["vocab"], W)}
    for i, lay in enumerate(cfg["layers"]):
        if lay.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", lay["mixer"]
        out.update({p + "norm1": (W,), p + "norm2": (W,)})
        if lay["type"] == "parallel":
            l, r = m["left"], m["right"]
            q = p + "mix.left."
            out.update({q + "q": (l["heads"] * l["dim"], W), q + "k": (l["kv_heads"] * l["dim"], W), q + "v": (l["kv_heads"] * l["vdim"], W),
                        q + "o": (W, l["heads"] * l["vdim"])})
            q, HD, HV = p + "mix.right.", r["heads"] * r["dim"], r["heads"] * r["vdim"]
            out.update({q + "q": (HD, W), q + "k": (HD, W), q + "v": (HV, W), q + "g": (HV, W), q + "o": (W, HV)})
        else:
            HD, HV, R, q = m["heads"] * m["dim"], m["heads"] * m["vdim"], lay["_rank"], p + "mix."
            out.update({q + "q": (HD, W), q + "k": (HD, W), q + "v": (HV, W), q + "g": (HV, W), q + "o": (W, HV), q + "norm": (m["vdim"],),
                        q + "a1": (R, W), q + "a2": (HD, R), q + "a2.b": (HD,)})
        f = lay.get("mlp")
        if f:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            out[p + "mlp.router"] = (E, W)
            for e in range(E):
                out.update({p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
            if f.get("shared"):
                out.update({p + "mlp.shared.up": (f["shared"]["ff"], W), p + "mlp.shared.down": (W, f["shared"]["ff"]), p + "mlp.shared.sg": (1, W)})
    return out


def draw(cfg, seed, dtype=torch.bfloat16, slow=False):
    """Random tensors: matrices N(0, 1/fan_in), norms around one, routers large enough that choices differ between
    tokens, shared experts' gates over a wide range, decays over a wide range (`slow`: all near one, so that the first tokens
    still count hundreds of tokens later)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        r = lambda: torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t = 1.0 + 0.2 * r()
        elif name.endswith("a2.b"):
            t = 4.0 + 0.3 * r() if slow else 1.0 + 2.0 * r()
        elif name.endswith(".a2") and slow:
            t = 0.3 * r() / shape[-1] ** 0.5
        elif name.endswith("router"):
            t = 4.0 * r() / shape[-1] ** 0.5
        elif name.endswith("shared.sg"):
            t = 2.0 * r() / shape[-1] ** 0.5
        elif ".mlp.e" in name and name.endswith(".down"):
            t = 0.4 * r() / shape[-1] ** 0.5             # (a router's near tie that falls the other way swaps whole experts)
        elif name == "embed":
            t = r()
        else:
            t = r() / max(shape[-1], 1) ** 0.5
        out[name] = t.to(dtype)
    return out


def make_folder(path, name, tensors=None, cfg=None, slow=False):
    """Write config.json + model.safetensors (bfloat16) for configuration `name` (or `cfg`); returns (path, cfg, tensors)."""
    from xyntetik_runner_b200.weights.safetensors_io import write_safetensors
    cfg = cfg or CONFIGS[name]
    tensors = tensors if tensors is not None else draw(cfg, SEEDS.get(name, 1), slow=slow)
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"), list(tensors.items()), metadata={"format": "pt"})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(clean(cfg), f, indent=1)
    return path, cfg, tensors


def plain_logits(cfg, tensors, tokens):
    import plain_lilalorn
    return plain_lilalorn.forward(cfg, tensors, tokens, dtype=torch.float64).to(torch.float32).numpy()


def plain_greedy(cfg, tensors, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(plain_logits(cfg, tensors, toks)[-1])))
    return toks[len(prompt):]


NEAR_TIE = 0.02        # scores closer than this may change places under bfloat16 rounding of what the router reads


def near_tie_sensitivity(cfg, tensors, tokens, ref, at=(), most=32):
    """What a change of places does to every position's logits, for the (layer, position) pairs where the last chosen expert of a router
    and the first one left out have scores within NEAR_TIE of each other (the `most` closest, and all at the positions `at`): the largest change per position over
    these pairs, one pair changed at a time.  A choice that close is made differently by ANY run that rounds the router's input, and
    what follows at that position and, through keys, values and states, at later ones, differs."""
    import plain_lilalorn as P
    orig = P.router_scores
    state = {"call": 0, "swap": None, "margins": []}
    tops = [lay["mlp"]["router"]["top"] for lay in cfg["layers"] if lay.get("mlp")]

    def router_scores(h, w):
        call = state["call"]
        state["call"] += 1
        s = orig(h, w)
        top = tops[call]
        if top >= s.shape[1]:
            return s
        order = torch.argsort(s, dim=-1, descending=True)
        if state["swap"] is None:
            for p in range(h.shape[0]):
                state["margins"].append((float(s[p, order[p, top - 1]] - s[p, order[p, top]]), call, p))
        elif state["swap"][0] == call:
            p = state["swap"][1]
            s = s.clone()
            a, b = order[p, top - 1].item(), order[p, top].item()
            s[p, a], s[p, b] = s[p, b].item(), s[p, a].item()
        return s

    worst = np.zeros(len(tokens))
    scale = float(np.abs(ref).max())
    try:
        P.router_scores = router_scores
        plain_logits(cfg, tensors, tokens)
        near = sorted(m for m in state["margins"] if m[0] < NEAR_TIE)
        for _, call, p in near[:most] + [m for m in near[most:] if m[2] in at]:
            state["call"], state["swap"] = 0, (call, p)
            worst = np.maximum(worst, np.abs(plain_logits(cfg, tensors, tokens) - ref).max(axis=1) / scale)
    finally:
        P.router_scores = orig
    return worst


def rounding_sensitivity(cfg, tensors, tokens, draws=3, at=()):
    """How far a rounding of every sublayer's input to bfloat16 moves each position's logits in the plain implementation, as a
    fraction of the largest logit: the largest of `draws` runs, the first with the rounding alone, the others with a relative
    nudge of up to 2^-8 before it; and the largest change that a near tie of a router makes when it falls the other way
    (``near_tie_sensitivity``).  Positions where this is large differ by more than the usual rounding in ANY bfloat16 run; a
    bfloat16 comparison allows for it position by position."""
    import plain_lilalorn as P
    ref = plain_logits(cfg, tensors, tokens)
    scale = float(np.abs(ref).max())
    orig = P.sublayer_input
    g = torch.Generator().manual_seed(len(tokens))
    worst = near_tie_sensitivity(cfg, tensors, tokens, ref, at)
    try:
        for d in range(draws):
            def rounded(x, d=d):
                if d:
                    x = x * (1.0 + (torch.rand(x.shape, generator=g, dtype=torch.float64) - 0.5) * 2.0 ** -7)
                return x.to(torch.bfloat16).to(torch.float64)
            P.sublayer_input = rounded
            worst = np.maximum(worst, np.abs(plain_logits(cfg, tensors, tokens) - ref).max(axis=1) / scale)
    finally:
        P.sublayer_input = orig
    return worst


def assert_close_bfloat16(got, ref, sens, what=""):
    """The fixed bfloat16 tolerance of `traces` at every position, except that a position may differ by three times what the
    rounding of the sublayers' inputs alone does to it in the plain implementation (`sens`, from ``rounding_sensitivity``); few
    positions may need that, and the mean over all (of a request of sixteen tokens or more) stays within the fixed mean."""
    import traces
    tol = traces.TOL["bfloat16"]
    assert got.shape == ref.shape and np.isfinite(got).all(), what
    scale = float(np.abs(ref).max())
    diff = np.abs(got.astype(np.float64) - ref.astype(np.float64))
    err = diff.max(axis=1) / scale
    allowed = np.maximum(tol["max_rel"], 3.0 * sens)
    bad = np.nonzero(err > allowed)[0]
    assert len(bad) == 0, f"{what}: positions {bad[:10].tolist()} differ by {err[bad[:10]].round(4).tolist()} of the largest logit, allowed {allowed[bad[:10]].round(4).tolist()}"
    over = int((err > tol["max_rel"]).sum())
    assert over <= max(1, len(err) // 10), f"{what}: {over} of {len(err)} positions beyond the fixed tolerance"
    if len(err) >= 16:              # (a mean over a handful of positions is no mean)
        assert diff.mean() <= 1.5 * tol["mean_rel"] * scale, f"{what}: mean |diff| {diff.mean():.3e} > {1.5 * tol['mean_rel']:.1e} * {scale:.3f}"
