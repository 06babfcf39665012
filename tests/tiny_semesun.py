"""Small Semesun configurations with random weights for the tests, as config.json + model.safetensors folders.

The sizes are awkward on purpose: widths that are no multiple of 8, one head, key sizes that differ from value sizes and are no
multiple of 16, as many key heads as heads and fewer, windows of one token and longer than the requests, kept tokens from none to
more than a page and more than the window, bias tables of few and many rows that end inside and beyond the window, layers that mix
their values beside layers that do not, recurrences of one group and several with one tap or several and norms over one part or
several, routers with and without identity experts and groups, of which all or few outputs are chosen, layers without a
feed-forward, models of one kind of layer alone.
"""
import json
import os

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, scale, size, keep, bias_max, rel, v_mix=False):
    """`rel`: rows of the bias table (a size that only the tensor's shape gives).  size None: no window."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep}
    return {"type": "attention", "mixer": m, "_rel": rel}


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5, identity=0, groups=None, scale=1.0):
    r = {"experts": experts, "top": top, "identity": identity, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff, "limit": limit}}


def layer(mixer, mlp):
    d = dict(mixer)
    d["mlp"] = mlp
    return d


def model(vocab, width, eps, layers):
    return {"architecture": "Semesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # both mixers and both feed-forwards; three layers that mix values around one that does not
    "mix": model(211, 96, 1e-5, [
        layer(attention(4, 2, 24, 16, 0.21, 20, 3, 30, 12, True), dense(80)),
        layer(mamba2(6, 10, 20, 3, 4, 5), moe(7, 3, 24, 0.8, identity=2, groups=(3, 2), scale=1.7)),
        layer(attention(6, 2, 12, 16, 0.3, 33, 9, 15, 6, True), moe(6, 2, 16, 2.0, identity=6, groups=(4, 1))),
        layer(attention(3, 3, 16, 20, 0.25, 9, 17, 90, 20), None),
        layer(attention(2, 1, 20, 32, 0.2, 20, 3, 50, 8, True), dense(40))]),
    # a width that is no multiple of 8; one head; the recurrence first; a window of one token; no kept tokens; experts without groups
    "odd": model(131, 68, 1e-6, [
        layer(mamba2(2, 9, 5, 1, 2, 1), dense(36)),
        layer(attention(1, 1, 18, 6, 0.2, 1, 2, 9, 4, True), moe(4, 1, 12, 0.5)),
        layer(attention(5, 1, 10, 6, 0.4, 40, 0, 11, 10, True), moe(3, 4, 20, 1.0, identity=1, scale=0.6)),
        layer(mamba2(3, 4, 33, 3, 1, 3), None)]),
    # sizes that the tensor-core kernels take (heads of 64 and 128, pages of 64); kept tokens over more than one tile
    "tc": model(160, 128, 1e-5, [
        layer(attention(4, 2, 64, 64, 0.12, 70, 5, 48, 16, True), dense(96)),
        layer(mamba2(8, 32, 64, 2, 4, 2), moe(8, 2, 64, 1.2, identity=4, groups=(3, 2), scale=2.0)),
        layer(attention(2, 1, 128, 128, 0.09, 130, 140, 200, 32, True), moe(12, 3, 32, 1.0, identity=4, groups=(4, 2))),
        layer(attention(16, 2, 64, 48, 0.15, 33, 1, 20, 8), None),
        layer(attention(8, 8, 48, 64, 0.16, 150, 66, 100, 24), dense(64))]),
    # recurrences alone (no keys are cached at all)
    "rec": model(90, 64, 1e-5, [
        layer(mamba2(4, 16, 16, 2, 3, 4), dense(40)),
        layer(mamba2(2, 24, 40, 1, 5, 1), None)]),
}
SEEDS = {"mix": 41, "odd": 42, "tc": 43, "rec": 44}


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
        p, m = f"l{i}.", lay["mixer"]
        out.update({p + "norm1": (W,), p + "norm2": (W,)})
        if lay["type"] == "attention":
            H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * D, W), p + "mix.k": (G * D, W), p + "mix.v": (G * V, W), p + "mix.q.norm": (D,), p + "mix.k.norm": (D,),
                        p + "mix.rel": (lay["_rel"], H), p + "mix.o": (W, H * V)})
            if m["v_mix"]:
                out[p + "mix.vmix"] = ()
        else:
            H, V, N, G, K = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            CH = H * V + 2 * G * N
            out.update({p + "mix.in": (H * V + CH + H, W), p + "mix.conv": (CH, K), p + "mix.conv.b": (CH,), p + "mix.dt_bias": (H,),
                        p + "mix.A_log": (H,), p + "mix.D": (H,), p + "mix.norm": (H * V,), p + "mix.o": (W, H * V)})
        f = lay.get("mlp")
        if f and f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
        elif f:
            E, ff = f["router"]["experts"], f["expert"]["ff"]
            R = E + f["router"].get("identity", 0)
            out.update({p + "mlp.router": (R, W), p + "mlp.correction": (R,)})
            for e in range(E):
                out.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
    return out


def draw(cfg, seed, dtype=torch.bfloat16, slow=False):
    """Random tensors: matrices N(0, 1/fan_in) (experts' gates and ups larger, so that clamps bite), norms around one, biases by
    distance N(0, 1), mixing numbers far from zero and one, routers wide enough that choices differ between tokens, corrections of
    both signs that change some choices (and make some choice scores negative), decay rates over a wide range (`slow`: all slow, so
    that the first tokens still count hundreds of tokens later)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        r = lambda: torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith(("norm1", "norm2")):
            t = 1.0 + 0.2 * r()
        elif name.endswith("mix.rel"):
            t = r()
        elif name.endswith("mix.vmix"):
            t = 0.4 + 0.2 * r()
        elif name.endswith("mix.conv"):
            t = 1.5 * r() / shape[-1] ** 0.5
        elif name.endswith("conv.b"):
            t = 0.5 * r()
        elif name.endswith("dt_bias"):
            t = -4.0 + 0.3 * r() if slow else -1.0 + r()
        elif name.endswith("A_log"):
            t = -2.0 + 0.3 * r() if slow else -0.5 + r()
        elif name.endswith("mix.D"):
            t = 1.0 + 0.5 * r()
        elif name.endswith("correction"):
            t = 0.15 * r()
        elif name.endswith("router"):
            t = 2.5 * r() / shape[-1] ** 0.5
        elif name.endswith((".gate", "mlp.up")) or (".e" in name and name.endswith(".up")):
            t = 1.5 * r() / shape[-1] ** 0.5
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
    import plain_semesun
    return plain_semesun.forward(cfg, tensors, tokens, dtype=torch.float64).to(torch.float32).numpy()


def plain_greedy(cfg, tensors, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(plain_logits(cfg, tensors, toks)[-1])))
    return toks[len(prompt):]


NEAR_TIE = 0.01        # choice scores closer than this may change places under bfloat16 rounding of what the router reads


def near_tie_sensitivity(cfg, tensors, tokens, ref, most=32):
    """What a change of places does to every position's logits, for the (layer, position) pairs where the last chosen output of a
    router and the first one left out, or the last kept group and the first one dropped, have choice scores within NEAR_TIE of each
    other (the `most` closest): the largest change per position over these pairs, one pair changed at a time.  A choice that close
    is made differently by ANY run that rounds the router's input, and what follows at that position and, through keys, values and
    states, at later ones, differs."""
    import plain_semesun as P
    orig = P.choice_scores
    state = {"call": 0, "swap": None, "margins": []}

    def choice_scores(h, w, r):
        call = state["call"]
        state["call"] += 1
        s, c = orig(h, w, r)
        top = r["top"]
        order = torch.argsort(c, dim=-1, descending=True)
        g = r.get("groups") or {"count": 1, "keep": 1}
        free = s + w["correction"]
        gmax = free.view(free.shape[0], g["count"], -1).max(dim=-1).values
        gorder = torch.argsort(gmax, dim=-1, descending=True)
        if state["swap"] is None:
            for p in range(h.shape[0]):
                if top < c.shape[1] and torch.isfinite(c[p, order[p, top]]):
                    state["margins"].append((float(c[p, order[p, top - 1]] - c[p, order[p, top]]), call, p, "choice"))
                if g["keep"] < g["count"]:
                    state["margins"].append((float(gmax[p, gorder[p, g["keep"] - 1]] - gmax[p, gorder[p, g["keep"]]]), call, p, "group"))
        elif state["swap"][0] == call:
            _, p, kind = state["swap"]
            c = c.clone()
            if kind == "choice":
                a, b = order[p, top - 1].item(), order[p, top].item()
                c[p, a], c[p, b] = c[p, b].item(), c[p, a].item()
            else:
                per = c.shape[1] // g["count"]
                a, b = gorder[p, g["keep"] - 1].item(), gorder[p, g["keep"]].item()
                c[p, a * per:(a + 1) * per] = float("-inf")
                c[p, b * per:(b + 1) * per] = free[p, b * per:(b + 1) * per]
        return s, c

    worst = np.zeros(len(tokens))
    scale = float(np.abs(ref).max())
    try:
        P.choice_scores = choice_scores
        plain_logits(cfg, tensors, tokens)
        near = sorted(m for m in state["margins"] if m[0] < NEAR_TIE)[:most]
        for _, call, p, kind in near:
            state["call"], state["swap"] = 0, (call, p, kind)
            worst = np.maximum(worst, np.abs(plain_logits(cfg, tensors, tokens) - ref).max(axis=1) / scale)
    finally:
        P.choice_scores = orig
    return worst


def rounding_sensitivity(cfg, tensors, tokens, draws=3):
    """How far a rounding of every sublayer's input to bfloat16 moves each position's logits in the plain implementation, as a
    fraction of the largest logit: the largest of `draws` runs, the first with the rounding alone, the others with a relative
    nudge of up to 2^-8 before it; and the largest change that a near tie of a router makes when it falls the other way
    (``near_tie_sensitivity``).  Positions where this is large differ by more than the usual rounding in ANY bfloat16 run; a
    bfloat16 comparison allows for it position by position."""
    import plain_semesun as P
    ref = plain_logits(cfg, tensors, tokens)
    scale = float(np.abs(ref).max())
    orig = P.sublayer_input
    g = torch.Generator().manual_seed(len(tokens))
    worst = near_tie_sensitivity(cfg, tensors, tokens, ref)
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
