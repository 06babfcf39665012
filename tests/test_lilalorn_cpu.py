"""Lilalorn without a GPU: the configuration reader, the plan the builder makes (which layers share a block, what every layer keeps,
where the multipliers go), the scaled frequencies, and the plain implementation's own consistency (each mechanism worked out by hand)."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_lilalorn as P
import tiny_lilalorn as tl
from xyntetik_runner_b200 import architectures  # noqa: F401
from xyntetik_runner_b200.config import registry
from xyntetik_runner_b200.config.base import ConfigError
from xyntetik_runner_b200.config.lilalorn import LilalornConfig
from xyntetik_runner_b200.config.llama import RopeScaling
from xyntetik_runner_b200.parts import MLP, Rope, RoutedExperts
from xyntetik_runner_b200.weights.loader import FolderSource, WeightsError, load_tensors

F64 = torch.float64


def plan_of(name):
    return registry.resolve("Lilalorn").build_plan(LilalornConfig.from_dict(tl.clean(tl.CONFIGS[name])))


@pytest.mark.parametrize("name", list(tl.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    cfg = LilalornConfig.from_dict(tl.clean(tl.CONFIGS[name]))
    assert LilalornConfig.from_dict(cfg.to_dict()) == cfg
    plan = plan_of(name)
    plan.validate()
    want = {n: tuple(s) for n, s in tl.shapes(tl.CONFIGS[name]).items()}
    specs = {n: s for n, s in plan.tensor_specs().items() if not s.optional or n in want}
    assert set(specs) == set(want)
    for n, s in specs.items():
        fixed = slice(1 if s.any_rows else 0, -1 if s.any_cols else None)
        assert tuple(s.shape)[fixed] == want[n][fixed], n
    assert {n for n, s in specs.items() if s.any_rows} == {n for n in want if n.endswith(".a1")}
    assert {n for n, s in specs.items() if s.any_cols} == {n for n in want if n.endswith(".a2")}


def test_layers_that_share_tensors_and_what_each_layer_keeps():
    plan = plan_of("mix")
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 1, 3, 0, 1]
    needs = [(b.mixer.kv_need(), b.mixer.state_need()) for b in plan.blocks]
    assert (needs[0][0].kv_heads, needs[0][0].head_dim, needs[0][0].window) == (2, 32, None) and needs[0][1].shape == (3 * 10 * 12,)
    assert needs[1][0] is None and needs[1][1].shape == (3 * 20 * 14,)
    assert [e.layer for e in plan_of("odd").schedule] == [1, 0, 1, 2]                    # (a block stands where its tensors' layer does)
    assert all(b.mixer.kv_need() is None for b in plan_of("rec").blocks)


def test_multipliers_ride_in_the_sublayers_outputs():
    plan = plan_of("mix")
    left, right = plan.blocks[0].mixer.first, plan.blocks[0].mixer.second
    assert left.out_scale == pytest.approx(0.6 * 0.8) and right.out_scale == pytest.approx(0.6 * 1.3)
    assert right.read_scale == pytest.approx(10 ** -0.5) and plan.blocks[1].mixer.read_scale == pytest.approx(20 ** -0.5)
    assert plan.blocks[1].mixer.out_scale == 0.6 and plan.blocks[0].feed_forward.out_scale == 0.6 and plan.head.scale == 1.7


def test_folder_is_resolved_and_the_middle_gives_its_size(tmp_path):
    path, cfg, tensors = tl.make_folder(str(tmp_path / "m"), "mix")
    arch, typed = registry.load_config(path)
    assert arch.name == "Lilalorn" and typed.width == cfg["width"] and len(typed.layers) == 7
    plan = arch.build_plan(typed)
    got = load_tensors(plan.tensor_specs(), FolderSource(path), torch.device("cpu"))
    assert got["l1.mix.a1"].shape == (5, 96) and got["l1.mix.a2"].shape == (60, 5) and got["l4.mix.a1"].shape == (12, 96)
    # a layer that has no tensors of its own must not bring any; columns must fit
    extra = dict(tensors)
    extra["l3.norm1"] = tensors["l1.norm1"]
    tl.make_folder(str(tmp_path / "extra"), "mix", extra)
    with pytest.raises(WeightsError, match="l3.norm1"):
        load_tensors(plan.tensor_specs(), FolderSource(str(tmp_path / "extra")), torch.device("cpu"))
    bad = dict(tensors)
    bad["l1.mix.a2"] = torch.zeros(59, 5, dtype=torch.bfloat16)
    tl.make_folder(str(tmp_path / "bad"), "mix", bad)
    with pytest.raises(WeightsError, match="l1.mix.a2"):
        load_tensors(plan.tensor_specs(), FolderSource(str(tmp_path / "bad")), torch.device("cpu"))


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("heads"), "heads"),
    (lambda d: d["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"]["left"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 26), "rot.dims"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("high"), "high"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].__setitem__("low", 9.0), "low"),
    (lambda d: d["layers"][0]["mixer"]["right"].__setitem__("decay", [0.9, 0.8]), "decay"),
    (lambda d: d["layers"][0]["mixer"]["right"].__setitem__("decay", "slow"), "decay"),
    (lambda d: d["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("tau", 0), "tau"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("dim", 0), "positive"),
    (lambda d: d["layers"][1]["mlp"].__setitem__("kind", "dense"), "kind"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 9), "top"),
    (lambda d: d["layers"][1]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda d: d["layers"][1]["mlp"]["shared"].__setitem__("ff", 0), "shared.ff"),
    (lambda d: d["layers"][3].__setitem__("weights_of", 7), "weights_of"),
    (lambda d: d["layers"][3].__setitem__("weights_of", 3), "weights_of"),
    (lambda d: d["layers"][1].__setitem__("weights_of", 6), "back to itself"),
    (lambda d: d["layers"][3].__setitem__("weights_of", 0), "differs"),
    (lambda d: d["layers"][3]["mixer"].__setitem__("tau", 2.5), "differs"),
    (lambda d: d.pop("width"), "width"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.__setitem__("residual_mult", "half"), "residual_mult"),
    (lambda d: d.__setitem__("layers", []), "layers"),
])
def test_config_refusals(edit, word):
    d = copy.deepcopy(tl.clean(tl.CONFIGS["mix"]))
    edit(d)
    with pytest.raises(ConfigError, match=word):
        LilalornConfig.from_dict(d)


def test_what_a_configuration_may_leave_out():
    d = copy.deepcopy(tl.clean(tl.CONFIGS["odd"]))
    d.pop("residual_mult"); d.pop("logit_scale")
    m = d["layers"][3]["mixer"]
    m["left"].pop("kv_heads"); m["left"].pop("vdim"); m["left"].pop("rot"); m.pop("left_scale"); m.pop("right_scale")
    cfg = LilalornConfig.from_dict(d)
    left = cfg.layers[3].mixer.left
    assert (cfg.residual_mult, cfg.logit_scale, left.kv_heads, left.vdim, left.rot.dims) == (1.0, 1.0, 5, 10, 0)
    assert cfg.layers[1].mlp.shared_ff is None and cfg.layers[3].mlp is None
    registry.resolve("Lilalorn").build_plan(cfg).validate()


def test_parts_refuse_what_they_do_not_compute():
    with pytest.raises(ValueError, match="gated shared expert"):
        RoutedExperts(16, 4, 2, 8, "p.", shared=MLP(16, 8, "p.s."), shared_gate="s.sg", scoring="softmax_all")
    with pytest.raises(ValueError, match="factor on the output"):
        RoutedExperts(16, 4, 2, 8, "p.", shared=MLP(16, 8, "p.s."), out_scale=0.5)
    with pytest.raises(ValueError, match="swish_clamp"):
        RoutedExperts(16, 4, 2, 8, "p.", gate=None, activation="swish_clamp", limit=1.0)


# ---- frequencies ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [(16, 5000.0, (6.0, 1.0, 5.0, 40)), (18, 300.0, (3.0, 0.5, 2.0, 24)), (64, 1e5, (8.0, 1.0, 4.0, 128)),
                                               (32, 2e4, (5.0, 0.0, 4.0, 1000)), (32, 2e4, (5.0, 2.0, 2.0, 100)), (12, 1e4, None)])
def test_scaled_frequencies_against_the_plain_formula(dims, base, scaling):
    sc = None if scaling is None else RopeScaling(rope_type="llama3", factor=scaling[0], low_freq_factor=scaling[1], high_freq_factor=scaling[2],
                                                  original_max_position_embeddings=scaling[3])
    rope = Rope(dims, base, scaling=sc)
    d = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    if scaling is not None and scaling[1] == scaling[2]:
        want = [f if scaling[3] * f / (2 * math.pi) > scaling[2] else f / scaling[0] for f in (base ** (-2.0 * i / dims) for i in range(dims // 2))]
    else:
        want = P.frequencies(dims, base, d, F64).numpy()
    assert np.allclose(rope.inv_freq64_host, want, rtol=1e-13)
    assert np.allclose(rope.inv_freq_host, want, rtol=1e-6)


def test_three_ranges_of_wavelengths_by_hand():
    # base 1: every pair turns one radian a position, 2 pi positions a turn
    f = lambda factor, low, high, original: P.frequencies(4, 1.0, {"factor": factor, "low": low, "high": high, "original": original}, F64).tolist()
    assert f(8.0, 1.0, 4.0, 100 * 2 * math.pi) == [1.0, 1.0]                             # 100 turns: more than high
    assert f(8.0, 1.0, 4.0, 0.5 * 2 * math.pi) == [0.125, 0.125]                         # half a turn: less than low
    assert np.allclose(f(8.0, 1.0, 4.0, 2.5 * 2 * math.pi), [0.5 * 0.125 + 0.5, 0.5 * 0.125 + 0.5])   # halfway between


# ---- the plain implementation by hand --------------------------------------------------------------------------------------------
def _eye_weights(H, D, V, W):
    w = {n: torch.zeros(H * (D if n in "qk" else V), W, dtype=F64) for n in "qkvg"}
    w["o"] = torch.eye(H * V, dtype=F64)
    return w


def test_retention_by_hand():
    """One head, one key channel, one value channel: S and the read-out are numbers; the unit norm leaves their sign."""
    h = torch.tensor([[2.0, 1.0, 3.0, 0.5], [1.0, -1.0, 1.0, 1.0], [1.0, 2.0, -10.0, 2.0]], dtype=F64)
    w = {n: torch.zeros(1, 4, dtype=F64) for n in "qkvg"}
    for i, n in enumerate("qkvg"):
        w[n][0, i] = 1.0
    w["o"] = torch.eye(1, dtype=F64)
    S, want = 0.0, []
    for q, k, v, g in h.tolist():
        S = 0.5 * S + k * v
        o = S * q
        want.append(o / math.sqrt(o * o + 0.25) * g / (1 + math.exp(-g)))
    got = P.retention(h, w, {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5]}, 0.25)
    assert torch.allclose(got[:, 0], torch.tensor(want, dtype=F64))


def test_keys_of_retention_and_queries_of_gated_linear_attention_are_scaled():
    """Four key channels: a factor of one half, which eps makes visible behind the norms."""
    g = torch.Generator().manual_seed(0)
    T, W, D, V = 6, 20, 4, 3
    h = torch.randn(T, W, generator=g, dtype=F64)
    w = {n: torch.randn((D if n in "qk" else V), W, generator=g, dtype=F64) for n in "qkvg"}
    w.update(o=torch.eye(V, dtype=F64), norm=torch.ones(V, dtype=F64), a1=torch.zeros(2, W, dtype=F64), a2=torch.zeros(D, 2, dtype=F64))
    w["a2.b"] = torch.full((D,), math.log(3.0), dtype=F64)                                # sigmoid 0.75
    S, o = torch.zeros(D, V, dtype=F64), []
    for t in range(T):
        S = 0.75 ** 0.5 * S + torch.outer(w["k"] @ h[t], w["v"] @ h[t])
        o.append(0.5 * (S.T @ (w["q"] @ h[t])))
    o = torch.stack(o)
    want = o / torch.sqrt((o * o).mean(1, keepdim=True) + 2.0) * P.silu(h @ w["g"].T)
    assert torch.allclose(P.retention(h, w, {"heads": 1, "dim": D, "vdim": V, "decay": [0.75 ** 0.5]}, 2.0), want)
    assert torch.allclose(P.gated_linear_attention(h, w, {"heads": 1, "dim": D, "vdim": V, "tau": 2.0}, 2.0), want)


def test_decays_act_on_key_channels():
    """Two key channels with different decays: what each wrote fades at its own rate, whatever the value channel."""
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 1.0]], [[0.0, 0.0]], [[0.0, 0.0]]], dtype=F64)
    v = torch.tensor([[[5.0, 7.0]], [[0.0, 0.0]], [[0.0, 0.0]]], dtype=F64)
    a = torch.tensor([[[0.1, 0.1]], [[0.5, 0.25]], [[0.5, 0.25]]], dtype=F64)
    got = P.decayed_reads(q, k, v, a)
    assert torch.allclose(got[:, 0], torch.tensor([[5.0, 7.0], [2.5, 3.5], [5.0 / 16, 7.0 / 16]], dtype=F64))


def test_attention_by_hand():
    """Two tokens, no rotation: the second mixes both values by the softmax of its scores; with a rotation only distances count."""
    m = {"heads": 2, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 0.5}
    h = torch.tensor([[1.0, 0.0, 2.0], [0.0, 1.0, -1.0]], dtype=F64)
    w = {"q": torch.tensor([[1.0, 2.0, 0], [0, 1, 0], [0, 0, 1], [1, 0, 0]], dtype=F64), "k": torch.tensor([[1.0, 0, 0], [0, 1.0, 0]], dtype=F64),
         "v": torch.tensor([[0.0, 0, 1]], dtype=F64), "o": torch.eye(2, dtype=F64)}
    got = P.softmax_attention(h, w, m)
    assert torch.allclose(got[0], torch.tensor([2.0, 2.0], dtype=F64))
    # head 0: q = (2, 1), keys (1, 0) and (0, 1): scores 1 and 0.5; head 1: q = (-1, 0): -0.5 and 0
    p0, p1 = math.exp(1) / (math.exp(1) + math.exp(0.5)), math.exp(-0.5) / (math.exp(-0.5) + 1)
    assert torch.allclose(got[1], torch.tensor([2 * p0 - (1 - p0), 2 * p1 - (1 - p1)], dtype=F64))
    g = torch.Generator().manual_seed(1)
    v, pos, f = torch.randn(1, 2, 6, generator=g, dtype=F64), torch.tensor([11]), P.frequencies(4, 50.0, None, F64)
    a, b = P.rotate(v[:, :1], pos, 4, f), P.rotate(v[:, 1:], pos + 5, 4, f)
    c, d = P.rotate(v[:, :1], pos - 11, 4, f), P.rotate(v[:, 1:], pos - 6, 4, f)
    assert torch.allclose((a * b).sum(), (c * d).sum()) and torch.equal(a[..., 4:], v[:, :1, 4:])
    assert torch.allclose(P.rotate(v, torch.tensor([1]), 2, torch.tensor([math.pi / 2], dtype=F64))[..., :2], torch.stack([-v[..., 1], v[..., 0]], -1))


def test_sides_add_with_their_scales():
    d = tl.CONFIGS["odd"]["layers"][1]["mixer"]
    t = tl.draw(tl.CONFIGS["odd"], 3)
    w = {k[len("l1.mix."):]: v.to(F64) for k, v in t.items() if k.startswith("l1.mix.")}
    h = torch.randn(7, 68, generator=torch.Generator().manual_seed(2), dtype=F64)
    left = P.softmax_attention(h, P._sub(w, "left."), d["left"])
    right = P.retention(h, P._sub(w, "right."), d["right"], 1e-6)
    assert torch.allclose(P.parallel_mixer(h, w, d, 1e-6), 1.1 * left + 0.4 * right)


def test_experts_by_hand():
    """Three experts of one feature: the two best, by scores over their sum, and the shared one under its gate."""
    h = torch.tensor([[1.0, 2.0]], dtype=F64)
    w = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0], [0.0, 0.2]], dtype=F64), "shared.sg": torch.tensor([[0.5, 0.0]], dtype=F64),
         "shared.up": torch.tensor([[1.0, 1.0]], dtype=F64), "shared.down": torch.tensor([[1.0], [0.0]], dtype=F64)}
    for e in range(3):
        w[f"e{e}.up"] = torch.tensor([[1.0 + e, 0.0 if e != 1 else -3.0]], dtype=F64)
        w[f"e{e}.down"] = torch.tensor([[0.0], [1.0]], dtype=F64)
    z = [1.0, 2.0, 0.4]
    p = [math.exp(v) for v in z]
    first = p[1] / (p[0] + p[1])                                    # expert 1 sees 2 - 6 < 0: nothing; expert 0 sees 1
    want = torch.tensor([9.0 / (1 + math.exp(-0.5)), (1 - first) * 1.0], dtype=F64)
    f = {"router": {"experts": 3, "top": 2}, "expert": {"ff": 1}, "shared": {"ff": 1}}
    assert torch.allclose(P.routed_ff(h, w, f)[0], want)


def test_layers_that_share_tensors_equal_layers_with_copies_of_them():
    cfg = tl.CONFIGS["mix"]
    t = tl.draw(cfg, 9)
    toks = [3, 50, 7, 7, 120, 4, 200]
    own = [P.owner(cfg["layers"], i) for i in range(7)]
    assert own == [0, 1, 2, 1, 4, 0, 1]
    copies = dict(t)
    for i, j in enumerate(own):
        for n, v in t.items():
            if n.startswith(f"l{j}."):
                copies[f"l{i}." + n[len(f"l{j}."):]] = v
    flat = dict(cfg, layers=[{k: v for k, v in lay.items() if k != "weights_of"} for lay in cfg["layers"]])
    assert torch.equal(P.forward(cfg, t, toks), P.forward(flat, copies, toks))


def test_multipliers_of_the_stream_and_the_logits():
    cfg = dict(tl.CONFIGS["rec"], layers=tl.CONFIGS["rec"]["layers"][1:])
    cfg["layers"] = [dict(cfg["layers"][0])]
    t = {n.replace("l1.", "l0."): v for n, v in tl.draw(tl.CONFIGS["rec"], 4).items() if not n.startswith("l0.")}
    out = []
    full = P.forward(cfg, t, [1, 2, 3], layers_out=out)
    x0 = t["embed"][[1, 2, 3]].to(F64)
    one = []
    P.forward(dict(cfg, residual_mult=1.0), t, [1, 2, 3], layers_out=one)
    assert torch.allclose(out[0] - x0, 0.9 * (one[0] - x0))
    assert torch.allclose(full, 1.2 * P.forward(dict(cfg, logit_scale=1.0), t, [1, 2, 3]))
