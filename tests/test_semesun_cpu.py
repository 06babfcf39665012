"""Semesun without a GPU: the configuration reader, the plan the builder makes (which layer leaves its values, what every layer
keeps), the distance buckets, and the plain implementation's own consistency (each mechanism worked out by hand)."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_semesun as P
import tiny_semesun as ts
from xyntetik_runner_b200 import architectures  # noqa: F401
from xyntetik_runner_b200.config import registry
from xyntetik_runner_b200.config.base import ConfigError
from xyntetik_runner_b200.config.semesun import SemesunConfig
from xyntetik_runner_b200.parts import DistanceBuckets
from xyntetik_runner_b200.weights.loader import FolderSource, WeightsError, load_tensors

F64 = torch.float64


@pytest.mark.parametrize("name", list(ts.CONFIGS))
def test_config_round_trip_and_tensor_names(name):
    d = ts.clean(ts.CONFIGS[name])
    cfg = SemesunConfig.from_dict(d)
    assert SemesunConfig.from_dict(cfg.to_dict()) == cfg
    plan = registry.resolve("Semesun").build_plan(cfg)
    plan.validate()
    want = {n: tuple(s) for n, s in ts.shapes(ts.CONFIGS[name]).items()}
    specs = {n: s for n, s in plan.tensor_specs().items() if not s.optional or n in want}
    assert set(specs) == set(want)
    for n, s in specs.items():
        assert tuple(s.shape)[1 if s.any_rows else 0:] == want[n][1 if s.any_rows else 0:], n
    assert {n for n, s in specs.items() if s.any_rows} == {n for n in want if n.endswith(".rel")}


def test_what_each_layer_keeps_and_shares():
    plan = registry.resolve("Semesun").build_plan(SemesunConfig.from_dict(ts.clean(ts.CONFIGS["mix"])))
    needs = [(b.mixer.kv_need(), b.mixer.state_need()) for b in plan.blocks]
    assert (needs[0][0].kv_heads, needs[0][0].head_dim, needs[0][0].window, needs[0][0].keep_first) == (2, 32, 20, 3)
    assert needs[1][0] is None and needs[1][1].shape == (6 * 10 * 20 + 3 * (6 * 10 + 2 * 3 * 20),)
    assert (needs[3][0].window, needs[3][0].keep_first) == (9, 17)
    assert [getattr(b.mixer, "value_share", None) for b in plan.blocks] == ["first", None, "mix", None, "mix"]
    odd = registry.resolve("Semesun").build_plan(SemesunConfig.from_dict(ts.clean(ts.CONFIGS["odd"])))
    assert odd.blocks[3].mixer.state_need().shape == (3 * 4 * 33,)                      # one tap: no tail
    rec = registry.resolve("Semesun").build_plan(SemesunConfig.from_dict(ts.clean(ts.CONFIGS["rec"])))
    assert all(b.mixer.kv_need() is None for b in rec.blocks)


def test_folder_is_resolved_and_its_tables_give_their_rows(tmp_path):
    path, cfg, tensors = ts.make_folder(str(tmp_path / "m"), "mix")
    arch, typed = registry.load_config(path)
    assert arch.name == "Semesun" and typed.width == cfg["width"] and len(typed.layers) == 5
    plan = arch.build_plan(typed)
    got = load_tensors(plan.tensor_specs(), FolderSource(path), torch.device("cpu"))
    assert got["l0.mix.rel"].shape == (12, 4) and got["l3.mix.rel"].shape == (20, 3) and got["l2.mix.vmix"].shape == ()
    # the first mixing layer's number may be absent (nothing reads it), a later one's may not; columns must fit
    for drop, fails in (("l0.mix.vmix", False), ("l4.mix.vmix", True)):
        ts.make_folder(str(tmp_path / drop), "mix", {n: t for n, t in tensors.items() if n != drop})
        if fails:
            with pytest.raises(WeightsError, match="l4.mix.vmix"):
                load_tensors(plan.tensor_specs(), FolderSource(str(tmp_path / drop)), torch.device("cpu"))
        else:
            load_tensors(plan.tensor_specs(), FolderSource(str(tmp_path / drop)), torch.device("cpu"))
    bad = dict(tensors)
    bad["l0.mix.rel"] = torch.zeros(12, 5, dtype=torch.bfloat16)
    ts.make_folder(str(tmp_path / "bad"), "mix", bad)
    with pytest.raises(WeightsError, match="l0.mix.rel"):
        load_tensors(plan.tensor_specs(), FolderSource(str(tmp_path / "bad")), torch.device("cpu"))


@pytest.mark.parametrize("edit, word", [
    (lambda d: d["layers"][0].__setitem__("type", "conv"), "type"),
    (lambda d: d["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("scale", 0.0), "scale"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("bias_max", 1), "bias_max"),
    (lambda d: d["layers"][0]["mixer"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda d: d["layers"][0]["mixer"].__setitem__("v_mix", 1), "v_mix"),
    (lambda d: d["layers"][2]["mixer"].__setitem__("vdim", 24), "another size"),
    (lambda d: d["layers"][1]["mixer"].pop("state"), "state"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("groups", 4), "groups"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("norm_groups", 7), "norm_groups"),
    (lambda d: d["layers"][1]["mixer"].__setitem__("conv", 0), "positive"),
    (lambda d: d["layers"][0]["mlp"].__setitem__("kind", "glu"), "kind"),
    (lambda d: d["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda d: d["layers"][1]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda d: d["layers"][1]["mlp"]["router"].__setitem__("top", 7), "top"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 4), "groups"),
    (lambda d: d["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 4), "groups"),
    (lambda d: d.pop("width"), "width"),
    (lambda d: d["norm"].pop("eps"), "eps"),
    (lambda d: d.__setitem__("layers", []), "layers"),
])
def test_config_refusals(edit, word):
    d = copy.deepcopy(ts.clean(ts.CONFIGS["mix"]))
    edit(d)
    with pytest.raises(ConfigError, match=word):
        SemesunConfig.from_dict(d)


def test_what_a_configuration_may_leave_out():
    d = copy.deepcopy(ts.clean(ts.CONFIGS["mix"]))
    d["layers"][0]["mixer"].pop("kv_heads")
    d["layers"][0]["mixer"]["vdim"] = 8                       # (4 heads of 8: as many value elements as the other mixing layers have)
    d["layers"][3]["mixer"].pop("mask")
    d["layers"][3]["mixer"].pop("v_mix")
    d["layers"][1]["mixer"].update(groups=1)
    for k in ("identity", "groups", "scale"):
        d["layers"][1]["mlp"]["router"].pop(k)
    cfg = SemesunConfig.from_dict(d)
    assert cfg.layers[0].mixer.kv_heads == 4 and cfg.layers[3].mixer.window is None and not cfg.layers[3].mixer.v_mix
    f = cfg.layers[1].mlp
    assert (f.identity, f.group_count, f.group_keep, f.scale) == (0, 1, 1, 1.0)
    registry.resolve("Semesun").build_plan(cfg).validate()


# ---- distance buckets ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,far", [(16, 240), (12, 30), (2, 5), (4, 9), (6, 300), (20, 90), (64, 1000), (16, 8.5), (32, 128), (10, 160), (20, 320)])
def test_distance_buckets_match_the_plain_formula(rows, far):
    table = DistanceBuckets(rows, far).table()
    assert table[-1] == rows - 1 and (len(table) == 1 or table[-2] < rows - 1)
    for n in range(len(table) + 40):
        assert table[min(n, len(table) - 1)] == P.bucket(n, rows, far), n


def test_distance_buckets_by_hand():
    # 8 rows up to 64: distances 0..3 are their own, then 4 (64 / 4)^(k / 4) = 4 2^k starts row 4 + k: 4, 8, 16, 32
    assert DistanceBuckets(8, 64).table().tolist() == [0, 1, 2, 3] + [4] * 4 + [5] * 8 + [6] * 16 + [7]
    for rows, far in ((1, 10), (8, 4), (8, 3)):
        with pytest.raises(ValueError):
            DistanceBuckets(rows, far)


# ---- the plain implementation against hand-worked numbers ----------------------------------------------------------------------
def test_window_and_kept_tokens_by_hand():
    v = P.visible(7, {"size": 2, "keep_first": 2})
    assert [[j for j in range(7) if v[i, j]] for i in range(7)] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 3, 4], [0, 1, 4, 5], [0, 1, 5, 6]]
    assert torch.equal(P.visible(5, None), torch.ones(5, 5).tril().bool())
    assert torch.equal(P.visible(5, {"size": 1}), torch.eye(5).bool())


def test_attention_by_hand():
    """Two tokens, one head of one element: unit-RMS makes queries and keys +-1 (eps 0), so the scores are scale * (+-1) * weights plus
    the bias of distances 0 and 1; the bias is not scaled."""
    w = {"q": torch.tensor([[3.0]]), "k": torch.tensor([[-2.0]]), "v": torch.tensor([[1.0]]), "q.norm": torch.tensor([2.0]), "k.norm": torch.tensor([0.5]),
         "rel": torch.tensor([[0.3], [-0.4]]), "o": torch.tensor([[1.0]])}
    w = {k: t.to(F64) for k, t in w.items()}
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.7, "bias_max": 4, "mask": {"size": 5, "keep_first": 0}}
    h = torch.tensor([[1.0], [-2.0]], dtype=F64)
    out = P.attention(h, w, m, 0.0, {})
    # keys: -0.5, +0.5; the second query: -2.  Scores of query 1: key 0: 0.7 * 1 - 0.4, key 1: 0.7 * -1 + 0.3
    e0, e1 = math.exp(0.7 - 0.4), math.exp(-0.7 + 0.3)
    f32 = lambda x: float(torch.tensor(x, dtype=torch.float32))
    assert abs(out[0].item() - 1.0) < 1e-12 and abs(out[1].item() - (e0 - 2.0 * e1) / (e0 + e1)) < 1e-6
    assert f32(0.3) != 0.3                                                             # (the biases above are float32 numbers)


def test_value_mixing_by_hand():
    shared = {}
    base = {"q": torch.eye(2), "k": torch.eye(2), "q.norm": torch.ones(2), "k.norm": torch.ones(2), "rel": torch.zeros(2, 1), "o": torch.eye(2)}
    base = {k: t.to(F64) for k, t in base.items()}
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "bias_max": 4, "mask": {"size": 1, "keep_first": 0}, "v_mix": True}
    h = torch.tensor([[1.0, 3.0]], dtype=F64)
    first = P.attention(h, dict(base, v=torch.eye(2, dtype=F64), vmix=torch.tensor(9.0, dtype=F64)), m, 1e-6, shared)
    second = P.attention(h, dict(base, v=2.0 * torch.eye(2, dtype=F64), vmix=torch.tensor(0.25, dtype=F64)), m, 1e-6, shared)
    third = P.attention(h, dict(base, v=4.0 * torch.eye(2, dtype=F64), vmix=torch.tensor(0.5, dtype=F64)), m, 1e-6, shared)
    plain = P.attention(h, dict(base, v=4.0 * torch.eye(2, dtype=F64)), dict(m, v_mix=False), 1e-6, shared)
    # one visible key each: what comes out is the cached value.  The first layer's own number does not matter; every later layer mixes
    # with the FIRST one's values, not with what the layer before it cached
    assert torch.allclose(first, h) and torch.allclose(second, 1.75 * h) and torch.allclose(third, 2.5 * h) and torch.allclose(plain, 4.0 * h)


def test_recurrence_by_hand():
    """One head, one state, one tap: x, B, C pass silu; S_t = exp(-e^A dt) S + dt B x, y = C S + D x, then silu(z) ahead of the norm."""
    silu = lambda z: z / (1.0 + math.exp(-z))
    sp = lambda z: math.log1p(math.exp(z))
    rows = {"z": 0.5, "x": 1.0, "B": -0.7, "C": 1.3, "dt": 0.2}
    w = {"in": torch.tensor([[v] for v in rows.values()]), "conv": torch.tensor([[2.0], [1.0], [0.5]]), "conv.b": torch.tensor([0.1, 0.2, -0.3]),
         "dt_bias": torch.tensor([-0.4]), "A_log": torch.tensor([0.3]), "D": torch.tensor([1.5]), "norm": torch.tensor([2.0]), "o": torch.tensor([[1.0]])}
    w = {k: t.to(F64) for k, t in w.items()}
    S, want = 0.0, []
    for t in (1.0, -2.0, 0.5):
        f = {k: float(torch.tensor(v, dtype=torch.float32)) * t for k, v in rows.items()}
        c = lambda v: float(torch.tensor(v, dtype=torch.float32))
        x, B, C = silu(2.0 * f["x"] + c(0.1)), silu(f["B"] + c(0.2)), silu(0.5 * f["C"] + c(-0.3))
        dt = sp(f["dt"] + c(-0.4))
        S = math.exp(-math.exp(c(0.3)) * dt) * S + dt * B * x
        y = (S * C + 1.5 * x) * silu(f["z"])
        want.append(2.0 * y / math.sqrt(y * y + 1e-3))
    m = {"heads": 1, "vdim": 1, "state": 1, "groups": 1, "conv": 1, "norm_groups": 1}
    out = P.mamba2(torch.tensor([[1.0], [-2.0], [0.5]], dtype=F64), w, m, 1e-3, {})
    assert torch.allclose(out.reshape(-1), torch.tensor(want, dtype=F64), rtol=1e-9)


def test_convolution_and_group_norm_by_hand():
    z = torch.tensor([[1.0], [2.0], [3.0]], dtype=F64)
    out = P.causal_conv(z, torch.tensor([[100.0, 10.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert out.reshape(-1).tolist() == [1.5, 12.5, 123.5]
    y, gate = torch.tensor([[3.0, 4.0, 10.0, 0.0]], dtype=F64), torch.full((1, 4), 40.0, dtype=F64)       # silu(40) = 40
    out = P.gated_group_norm(y, gate, torch.tensor([1.0, 2.0, 1.0, 1.0], dtype=F64), 2, 0.0)
    r = math.sqrt(12.5)
    assert torch.allclose(out, torch.tensor([[3 / r, 8 / r, math.sqrt(2.0), 0.0]], dtype=F64))


def test_choice_by_groups_with_identity_experts_by_hand():
    """Six outputs (four experts, two identity experts) in three groups: scores are a softmax over all six; the correction moves the
    choice of groups and inside them; all choice scores are negative and a dropped group must not come back as zero."""
    logits = torch.tensor([2.0, 0.0, 1.0, 1.5, 0.5, 0.0], dtype=F64)
    s = torch.softmax(logits, 0)
    w = {"router": logits[:, None], "correction": torch.tensor([-2.0, -1.0, -0.9, -1.2, -0.95, -1.0], dtype=F64)}
    r = {"experts": 4, "identity": 2, "top": 3, "groups": {"count": 3, "keep": 2}, "scale": 2.5}
    chosen, weight = P.routing(torch.tensor([[1.0]], dtype=F64), w, r)
    c = (s + w["correction"]).tolist()
    # groups {0, 1}, {2, 3}, {4, 5}: their best are 1, 2, 4; the first is dropped
    assert max(c) < 0 and max(c[0], c[1]) < min(max(c[2], c[3]), max(c[4], c[5]))
    assert chosen.tolist() == [sorted((2, 3, 4, 5), key=lambda e: -c[e])[:3]]
    assert torch.allclose(weight[0], 2.5 * s[chosen[0]])
    # identity experts give the input itself, experts their clamped gate
    f = {"router": r, "expert": {"ff": 1, "limit": 0.5}}
    for e in range(4):
        w.update({f"e{e}.gate": torch.ones(1, 1, dtype=F64), f"e{e}.up": -3.0 * torch.ones(1, 1, dtype=F64), f"e{e}.down": (e + 1.0) * torch.ones(1, 1, dtype=F64)})
    out = P.routed_ff(torch.tensor([[1.0]], dtype=F64), w, f)
    gate = 0.5 / (1.0 + math.exp(-1.702 * 0.5)) * (-0.5 + 1.0)
    want = sum(2.5 * s[e].item() * (1.0 if e >= 4 else (e + 1.0) * gate) for e in chosen[0].tolist())
    assert abs(out.item() - want) < 1e-12


def test_dense_feed_forward_by_hand():
    w = {"up": torch.tensor([[1.0], [-2.0]], dtype=F64), "down": torch.tensor([[1.0, 10.0]], dtype=F64)}
    assert P.dense_ff(torch.tensor([[3.0], [-0.5]], dtype=F64), w, {}).reshape(-1).tolist() == [9.0, 10.0]
