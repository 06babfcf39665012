"""Lilalorn on the GPU against the plain implementation: every way of cutting a request, mixed batches with pages and slots used
again, each mechanism alone, the kernels alone (the walks from states in other slots, decays per key channel, head norms without a
weight, ungated experts, the experts' sum with a gated shared expert and the norm behind it, factors in the products, rotations far
out), token sequences made so that one key stands out at page borders and far back, recurrences whose first tokens still count
hundreds of tokens later, long decoding, other sizes, greedy generation through the entry points."""
import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

import plain_lilalorn as P
import tiny_lilalorn as tl
import traces

pytestmark = pytest.mark.gpu

LENGTHS = {"mix": [5, 41, 17, 70, 130, 23], "odd": [1, 9, 33, 70, 150, 64], "tc": [5, 300, 17, 70, 160, 33], "rec": [2, 19, 90, 35, 60, 77]}
PAGE = {"mix": 16, "odd": 8, "tc": 64, "rec": 32}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name in tl.CONFIGS:
        path, cfg, tensors = tl.make_folder(str(tmp_path_factory.mktemp("li_" + name)), name)
        reqs = {f"r{i}": traces.random_tokens(100 * i + len(name), n, cfg["vocab"]) for i, n in enumerate(LENGTHS[name])}
        ref = {rid: tl.plain_logits(cfg, tensors, t) for rid, t in reqs.items()}
        out[name] = (path, cfg, tensors, reqs, ref)
    return out


_sens = {}


def close(got, ref, dtype, what, cfg, tensors, toks, key):
    """float32: the fixed tolerance.  bfloat16: the fixed tolerance, with the allowance of ``tiny_lilalorn.assert_close_bfloat16``
    for positions that the plain implementation itself shows to hang on a rounding (worked out only where one is needed)."""
    if dtype == "float32":
        return traces.assert_close(got, ref, dtype, what)
    err = np.abs(got.astype(np.float64) - ref).max(axis=1) / float(np.abs(ref).max())
    at = tuple(np.nonzero(err > traces.TOL["bfloat16"]["max_rel"])[0].tolist())
    if at and (key, at) not in _sens:
        _sens[key, at] = tl.rounding_sensitivity(cfg, tensors, toks, at=at)
    tl.assert_close_bfloat16(got, ref, _sens[key, at] if at else np.zeros(len(ref)), what)


def run(folder, dtype, steps, page_size, max_tokens=None, max_requests=4, graphs=True, longest=None):
    from xyntetik_runner_b200.engine.engine import Engine, EngineParams
    from xyntetik_runner_b200.engine.replay import replay
    mt = max_tokens if max_tokens is not None else traces.pool_tokens(steps, page_size)
    eng = Engine(folder, EngineParams(dtype=dtype, max_tokens=mt, page_size=page_size, max_requests=max_requests, cuda_graphs=graphs,
                                      max_request_tokens=longest))
    res = replay(eng, steps)
    eng.check_status()
    eng.cache.audit()
    assert not eng.cache.live_requests()
    return res, eng


CUTS = {
    "whole": lambda reqs: traces.whole(reqs),
    "tail": lambda reqs: traces.tail_decoded(reqs, 32),
    "portions": lambda reqs: traces.portions(reqs),
    "pairs": lambda reqs: traces.portions(reqs, sizes=(2,)),
    "mixed": lambda reqs: traces.mixed(reqs, seed=3),
    "mixed2": lambda reqs: traces.mixed(reqs, seed=8, max_live=2, sizes=(1, 2, 31, 1, 64, 3)),
}


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("name", list(tl.CONFIGS))
def test_float32_matches_plain_in_every_cut(models, name, cut):
    path, cfg, tensors, reqs, ref = models[name]
    steps = CUTS[cut](reqs)
    res, eng = run(path, "float32", steps, PAGE[name])
    got = traces.collect(steps, res, cfg["vocab"])
    for rid in reqs:
        traces.assert_close(got[rid], ref[rid], "float32", f"{name}/{cut}/{rid}")
    if cut.startswith("mixed"):
        assert len(reqs) > 4                                                                         # slots were used again
        if eng.cache.pools:
            assert sum(-(-len(t) // PAGE[name]) for t in reqs.values()) > eng.cache.pools[0].n_pages  # and so were pages


@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
@pytest.mark.parametrize("name", list(tl.CONFIGS))
def test_bfloat16_matches_plain(models, name, cut):
    path, cfg, tensors, reqs, ref = models[name]
    steps = CUTS[cut](reqs)
    res, _ = run(path, "bfloat16", steps, PAGE[name])
    got = traces.collect(steps, res, cfg["vocab"])
    for rid in reqs:
        close(got[rid], ref[rid], "bfloat16", f"{name}/{cut}/{rid}", cfg, tensors, reqs[rid], (name, rid))


def test_a_batch_gives_what_each_request_gives_alone(models):
    """Unequal requests side by side, against each alone: in float32 within the rounding of the sums' order."""
    path, cfg, tensors, reqs, ref = models["mix"]
    alone = traces.collect(CUTS["whole"](reqs), run(path, "float32", CUTS["whole"](reqs), PAGE["mix"])[0], cfg["vocab"])
    steps = CUTS["mixed"](reqs)
    batch = traces.collect(steps, run(path, "float32", steps, PAGE["mix"])[0], cfg["vocab"])
    for rid in reqs:
        scale = np.abs(alone[rid]).max()
        assert np.abs(batch[rid] - alone[rid]).max() <= 2e-5 * scale, rid


def test_recurrences_do_not_depend_on_the_cutting(models):
    """A model of recurrences alone walks token by token: the logits of any two cuttings agree to a few units in the last place."""
    path, cfg, tensors, reqs, ref = models["rec"]
    outs = []
    for cut in ("whole", "pairs", "mixed"):
        steps = CUTS[cut](reqs)
        outs.append(traces.collect(steps, run(path, "float32", steps, PAGE["rec"])[0], cfg["vocab"]))
    for rid in reqs:
        scale = np.abs(outs[0][rid]).max()
        assert np.abs(outs[0][rid] - outs[1][rid]).max() <= 2e-6 * scale and np.abs(outs[0][rid] - outs[2][rid]).max() <= 2e-6 * scale, rid


def test_long_decoding(models):
    """Three tokens at once, then 300 one by one, over many small pages."""
    path, cfg, tensors, _, _ = models["mix"]
    toks = traces.random_tokens(77, 303, cfg["vocab"])
    ref = tl.plain_logits(cfg, tensors, toks)
    steps = traces.tail_decoded({"long": toks}, tail=300)
    for dtype in ("float32", "bfloat16"):
        res, eng = run(path, dtype, steps, page_size=8)
        got = traces.collect(steps, res, cfg["vocab"])["long"]
        close(got, ref, dtype, "long decoding", cfg, tensors, toks, ("mix", "long"))
        if dtype == "float32":
            traces.assert_close(got[:3], ref[:3], dtype, "first tokens")


def test_graphs_change_nothing(models):
    path, cfg, tensors, reqs, ref = models["mix"]
    steps = CUTS["tail"](reqs)
    a, _ = run(path, "bfloat16", steps, PAGE["mix"], graphs=True)
    b, eng = run(path, "bfloat16", steps, PAGE["mix"], graphs=False)
    for k in a:
        assert np.array_equal(a[k], b[k])


def test_decode_steps_are_replayed_and_tensor_core_kernels_ran(models):
    from xyntetik_runner_b200.parts import attention, linear
    path, cfg, tensors, reqs, ref = models["tc"]
    before = (attention.counters["tcgen05"], attention.counters["mma"], linear.counters["tcgen05"])
    _, eng = run(path, "bfloat16", CUTS["tail"]({"r1": reqs["r1"]}), PAGE["tc"])
    after = (attention.counters["tcgen05"], attention.counters["mma"], linear.counters["tcgen05"])
    assert eng.graph_replays > 20
    assert all(b > a for a, b in zip(before, after)), (before, after)


# ---- one mechanism at a time ------------------------------------------------------------------------------------------
_g = tl.gla(1, 6, 8, 4.0, 2)
_l = tl.softmax_side
_r = tl.retention_side
_off = _r(1, 4, 4, (0.5,))                       # (a retention side that the mixer's scale of zero leaves out)
_none = _l(1, 1, 4, 4, 0.5, 0)
SINGLE = {
    "attention": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(6, 2, 12, 20, 0.3, 8), _off, 1.0, 0.0), None)]),
    "attention_scaled_frequencies": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(4, 1, 16, 16, 0.25, 16, 900.0, (4.0, 0.7, 3.0, 30)), _off, 1.0, 0.0), None)]),
    "attention_scale": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(3, 3, 10, 6, 0.4, 10), _off, -1.7, 0.0), None)]),
    "attention_no_rotation": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(2, 1, 24, 8, 0.4, 0), _off, 1.0, 0.0), None)]),
    "retention": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_none, _r(3, 12, 20, (0.9, 0.5, 0.99)), 0.0, 1.0), None)]),
    "retention_scale": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_none, _r(1, 40, 6, (0.97,)), 0.0, 0.3), None)]),
    "retention_without_decay": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_none, _r(2, 8, 9, (1.0, 1.0)), 0.0, 1.0), None)]),
    "both_sides": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(4, 2, 8, 12, 0.3, 4), _r(2, 8, 9, (0.9, 0.8)), 0.7, 1.9), None)]),
    "gated_linear": tl.model(60, 40, 1e-5, [tl.layer(tl.gla(3, 12, 20, 8.0, 6), None)]),
    "gated_linear_no_root": tl.model(60, 40, 1e-5, [tl.layer(tl.gla(2, 40, 9, 1.0, 1), None)]),
    "gated_linear_many_channels": tl.model(60, 40, 1e-5, [tl.layer(tl.gla(1, 150, 7, 20.0, 100), None)]),
    "experts_alone": tl.model(60, 40, 1e-5, [tl.layer(_g, tl.moe(7, 3, 20))]),
    "experts_and_shared": tl.model(60, 40, 1e-5, [tl.layer(_g, tl.moe(5, 2, 20, 12))]),
    "one_expert_chosen": tl.model(60, 40, 1e-5, [tl.layer(_g, tl.moe(4, 1, 16, 40))]),
    "every_expert_chosen": tl.model(60, 40, 1e-5, [tl.layer(_g, tl.moe(3, 3, 16, 16))]),
    "one_expert_in_all": tl.model(60, 40, 1e-5, [tl.layer(_g, tl.moe(1, 1, 16, 16))]),
    "multipliers": tl.model(60, 40, 1e-5, [tl.layer(tl.parallel(_l(2, 2, 8, 8, 0.3, 8), _r(2, 8, 8, (0.9, 0.8)), 0.7, 1.9), tl.moe(4, 2, 16, 24)),
                                           tl.layer(_g, tl.moe(4, 2, 16))], 0.3, 2.5),
    "tensors_used_again": tl.model(60, 40, 1e-5, [tl.layer(_g, None), tl.again(tl.layer(_g, None), 0), tl.again(tl.layer(_g, None), 1)], 0.8),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_one_mechanism_alone(name, dtype):
    cfg = SINGLE[name]
    t = tl.draw(cfg, 7)
    reqs = {"a": traces.random_tokens(3, 45, cfg["vocab"]), "b": traces.random_tokens(4, 9, cfg["vocab"]), "c": traces.random_tokens(5, 1, cfg["vocab"])}
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = tl.make_folder(tmp, None, t, cfg)
        for cut in ("whole", "portions", "mixed"):
            steps = CUTS[cut](reqs)
            res, _ = run(path, dtype, steps, 8)
            got = traces.collect(steps, res, cfg["vocab"])
            for rid in reqs:
                close(got[rid], tl.plain_logits(cfg, t, reqs[rid]), dtype, f"{name}/{cut}/{rid}", cfg, t, reqs[rid], (name, rid))


# ---- kernels alone ------------------------------------------------------------------------------------------------------
def _dev(t, dtype=torch.float32):
    return t.to(dtype).cuda().contiguous()


def _i32(v):
    return torch.tensor(v, dtype=torch.int32).cuda()


# key sizes on both sides of the walk's register tiles, sizes whose rows do not fall on 16 bytes, more value columns than a block has
WALKS = [(3, 12, 20, 5), (4, 16, 16, 16), (2, 33, 10, 3), (1, 64, 100, 8), (2, 100, 36, 70), (4, 128, 64, 16), (2, 130, 33, 4), (1, 256, 48, 130), (1, 1, 1, 1), (9, 30, 18, 12)]


@pytest.mark.parametrize("keyed", [False, True])
@pytest.mark.parametrize("H,D,V,R", WALKS)
def test_walks_from_states_in_other_slots(H, D, V, R, keyed):
    """Two portions in one launch, in slots 2 and 0 of four, one continuing a state that an earlier launch left; whole against cut, bit
    for bit, also where many portions make the walk take more columns a warp; retention's constant decays and decays per key channel."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(H * D + V)
    r = lambda *s: torch.randn(*s, generator=g)
    C, cols = H * D, 2 * H * D + 2 * H * V + R
    lens = (150, 11)
    pre = r(sum(lens), cols)
    a2, b, tau, scale = r(C, R) / R ** 0.5, 1.0 + r(C), 6.0, D ** -0.5
    decay = 0.5 + 0.5 * torch.rand(H, generator=g)
    q, k, v, inner = (pre[:, x:y].double() for x, y in ((0, C), (C, 2 * C), (2 * C, 2 * C + H * V), (cols - R, cols)))
    if keyed:
        a = torch.exp(torch.nn.functional.logsigmoid(inner @ a2.double().T + b.double()) / tau).view(-1, H, D)
    else:
        a = decay.double()[None, :, None].expand(pre.shape[0], H, D)
    cut = lambda x, w, lo, hi: x[lo:hi].reshape(hi - lo, H, w)
    want = [scale * P.decayed_reads(cut(q, D, lo, hi), cut(k, D, lo, hi), cut(v, V, lo, hi), a[lo:hi]).reshape(hi - lo, H * V)
            for lo, hi in ((0, lens[0]), (lens[0], sum(lens)))]
    wide = -(-cols // 8) * 8
    w_t, bias, dec = _dev(a2.T), _dev(b), _dev(decay)

    def launch(state, rows, starts, lns, slots):
        n = rows.shape[0]
        proj = torch.full((n, wide), float("nan")).cuda()[:, :cols]
        proj.copy_(rows)
        o = torch.full((n, H * V), float("nan")).cuda()
        at = (0, C, 2 * C)
        if keyed:
            kernels.key_decay_attention(proj, at + (cols - R,), R, w_t, bias, tau, torch.empty(n, C).cuda(), state, _i32(starts), _i32(lns), _i32(slots), o,
                                        len(lns), H, D, V, read_scale=scale)
        else:
            kernels.decay_attention(proj, at, dec, state, _i32(starts), _i32(lns), _i32(slots), o, len(lns), H, D, V, silu=False, read_scale=scale)
        return o.cpu()

    noise = r(4, H * D * V + 4)                                    # (rows wider than needed, filled with noise)
    state = noise.clone().cuda()
    state[2].zero_(); state[0].zero_()
    n0 = 131
    first = launch(state, pre[:n0], [0], [n0], [2])
    second = launch(state, torch.cat([pre[lens[0]:], pre[n0:lens[0]]]), [0, lens[1]], [lens[1], lens[0] - n0], [0, 2])
    tol = dict(rtol=1e-4, atol=1e-4 * float(want[0].abs().max()))
    assert torch.allclose(first.double(), want[0][:n0], **tol) and torch.allclose(second[:lens[1]].double(), want[1], **tol)
    assert torch.allclose(second[lens[1]:].double(), want[0][n0:], **tol)
    assert torch.equal(state[1].cpu(), noise[1]) and torch.equal(state[3].cpu(), noise[3])            # other slots untouched
    whole = launch(torch.zeros_like(state), pre[:lens[0]], [0], [lens[0]], [3])
    assert torch.equal(whole, torch.cat([first, second[lens[1]:]]))
    one = torch.zeros_like(state)
    assert torch.equal(torch.cat([launch(one, pre[t:t + 1], [0], [1], [1]) for t in range(20)]), whole[:20])
    S = max(4, -(-400 // (H * -(-V // 16))))
    many = launch(torch.zeros(S, state.shape[1]).cuda(), pre[:37].repeat(S, 1), [37 * s for s in range(S)], [37] * S, list(range(S)))
    assert torch.equal(many, whole[:37].repeat(S, 1))


@pytest.mark.parametrize("n", [1, 5, 64, 65, 200])
@pytest.mark.parametrize("R,C,tau", [(1, 3, 1.0), (16, 96, 16.0), (70, 130, 4.0), (200, 1, 9.0)])
def test_decays_per_key_channel_over_their_whole_range(n, R, C, tau):
    """The decays kernel behind a walk of one value column with unit keys: S counts the decays up.  Biases from -80 to 80."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(R + C + n)
    pre, a2 = torch.randn(n, 2 * C + 1 + R, generator=g), torch.randn(C, R, generator=g) / R ** 0.5
    b = torch.linspace(-80.0, 80.0, C) if C > 1 else torch.tensor([0.3])
    decays = torch.full((n, C), float("nan")).cuda()
    kernels.key_decay_attention(_dev(pre), (0, C, 2 * C, 2 * C + 1), R, _dev(a2.T), _dev(b), tau, decays, torch.zeros(1, C).cuda(), _i32([0]), _i32([n]), _i32([0]),
                                torch.empty(n, C).cuda(), 1, C, 1, 1)
    z = pre[:, 2 * C + 1:].double() @ a2.double().T + b.double()
    want = torch.exp(torch.nn.functional.logsigmoid(z) / tau)
    assert torch.allclose(decays.double().cpu(), want, rtol=3e-5, atol=1e-30)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,V", [(3, 12), (8, 128), (1, 200), (5, 7)])
def test_head_norm_without_a_weight_and_with_one_for_all_heads(dtype, H, V):
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(V)
    o, gate, w = torch.randn(17, H * V, generator=g), 3.0 * torch.randn(17, H * V + 3, generator=g), 1.0 + 0.3 * torch.randn(V, generator=g)
    o[3] *= 1e-4                                                   # (eps counts)
    for weight in (None, w):
        y = torch.empty(17, H * V, dtype=dtype).cuda()
        kernels.head_norm_gate(_dev(o), _dev(gate), 3, None if weight is None else _dev(weight), y, H, V, 1e-5, silu=True)
        u = P.unit_rms(o.double().view(17, H, V), 1e-5)
        want = (u if weight is None else u * weight.double()).reshape(17, -1) * P.silu(gate[:, 3:].double())
        assert torch.allclose(y.double().cpu(), want, rtol=1e-5 if dtype == torch.float32 else 1e-2, atol=1e-6 if dtype == torch.float32 else 1e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,E,top,W,F", [(1, 4, 2, 40, 24), (9, 7, 3, 68, 20), (70, 3, 3, 64, 72), (300, 5, 2, 136, 200)])
def test_ungated_experts_over_a_plan(dtype, n, E, top, W, F):
    """The first product takes its token's row and the square of relu, the second the planned rows; both kernels."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(n + E)
    h = torch.randn(n, W, generator=g).to(dtype)
    up, down = (torch.randn(E, F, W, generator=g) / W ** 0.5).to(torch.bfloat16), (torch.randn(E, W, F, generator=g) / F ** 0.5).to(torch.bfloat16)
    ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    want = torch.stack([torch.stack([P.relu2_ff(h[t].double(), up[e].double(), down[e].double()) for e in ids[t].tolist()]) for t in range(n)])
    for tc in ((False,) if dtype == torch.float32 or W % 8 or F % 8 else (False, True)):
        align = 16 if tc else kernels.moe_tile_rows()
        tiles = kernels.moe_max_tiles(n * top, E, align)
        row_src, pair_row, tile_group = (torch.empty(m, dtype=torch.int32).cuda() for m in (tiles * align, n * top, tiles))
        kernels.moe_plan(ids.cuda(), row_src, pair_row, tile_group, E, align)
        y, z = torch.empty(tiles * align, F, dtype=dtype).cuda(), torch.zeros(tiles * align, W).cuda()
        if tc:
            xs = torch.empty(tiles * align, W, dtype=dtype).cuda()
            kernels.moe_gather(h.cuda(), xs, row_src, tile_group, top, align)
            kernels.gemm_tc_grouped(xs, kernels.pack_weight_groups(up.cuda()), y, tile_group, align, F, kernels.EPI_STORE, kernels.ACT_RELU2)
            kernels.gemm_tc_grouped(y, kernels.pack_weight_groups(down.cuda()), z, tile_group, align, W)
            kernels.tc_check_status(y.device)
        else:
            kernels.moe_gemm(h.cuda(), up.cuda(), y, row_src, tile_group, top, False, kernels.ACT_RELU2, gather=True)
            kernels.moe_gemm(y, down.cuda(), z, row_src, tile_group, top, False)
        got = z[pair_row.long()].view(n, top, W).double().cpu()
        assert torch.allclose(got, want, rtol=1e-4 if dtype == torch.float32 else 2e-2, atol=(1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max()))


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,W,top,splits", [(3, 44, 2, 1), (7, 70, 5, 3), (5, 5000, 1, 6), (200, 320, 4, 1), (160, 1028, 3, 2), (1, 4100, 9, 1)])
def test_sum_of_experts_with_a_gated_shared_expert_and_the_norm_behind_it(n, W, top, splits, out_dtype):
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(n + W)
    r = lambda *s: torch.randn(*s, generator=g)
    rows = n * top + 5
    z, wts, x, shared, logits, w = r(rows, W), torch.rand(n, top, generator=g), 3.0 * r(n, W), r(splits, n, W), 2.0 * r(n, 8), 1.0 + 0.2 * r(W)
    pair_row = torch.randperm(rows, generator=g)[:n * top].to(torch.int32)
    parts = (wts.double()[:, :, None] * z.double()[pair_row.long()].view(n, top, W)).sum(1)
    for gated in (None, True, False):                              # no shared expert; under its gate (a column of wider rows); without one
        sh = None if gated is None else _dev(shared)
        gate = _dev(logits)[:, 7] if gated else None
        add = 0 if gated is None else shared.double().sum(0) * (torch.sigmoid(logits[:, 7:].double()) if gated else 1.0)
        want = x.double() + 0.37 * (parts + add)
        outs = []
        for normed in (False, True):
            d = _dev(x)
            out = torch.empty(n, W, dtype=out_dtype).cuda() if normed else None
            kernels.moe_combine(d, _dev(z), _dev(wts), pair_row.cuda(), top, shared=sh, splits=splits if sh is not None else 1, gate=gate, scale=0.37,
                                norm_w=_dev(w) if normed else None, out=out, eps=1e-5)
            outs.append(d.cpu())
            assert torch.allclose(d.double().cpu(), want, rtol=1e-5, atol=1e-5)
        assert torch.equal(outs[0], outs[1])
        assert torch.allclose(out.double().cpu(), P.rms_norm(want, w.double(), 1e-5), rtol=1e-5 if out_dtype == torch.float32 else 1e-2, atol=1e-5 if out_dtype == torch.float32 else 1e-3)


def test_choice_reads_rows_of_a_wider_product():
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(2)
    for E, top in ((7, 3), (40, 40), (33, 1)):
        z = torch.randn(50, E + 1, generator=g) * 2
        z[:, E] = 99.0                                             # (the gate's column must not be chosen)
        ids, wts = torch.empty(50, top, dtype=torch.int32).cuda(), torch.empty(50, top).cuda()
        kernels.route_topk(_dev(z)[:, :E], ids, wts, top)
        s = torch.softmax(z[:, :E].double(), dim=-1)
        got = ids.cpu().long()
        assert torch.equal(got.sort(1).values, torch.topk(s, top, dim=-1).indices.sort(1).values)
        p = torch.gather(s, 1, got)
        assert torch.allclose(wts.double().cpu(), p / (p.sum(1, keepdim=True) + 1e-20), rtol=1e-5)


@pytest.mark.parametrize("n", [1, 7, 100, 300])
def test_a_factor_on_the_products_sums(n):
    """Stored and added, whole and cut along K, the sum left to the caller, ahead of bias and activation; FMA and tcgen05."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(n)
    x, w, b, x0 = torch.randn(n, 512, generator=g), torch.randn(136, 512, generator=g) / 16, torch.randn(136, generator=g), torch.randn(n, 136, generator=g)
    xb, wb = x.to(torch.bfloat16), w.to(torch.bfloat16)
    exact = xb.double() @ wb.double().T
    tol = dict(rtol=1e-4, atol=1e-4)
    out = _dev(x0)
    kernels.gemm_simt(xb.cuda(), wb.cuda(), out, _dev(b), True, -0.3)
    assert torch.allclose(out.double().cpu(), x0.double() - 0.3 * exact + b.double(), **tol)
    for splits in (1, 3):
        out = _dev(x0)
        kernels.gemm_tc(xb.cuda(), wb.cuda(), out, _dev(b), kernels.EPI_ADD, force_splits=splits, alpha=-0.3)
        assert torch.allclose(out.double().cpu(), x0.double() - 0.3 * exact + b.double(), **tol)
        out = torch.empty(n, 136).cuda()
        kernels.gemm_tc(xb.cuda(), wb.cuda(), out, _dev(b), kernels.EPI_STORE, force_splits=splits, act=kernels.ACT_RELU2, alpha=2.5)
        assert torch.allclose(out.double().cpu(), torch.relu(2.5 * exact + b.double()) ** 2, rtol=1e-3, atol=1e-3)
    out = _dev(x0)
    sums = kernels.gemm_tc_deferred(xb.cuda(), wb.cuda(), out, None, kernels.EPI_ADD, force_splits=4, alpha=0.7)
    kernels.finish_plain(sums.partial, sums.splits, None, out, True)
    sums.release()
    kernels.tc_check_status(out.device)
    assert torch.allclose(out.double().cpu(), x0.double() + 0.7 * exact, **tol)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,K,D,Vd,dims", [(4, 2, 24, 16, 16), (2, 1, 64, 64, 64), (3, 3, 10, 13, 10), (2, 2, 64, 128, 32)])
def test_rotation_with_scaled_frequencies_far_out(dtype, H, K, D, Vd, dims):
    """Angles are float64 products: at position 200,000 the rotation is as exact as at 3; no norm, values beside the keys untouched."""
    from xyntetik_runner_b200 import kernels
    from xyntetik_runner_b200.config.llama import RopeScaling
    from xyntetik_runner_b200.parts import Rope
    g = torch.Generator().manual_seed(D + Vd)
    page, hd, cols = 8, -(-max(D, Vd) // 16) * 16, (H + K) * D + K * Vd
    rope = Rope(D, 7000.0, rotary_dim=dims, scaling=RopeScaling(rope_type="llama3", factor=6.0, low_freq_factor=1.0, high_freq_factor=4.0,
                                                                original_max_position_embeddings=64))
    pos = [0, 3, 15, 4096, 65537, 199999]
    n = len(pos)
    pages = max(pos) // page + 1
    bt = torch.full((n, pages), -1, dtype=torch.int32)
    for t, p in enumerate(pos):
        bt[t, p // page] = t                                       # each token its own request and page
    rows = torch.randn(n, cols, generator=g).to(dtype)
    inp = torch.zeros(n, -(-cols // 8) * 8, dtype=dtype).cuda()[:, :cols]
    inp.copy_(rows)
    cache, q_out = torch.zeros(n, 1, 2, K, page, hd, dtype=dtype).cuda(), torch.zeros(n, H * hd, dtype=dtype).cuda()
    kernels.qk_norm_rope_store(inp, q_out, _i32(pos), _i32(list(range(n))), bt.cuda(), torch.from_numpy(rope.inv_freq64_host).cuda(), None, None,
                               cache.data_ptr(), cache.stride(0), cache.stride(2), H, K, D, Vd, hd, dims, pages, page, False, 1e-6)
    freq = P.frequencies(dims, 7000.0, {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 64}, torch.float64)
    r = rows.double()
    rot = lambda v: P.rotate(v, torch.tensor(pos), dims, freq)
    tol = dict(rtol=1e-5, atol=2e-6) if dtype == torch.float32 else dict(rtol=1e-2, atol=2e-2)
    assert torch.allclose(q_out.double().cpu().view(n, H, hd)[:, :, :D], rot(r[:, :H * D].view(n, H, D)), **tol)
    at = torch.stack([cache[t, 0, :, :, p % page] for t, p in enumerate(pos)]).double().cpu()
    assert torch.allclose(at[:, 0, :, :D], rot(r[:, H * D:(H + K) * D].view(n, K, D)), **tol)
    assert torch.equal(at[:, 1, :, :Vd].reshape(n, -1), r[:, (H + K) * D:]) and at[:, 0, :, D:].abs().sum() == 0 and at[:, 1, :, Vd:].abs().sum() == 0


# ---- keys that stand out ---------------------------------------------------------------------------------------------------
def _echo_model(dim, vdim, heads, kv_heads, scale, rot_dims=2):
    """One parallel mixer in which an odd token asks for the even one below it: queries read the first half of the embedding, keys the
    second half, by the same matrix, and an odd token's first half is the second half of its even one.  The score of that pair is
    about dim * scale whatever lies between them (few elements are rotated), all others scatter around zero."""
    cfg = tl.model(700, 64, 1e-6, [tl.layer(tl.parallel(_l(heads, kv_heads, dim, vdim, scale, rot_dims), _r(2, 8, 8, (0.9, 0.95)), 2.0, 0.2), None)])
    t = tl.draw(cfg, 50)
    t["embed"][1::2, :32] = t["embed"][0::2, 32:]
    t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
    p = "l0.mix.left."
    base = 2.0 ** 0.5 * t[p + "q"][:dim, :32].float()
    q, k = torch.zeros(heads * dim, 64), torch.zeros(kv_heads * dim, 64)
    q[:, :32], k[:, 32:] = base.repeat(heads, 1), base.repeat(kv_heads, 1)
    t[p + "q"], t[p + "k"] = q.to(torch.bfloat16), k.to(torch.bfloat16)
    t[p + "v"] = t[p + "v"] * 3.0
    return cfg, t


def _echo_tokens(n, at, seed):
    """n tokens, the last an odd one that asks for the one at position `at`; the rest are other tokens."""
    rng = np.random.RandomState(seed)
    pair = int(rng.randint(0, 350))
    toks = [int(v) for v in rng.permutation([v for v in range(700) if v // 2 != pair])[:n]]
    toks[at], toks[-1] = 2 * pair, 2 * pair + 1
    return toks


@pytest.mark.parametrize("dim,vdim,heads,kv_heads,scale,page,n", [(32, 24, 2, 2, 0.6, 16, 150), (64, 64, 4, 2, 0.3, 64, 420), (128, 128, 8, 1, 0.15, 64, 420), (40, 80, 6, 1, 0.4, 16, 300)])
def test_a_key_that_stands_out_wherever_it_lies(dim, vdim, heads, kv_heads, scale, page, n):
    """The asking token is the last: places at the start, at the borders of pages and tiles, far back and right before it, in a prompt,
    decoded alone and behind portions of two."""
    cfg, t = _echo_model(dim, vdim, heads, kv_heads, scale)
    places = sorted({p for p in (0, 1, page - 1, page, 2 * page - 1, 2 * page, 63, 64, 127, 128, n // 2, n - page - 1, n - 3, n - 2) if 0 <= p < n - 1})
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = tl.make_folder(tmp, None, t, cfg)
        reqs, ref = {}, {}
        for at in places:
            # tokens whose pair is a strong one: without the asked-for key the last logits are others
            for seed in range(at, at + 50000, 1000):
                toks = _echo_tokens(n, at, seed)
                other = list(toks)
                other[at] = next(v for v in range(0, 700, 2) if v not in other)
                full = tl.plain_logits(cfg, t, toks)
                if np.abs(tl.plain_logits(cfg, t, other)[-1] - full[-1]).max() > 0.1 * np.abs(full).max():
                    break
            else:
                raise AssertionError(f"no strong pair for place {at}")
            reqs[f"p{at}"], ref[f"p{at}"] = toks, full
        cuts = [("whole", "float32"), ("tail", "float32"), ("mixed", "float32"), ("whole", "bfloat16"), ("tail", "bfloat16")]
        for cut, dtype in cuts + ([("pairs", "float32")] if n < 200 else []):
            steps = CUTS[cut](reqs)
            res, _ = run(path, dtype, steps, page)
            got = traces.collect(steps, res, cfg["vocab"])
            for rid in reqs:
                close(got[rid], ref[rid], dtype, f"echo {rid}/{cut}/{dtype}", cfg, t, reqs[rid], ("echo", dim, rid))


@pytest.mark.parametrize("kind", ["gla", "retention"])
def test_slow_recurrences_remember_the_first_tokens_in_a_slot_used_before(kind):
    """Decays near one: changing the FIRST tokens changes the logits 200 tokens later, and the engine follows, in a slot that another
    request used before and across decoded tokens."""
    if kind == "gla":
        cfg = tl.CONFIGS["rec"]
    else:
        cfg = tl.model(90, 64, 1e-5, [tl.layer(tl.parallel(_none, _r(2, 8, 12, (0.9995, 1.0)), 0.0, 1.0), None)])
    t = tl.draw(cfg, 61, slow=True)
    a = traces.random_tokens(1, 230, cfg["vocab"])
    b = [(a[0] + 1) % cfg["vocab"], (a[1] + 7) % cfg["vocab"]] + a[2:]
    ra, rb = tl.plain_logits(cfg, t, a), tl.plain_logits(cfg, t, b)
    assert np.abs(ra[-1] - rb[-1]).max() > 1e-3 * np.abs(ra).max()
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = tl.make_folder(tmp, None, t, cfg)
        steps = traces.tail_decoded({"a": a, "b": b}, 40)
        res, _ = run(path, "float32", steps, 16, max_requests=1)
        got = traces.collect(steps, res, cfg["vocab"])
        traces.assert_close(got["a"], ra, "float32", "slow a")
        traces.assert_close(got["b"], rb, "float32", "slow b")
        assert np.abs(got["b"][-1] - rb[-1]).max() < 0.05 * np.abs(ra[-1] - rb[-1]).max()


# ---- other sizes -------------------------------------------------------------------------------------------------------------
def _drawn_config(rng, layer_sizes):
    pick = lambda *v: v[rng.randint(len(v))]
    W = int(pick(128, 192, 256)) if layer_sizes else int(pick(36, 52, 68, 70, 96))
    layers = []
    for i in range(rng.randint(1, 7)):
        own = [j for j in range(i) if rng.rand() < 0.25]
        if own:
            layers.append(tl.again({k: v for k, v in layers[own[0]].items() if k != "weights_of"}, own[0]))
            continue
        if rng.rand() < 0.55:
            G = int(pick(1, 2, 3))
            H, D = G * int(pick(1, 2, 8 if layer_sizes else 4)), int(pick(48, 64, 128)) if layer_sizes else int(pick(6, 10, 16, 24, 34))
            Vd = int(pick(64, 80, 128)) if layer_sizes else int(pick(4, 12, 16, 30))
            scaling = (float(pick(2.0, 8.0)), 1.0, float(pick(2.0, 4.0)), int(pick(32, 100, 1000))) if rng.rand() < 0.7 else None
            left = _l(H, G, D, Vd, float(pick(0.1, 0.3, D ** -0.5)), int(pick(D, D // 4 * 2, 0, 4)), float(pick(100.0, 10000.0, 500000.0)), scaling)
            rh = int(pick(1, 2, 3, 5))
            right = _r(rh, int(pick(4, 16, 33, 64)), int(pick(4, 8, 30, 64)), [float(v) for v in 1.0 - 2.0 ** -rng.uniform(0.5, 9, size=rh)])
            mixer = tl.parallel(left, right, float(pick(0.5, 1.0, 1.4)), float(pick(0.3, 1.0, 1.2)))
        else:
            mixer = tl.gla(int(pick(1, 2, 3)), int(pick(8, 24, 33, 64, 100)), int(pick(4, 16, 30, 64)), float(pick(1.0, 6.0, 16.0)), int(pick(1, 8, 16, 40)))
        E = int(pick(1, 2, 5, 8, 16))
        mlp = None if rng.rand() < 0.2 else tl.moe(E, int(rng.randint(1, min(E, 4) + 1)), int(pick(8, 24, 64)), None if rng.rand() < 0.2 else int(pick(8, 40, 64)))
        layers.append(tl.layer(mixer, mlp))
    return tl.model(int(pick(61, 128, 333)), W, float(pick(1e-6, 1e-5)), layers, float(pick(0.3, 0.7, 1.0)), float(pick(0.5, 1.0, 3.0)))


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(seed):
    rng = np.random.RandomState(5000 + seed)
    cfg = _drawn_config(rng, layer_sizes=seed >= 10)
    t = tl.draw(cfg, 90 + seed)
    page = int(rng.choice([4, 8, 16, 64])) if seed < 10 else 64
    reqs = {f"r{i}": traces.random_tokens(11 * seed + i, n, cfg["vocab"]) for i, n in enumerate((3, 90, 17, 140, 1, 45))}
    ref = {rid: tl.plain_logits(cfg, t, toks) for rid, toks in reqs.items()}
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = tl.make_folder(tmp, None, t, cfg)
        for dtype in ("float32", "bfloat16"):
            for cut in ("whole", "mixed"):
                steps = CUTS[cut](reqs)
                res, _ = run(path, dtype, steps, page)
                got = traces.collect(steps, res, cfg["vocab"])
                for rid in reqs:
                    close(got[rid], ref[rid], dtype, f"drawn {seed}/{cut}/{dtype}/{rid}: {cfg['layers']}", cfg, t, reqs[rid], ("drawn", seed, rid))


# ---- entry points ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(models, dtype):
    from xyntetik_runner_b200.engine.runner import Runner
    path, cfg, tensors, _, _ = models["mix"]
    prompts = [traces.random_tokens(i + 40, n, cfg["vocab"]) for i, n in enumerate((5, 11, 17, 3, 30))]
    r = Runner(path, dtype=dtype, ctx=128, parallel=3, page_size=16)          # five requests over three slots
    res = r.generate(prompts, n=12, temp=0.0, ignore_eos=True)
    for p, g in zip(prompts, res):
        assert len(g.tokens) == 12 and g.finish_reason == "length"
        if dtype == "float32":
            assert g.tokens == tl.plain_greedy(cfg, tensors, p, 12)
        else:
            # teacher-forced: every token is the plain argmax for the engine's own prefix, or within rounding of it
            for i, tok in enumerate(g.tokens):
                toks = list(p) + list(g.tokens[:i])
                ref = tl.plain_logits(cfg, tensors, toks)
                miss = (ref[-1].max() - ref[-1][tok]) / np.abs(ref).max()
                assert miss <= 0.06 or miss <= 6.0 * tl.rounding_sensitivity(cfg, tensors, toks, at=(len(toks) - 1,))[-1], (i, miss)


def test_command_line_generates_what_the_plain_implementation_does(models):
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    path, cfg, tensors, _, _ = models["odd"]
    prompt = traces.random_tokens(9, 7, cfg["vocab"])
    ids = "ids:" + ",".join(str(t) for t in prompt)
    out = {}
    for extra in (["--dtype", "float32"], ["--ref"]):
        r = subprocess.run([sys.executable, os.path.join(root, "bin", "runner"), "-m", path, "-p", ids, "-n", "6", "--ignore-eos"] + extra,
                           capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        out[extra[-1]] = [ln for ln in r.stdout.splitlines() if ln.startswith("ids:")][0]
    want = "ids:" + ",".join(str(t) for t in tl.plain_greedy(cfg, tensors, prompt, 6))
    assert out["--ref"] == want and out["float32"] == want, out


def test_trace_runner_program(models):
    """bin/trace_run on a folder: steps on standard input, logits in files, a line per step."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    path, cfg, tensors, reqs, ref = models["mix"]
    steps = traces.mixed(reqs, seed=5)
    with tempfile.TemporaryDirectory() as out:
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", out, "--max-tokens",
                            str(traces.pool_tokens(steps, 64))], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=900)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [ln for ln in r.stdout.splitlines() if ln.startswith("done ")] == [f"done {s['step']}" for s in steps]
        res = {s["step"]: np.fromfile(os.path.join(out, f"{s['step']}.f32"), dtype="<f4") for s in steps}
    got = traces.collect(steps, res, cfg["vocab"])
    for rid in reqs:
        traces.assert_close(got[rid], ref[rid], "float32", f"trace_run/{rid}")
