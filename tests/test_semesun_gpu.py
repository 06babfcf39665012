"""Semesun on the GPU against the plain implementation: every way of cutting a request, mixed batches with pages and slots used
again, each mechanism alone, the kernels alone (attention over windows with kept first keys and a bias by distance on every path,
the state-space recurrence from states in other slots, the choice by groups, shared values), token sequences made so that one key
stands out far back, at page borders and just inside and outside every window and the kept tokens, recurrences whose first tokens
still count hundreds of tokens later, long decoding in a small pool, other sizes, greedy generation through the entry points."""
import json
import os
import subprocess
import sys
import tempfile

import numpy as np
import pytest
import torch

import plain_semesun as P
import tiny_semesun as ts
import traces

pytestmark = pytest.mark.gpu

LENGTHS = {"mix": [5, 41, 17, 70, 130, 23], "odd": [1, 9, 33, 70, 150, 64], "tc": [5, 300, 17, 70, 160, 33], "rec": [2, 19, 90, 35, 60, 77]}
PAGE = {"mix": 16, "odd": 8, "tc": 64, "rec": 32}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name in ts.CONFIGS:
        path, cfg, tensors = ts.make_folder(str(tmp_path_factory.mktemp("sm_" + name)), name)
        reqs = {f"r{i}": traces.random_tokens(100 * i + len(name), n, cfg["vocab"]) for i, n in enumerate(LENGTHS[name])}
        ref = {rid: ts.plain_logits(cfg, tensors, t) for rid, t in reqs.items()}
        out[name] = (path, cfg, tensors, reqs, ref)
    return out


_sens = {}


def close(got, ref, dtype, what, cfg, tensors, toks, key):
    """float32: the fixed tolerance.  bfloat16: the fixed tolerance, with the allowance of ``tiny_semesun.assert_close_bfloat16``
    for positions that the plain implementation itself shows to hang on a rounding (worked out only where one is needed)."""
    if dtype == "float32":
        return traces.assert_close(got, ref, dtype, what)
    if key not in _sens:
        try:
            return ts.assert_close_bfloat16(got, ref, np.zeros(len(ref)), what)
        except AssertionError:
            _sens[key] = ts.rounding_sensitivity(cfg, tensors, toks)
    ts.assert_close_bfloat16(got, ref, _sens[key], what)


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
@pytest.mark.parametrize("name", list(ts.CONFIGS))
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
@pytest.mark.parametrize("name", list(ts.CONFIGS))
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


def test_long_decoding_in_a_small_pool(models):
    """Three tokens at once, then 300 one by one, in a pool that holds only the windows and the kept tokens: pages behind the windows
    go and are used again while the kept first pages stay."""
    path, cfg, tensors, _, _ = models["mix"]
    toks = traces.random_tokens(77, 303, cfg["vocab"])
    ref = ts.plain_logits(cfg, tensors, toks)
    steps = traces.tail_decoded({"long": toks}, tail=300)
    for dtype in ("float32", "bfloat16"):
        res, eng = run(path, dtype, steps, page_size=8, max_tokens=64, longest=320)
        got = traces.collect(steps, res, cfg["vocab"])["long"]
        close(got, ref, dtype, "long decoding", cfg, tensors, toks, ("mix", "long"))
        if dtype == "float32":
            traces.assert_close(got[:3], ref[:3], dtype, "first tokens")
        assert all(p.n_pages == 8 for p in eng.cache.pools)


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
_a = ts.attention
_m = ts.mamba2(1, 8, 4, 1, 1, 1)
SINGLE = {
    "window_and_kept": ts.model(60, 40, 1e-5, [ts.layer(_a(6, 2, 12, 20, 0.3, 7, 4, 40, 8), None)]),
    "window_of_one_and_kept": ts.model(60, 40, 1e-5, [ts.layer(_a(2, 2, 16, 16, 0.25, 1, 1, 5, 2), None)]),
    "kept_more_than_the_window": ts.model(60, 40, 1e-5, [ts.layer(_a(3, 1, 24, 8, 0.4, 5, 20, 9, 6), None)]),
    "window_longer_than_everything": ts.model(60, 40, 1e-5, [ts.layer(_a(3, 1, 24, 8, 0.4, 1000, 3, 25, 14), None)]),
    "no_window": ts.model(60, 40, 1e-5, [ts.layer(_a(4, 1, 16, 24, 0.2, None, 0, 33, 10), None)]),
    "shared_values": ts.model(60, 40, 1e-5, [ts.layer(_a(2, 2, 8, 12, 0.5, 9, 2, 10, 4, True), None), ts.layer(_a(2, 1, 8, 12, 0.5, 9, 2, 10, 4), None),
                                             ts.layer(_a(4, 1, 10, 24, 0.5, 6, 0, 10, 4, True), None), ts.layer(_a(6, 3, 10, 8, 0.5, 30, 1, 7, 6, True), None)]),
    "recurrence": ts.model(60, 40, 1e-5, [ts.layer(ts.mamba2(6, 8, 12, 2, 4, 3), None)]),
    "recurrence_one_tap_one_head": ts.model(60, 40, 1e-5, [ts.layer(ts.mamba2(1, 30, 7, 1, 1, 5), None)]),
    "recurrence_many_taps_many_states": ts.model(60, 40, 1e-5, [ts.layer(ts.mamba2(4, 6, 150, 4, 9, 2), None)]),
    "dense_feed_forward": ts.model(60, 40, 1e-5, [ts.layer(_m, ts.dense(52))]),
    "experts_alone": ts.model(60, 40, 1e-5, [ts.layer(_m, ts.moe(7, 3, 20, 0.7))]),
    "identity_experts": ts.model(60, 40, 1e-5, [ts.layer(_m, ts.moe(2, 3, 20, 0.7, identity=5, scale=3.0))]),
    "experts_by_groups": ts.model(60, 40, 1e-5, [ts.layer(_m, ts.moe(10, 4, 16, 2.0, identity=2, groups=(6, 3), scale=0.5))]),
    "every_output_chosen": ts.model(60, 40, 1e-5, [ts.layer(_m, ts.moe(3, 5, 16, 2.0, identity=2, scale=1.3))]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SINGLE))
def test_one_mechanism_alone(name, dtype):
    cfg = SINGLE[name]
    t = ts.draw(cfg, 7)
    reqs = {"a": traces.random_tokens(3, 45, cfg["vocab"]), "b": traces.random_tokens(4, 9, cfg["vocab"]), "c": traces.random_tokens(5, 1, cfg["vocab"])}
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = ts.make_folder(tmp, None, t, cfg)
        for cut in ("whole", "portions", "mixed"):
            steps = CUTS[cut](reqs)
            res, _ = run(path, dtype, steps, 8)
            got = traces.collect(steps, res, cfg["vocab"])
            for rid in reqs:
                close(got[rid], ts.plain_logits(cfg, t, reqs[rid]), dtype, f"{name}/{cut}/{rid}", cfg, t, reqs[rid], (name, rid))


# ---- kernels alone ------------------------------------------------------------------------------------------------------
def _dev(t, dtype=torch.float32):
    return t.to(dtype).cuda().contiguous()


def _i32(v):
    return torch.tensor(v, dtype=torch.int32).cuda()


class AttentionCase:
    """Requests with random keys and values in scattered pages; a portion of each is the step.  Values are drawn with a few large
    ones among them, so that a single key too many or too few shows; pages that no visible key lies in are not held (their rows in
    the table are -1), and rows nobody may read hold large numbers."""

    def __init__(self, seed, H, K, hd, page, window, keep, bias_len, segs, dtype, layers=2):
        g = torch.Generator().manual_seed(seed)
        self.H, self.K, self.hd, self.page, self.window, self.keep, self.segs, self.dtype, self.layers = H, K, hd, page, window, keep, segs, dtype, layers
        self.layer = layers - 1
        r = lambda *s: torch.randn(*s, generator=g)
        longest = max(p0 + n for p0, n in segs)
        self.max_pages = -(-longest // page) + 1
        n_pages = sum(-(-(p0 + n) // page) for p0, n in segs) + 3
        order = torch.randperm(n_pages, generator=g).tolist()
        cache = 50.0 * r(n_pages, layers, 2, K, page, hd)
        bt = torch.full((len(segs), self.max_pages), -1, dtype=torch.int32)
        self.bias = None if bias_len is None else 1.5 * r(H, bias_len)
        self.scale = 1.0 / hd ** 0.5
        qs, want = [], []
        for si, (p0, n) in enumerate(segs):
            T = p0 + n
            k, v = r(K, T, hd).to(dtype), (r(K, T, hd) * (1.0 + 15.0 * (torch.rand(T, generator=g) < 0.15).float())[None, :, None]).to(dtype)
            q = r(n, H, hd).to(dtype)
            for pi in range(-(-T // page)):
                lo = max(0, p0 - window + 1) if window else 0
                if window and (pi + 1) * page <= lo and pi * page >= keep:
                    continue                                       # behind the window of every query of the step, and not kept
                p = order.pop()
                bt[si, pi] = p
                rows = min(page, T - pi * page)
                cache[p, self.layer, 0, :, :rows] = k[:, pi * page:pi * page + rows].float()
                cache[p, self.layer, 1, :, :rows] = v[:, pi * page:pi * page + rows].float()
            i, j = torch.arange(p0, T)[:, None], torch.arange(T)[None, :]
            see = (j <= i) & ((i - j < window) | (j < keep)) if window else j <= i
            s = torch.einsum("ihd,hjd->hij", q.double(), k.double().repeat_interleave(H // K, 0)) * self.scale
            if self.bias is not None:
                s = s + self.scale * self.bias.double()[:, (i - j).clamp(0, bias_len - 1)]
            p = torch.softmax(s.masked_fill(~see, float("-inf")), -1)
            want.append(torch.einsum("hij,hjd->ihd", p, v.double().repeat_interleave(H // K, 0)).reshape(n, H * hd))
            qs.append(q.reshape(n, H * hd))
        self.want, n = torch.cat(want), sum(m for _, m in segs)
        self.n = n
        self.qkv = torch.zeros(n, (H + 2 * K) * hd, dtype=dtype).cuda()
        self.qkv[:, :H * hd] = torch.cat(qs).cuda()
        self.cache = cache.to(dtype).cuda()
        starts = np.cumsum([0] + [m for _, m in segs])[:-1]
        self.seg_len_host = np.asarray([m for _, m in segs])
        self.seg_start, self.seg_len, self.seg_pos0 = _i32(starts.tolist()), _i32([m for _, m in segs]), _i32([p for p, _ in segs])
        self.positions = _i32([p0 + t for p0, m in segs for t in range(m)])
        self.tok_seg = _i32([si for si, (_, m) in enumerate(segs) for _ in range(m)])
        self.bt = bt.cuda()
        self.kw = dict(keep_first=keep, bias=None if self.bias is None else _dev(self.bias))
        es = self.cache.element_size()
        self.k_ptr = self.cache.data_ptr() + self.layer * self.cache.stride(1) * es
        self.strides = (self.cache.stride(0), self.cache.stride(2))

    def out(self):
        return torch.full((self.n, self.H * self.hd), float("nan"), dtype=self.dtype).cuda()

    def simt(self):
        from xyntetik_runner_b200 import kernels
        o = self.out()
        kernels.attention_simt(self.qkv, self.qkv.shape[1], o, self.k_ptr, self.positions, self.tok_seg, self.bt, *self.strides, self.H, self.K, self.hd,
                               self.max_pages, self.page, self.window, self.scale, **self.kw)
        return o

    def mma(self, bulk=True, uneven=False):
        from xyntetik_runner_b200 import kernels
        o, G, S = self.out(), self.H // self.K, len(self.segs)
        rows = self.seg_len_host * G
        kv = max(p + m for p, m in self.segs)
        splits = kernels.attention_mma_splits(kv, self.window, S * self.K)
        pa, pm = torch.empty(S * self.K * splits * 16 * self.hd).cuda(), torch.empty(S * self.K * splits * 32).cuda()
        kernels.attention_mma(self.qkv, self.qkv.shape[1], o, self.k_ptr, self.seg_start, self.seg_len, self.seg_pos0, self.bt, pa, pm, *self.strides,
                              self.H, self.K, self.hd, self.max_pages, self.page, self.window, self.scale, S, int(self.seg_len_host.max()), kv, splits,
                              bool((rows <= 16).any()), bool((rows > 16).any()),
                              group=(self.cache.data_ptr(), self.cache.shape[0], self.layers, self.layer) if bulk else None, uneven=uneven,
                              row_tiles=kernels.long_row_tiles(self.seg_len_host, G, 64), **self.kw)
        return o

    def tc(self):
        from xyntetik_runner_b200 import kernels
        o, G = self.out(), self.H // self.K
        kernels.attention_tc(self.qkv, o, self.seg_start, self.seg_len, self.seg_pos0, self.bt, (self.cache.data_ptr(), self.cache.shape[0], self.layers, self.layer),
                             self.H, self.K, self.hd, self.max_pages, self.page, self.window, self.scale, len(self.segs), int(self.seg_len_host.max()),
                             row_tiles=kernels.long_row_tiles(self.seg_len_host, G, 128), **self.kw)
        return o

    def check(self, o, what, only=None):
        from xyntetik_runner_b200 import kernels
        kernels.tc_check_status(o.device)
        got = o.double().cpu()
        diff = (got - self.want).abs()
        rows = slice(None) if only is None else only
        tol = 1e-4 if self.dtype == torch.float32 else 0.12
        assert torch.isfinite(got[rows]).all(), what
        bad = (diff[rows] > tol * (1.0 + 0.1 * self.want[rows].abs())).any(dim=1)
        assert not bad.any(), f"{what}: {int(bad.sum())} rows, worst {diff[rows].max():.3f}, first {int(bad.nonzero()[0])}"


# (window, keep, bias entries): windows and kept tokens on, one below and one above tiles of 64 and 128 and pages; bias tables that end
# inside the window, beyond it, and at once
MASKS = [(0, 0, 40), (5, 0, None), (5, 3, 7), (64, 1, 64), (65, 64, 300), (63, 65, 1), (100, 130, 90), (128, 6, 200), (129, 128, 33), (200, 150, None), (1, 2, 5)]


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("window,keep,bias_len", MASKS)
def test_float32_attention_over_windows_kept_keys_and_bias(window, keep, bias_len, page):
    segs = [(0, 70), (131, 40), (300, 1), (64, 1), (0, 1), (190, 13), (7, 1), (500, 2)]
    c = AttentionCase(window + page, 6, 2, 20, page, window, keep, bias_len, segs, torch.float32)
    c.check(c.simt(), "simt")


@pytest.mark.parametrize("hd,H,K,page", [(64, 8, 2, 64), (128, 4, 4, 64), (64, 16, 1, 16), (128, 16, 2, 64), (48, 6, 2, 16), (80, 3, 1, 64)])
@pytest.mark.parametrize("window,keep,bias_len", MASKS)
def test_prompt_attention_over_windows_kept_keys_and_bias(window, keep, bias_len, hd, H, K, page):
    from xyntetik_runner_b200 import kernels
    segs = [(0, 300), (131, 140), (300, 77), (63, 66), (700, 129), (128, 128)]
    c = AttentionCase(window + hd + H, H, K, hd, page, window, keep, bias_len, segs, torch.bfloat16)
    c.check(c.simt(), "simt")
    c.check(c.mma(), "rows kernel")
    if kernels.attention_tc_supported(torch.bfloat16, H, K, hd, page):
        c.check(c.tc(), "tcgen05")


@pytest.mark.parametrize("hd,H,K,page", [(64, 8, 2, 64), (128, 4, 4, 64), (64, 16, 1, 16), (128, 16, 2, 8), (48, 6, 2, 16), (96, 4, 1, 5)])
@pytest.mark.parametrize("window,keep,bias_len", MASKS)
def test_decode_attention_over_windows_kept_keys_and_bias(window, keep, bias_len, hd, H, K, page):
    """Single tokens and portions of a few rows, at positions around windows' edges, the kept tokens and page borders: copies by
    threads and bulk copies; few requests (spans in clusters), more (one span each)."""
    m = max(1, 16 // (H // K))
    edges = sorted({p for e in (window, keep, window + keep, 64, 128, 192) for p in (e - 2, e - 1, e, e + 1) if p >= 0})
    for segs in ([(700, 1), (333, min(2, m))], [(p, 1) for p in edges] + [(1000, min(3, m)), (0, 1), (1500, 1)]):
        c = AttentionCase(window + hd + len(segs), H, K, hd, page, window, keep, bias_len, segs, torch.bfloat16)
        c.check(c.mma(bulk=False), "copies by threads")
        c.check(c.mma(), "bulk copies")


@pytest.mark.parametrize("hd,H,K", [(64, 4, 2), (128, 8, 4)])
@pytest.mark.parametrize("window,keep,bias_len", [(0, 0, 50), (100, 70, 60), (65, 3, None), (300, 1, 400)])
def test_decode_attention_in_even_shares(window, keep, bias_len, hd, H, K):
    from xyntetik_runner_b200 import kernels
    rng = np.random.RandomState(window + hd)
    segs = [(int(p), 1) for p in rng.randint(0, 900, size=-(-300 // K))]
    c = AttentionCase(hd, H, K, hd, 64, window, keep, bias_len, segs, torch.bfloat16)
    before = kernels.attention_even_launches()
    o = c.mma(uneven=True)
    assert kernels.attention_even_launches() == before + 1
    c.check(o, "even shares")
    assert int(kernels.workspace(o.device).flags.abs().sum()) == 0


@pytest.mark.parametrize("H,G,N,V,taps", [(6, 2, 12, 20, 4), (4, 1, 64, 64, 4), (2, 2, 130, 33, 3), (8, 2, 128, 16, 4), (3, 3, 7, 5, 1), (4, 2, 40, 24, 9)])
def test_recurrence_kernel_from_states_in_other_slots(H, G, N, V, taps):
    """Two portions in one launch, in slots 2 and 0 of four, one continuing a state and a tail that an earlier launch left; whole
    against cut, bit for bit; the gated group norm behind it."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(H * N + taps)
    CH, inner = H * V + 2 * G * N, H * V
    r = lambda *s: torch.randn(*s, generator=g)
    groups = 2 if inner % 2 == 0 else 1
    w = {"conv": r(CH, taps), "conv.b": r(CH), "dt_bias": r(H) - 1.0, "A_log": r(H) - 0.5, "D": r(H), "norm": 1.0 + 0.2 * r(inner)}
    lens = (150, 11)
    pre = r(sum(lens), inner + CH + H)

    def plain(rows):
        ww = {k: v.double() for k, v in w.items()}
        ww["in"], ww["o"] = torch.eye(rows.shape[1]).double(), torch.eye(inner).double()
        return P.mamba2(rows.double(), ww, {"heads": H, "vdim": V, "state": N, "groups": G, "norm_groups": groups}, 1e-5, {})

    want = [plain(pre[:lens[0]]), plain(pre[lens[0]:])]
    wide = -(-pre.shape[1] // 8) * 8 + 8
    neg_a = -torch.exp(w["A_log"])

    def launch(state, rows, starts, lns, slots):
        n = rows.shape[0]
        proj = torch.full((n, wide), float("nan")).cuda()[:, :rows.shape[1]]
        proj.copy_(rows)
        seg = [s for s, m in enumerate(lns) for _ in range(m)]
        xbc, coef, y = torch.empty(n, CH).cuda(), torch.empty(n, 2 * H).cuda(), torch.empty(n, inner).cuda()
        kernels.ssd(proj, inner, inner + CH, _dev(w["conv"]), _dev(w["conv.b"]), _dev(w["dt_bias"]), _dev(neg_a), _dev(w["D"]), state, _i32(seg), _i32(starts),
                    _i32(lns), _i32(slots), xbc, coef, y, len(lns), H, G, N, V, taps)
        out = torch.empty(n, inner).cuda()
        kernels.silu_gate_norm(y, proj, 0, _dev(w["norm"]), out, groups, 1e-5)
        return y.cpu(), out.double().cpu()

    noise = r(4, kernels.ssd_state_floats(H, G, N, V, taps) + 4)          # (rows wider than needed, filled with noise)
    state = noise.clone().cuda()
    state[2].zero_(); state[0].zero_()
    n0 = 131
    y_a, first = launch(state, pre[:n0], [0], [n0], [2])
    y_b, second = launch(state, torch.cat([pre[lens[0]:], pre[n0:lens[0]]]), [0, lens[1]], [lens[1], lens[0] - n0], [0, 2])
    tol = dict(rtol=2e-4, atol=2e-4)
    assert torch.allclose(first, want[0][:n0], **tol) and torch.allclose(second[:lens[1]], want[1], **tol)
    assert torch.allclose(second[lens[1]:], want[0][n0:], **tol)
    assert torch.equal(state[1].cpu(), noise[1]) and torch.equal(state[3].cpu(), noise[3])            # other slots untouched
    fresh = torch.zeros_like(state)
    y_w, _ = launch(fresh, pre[:lens[0]], [0], [lens[0]], [3])
    assert torch.equal(y_w, torch.cat([y_a, y_b[lens[1]:]]))
    one = torch.zeros_like(state)
    ys = [launch(one, pre[t:t + 1], [0], [1], [1])[0] for t in range(20)]
    assert torch.equal(torch.cat(ys), y_w[:20])


@pytest.mark.parametrize("E,identity,groups,keep,top", [(16, 4, 2, 1, 4), (7, 0, 1, 1, 3), (10, 2, 6, 3, 6), (3, 5, 4, 4, 8), (1000, 24, 32, 4, 16), (64, 0, 64, 5, 5), (1, 0, 1, 1, 1)])
def test_choice_by_groups(E, identity, groups, keep, top):
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(E + groups)
    R, n = E + identity, 53
    z = 2.0 * torch.randn(n, R, generator=g)
    for corr in (None, 0.3 * torch.randn(R, generator=g), -3.0 + 0.3 * torch.randn(R, generator=g)):      # (the last: every choice score is negative)
        ids, wts = torch.empty(n, top, dtype=torch.int32).cuda(), torch.empty(n, top).cuda()
        kernels.route_groups(_dev(z), ids, wts, top, None if corr is None else _dev(corr), groups, keep, 1.7)
        w = {"router": torch.eye(R).double(), "correction": torch.zeros(R).double() if corr is None else corr.double()}
        chosen, weight = P.routing(z.double(), w, {"top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.7})
        s, c = P.choice_scores(z.double(), w, {"top": top, "groups": {"count": groups, "keep": keep}})
        got = ids.cpu().long()
        assert torch.equal(got.sort(dim=1).values, chosen.sort(dim=1).values)
        assert torch.allclose(wts.double().cpu(), 1.7 * torch.gather(s, 1, got), rtol=1e-5, atol=1e-8)
        assert (torch.gather(c, 1, got).diff(dim=1) <= 1e-9).all()                                         # in the order of the choice


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_plan_and_sum_with_identity_experts(dtype):
    """Pairs with an identity expert have no row in the plan and add their weight times the input."""
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(3)
    n, W, E, identity, top, align = 37, 44, 5, 3, 4, 16
    ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(n)]).to(torch.int32)
    ids[0] = torch.tensor([5, 6, 7, 5])                                   # a token of identity experts alone
    tiles = kernels.moe_max_tiles(n * top, E, align)
    row_src, pair_row, tile_group = (torch.full((m,), 99, dtype=torch.int32).cuda() for m in (tiles * align, n * top, tiles))
    kernels.moe_plan(ids.cuda(), row_src, pair_row, tile_group, E, align)
    rs, pr, tg = row_src.cpu(), pair_row.cpu(), tile_group.cpu()
    flat = ids.reshape(-1)
    for p in range(n * top):
        if flat[p] >= E:
            assert pr[p] == -1 and not (rs == p).any()
        else:
            assert rs[pr[p]] == p and tg[pr[p] // align] == flat[p]
    assert int((rs >= 0).sum()) == int((flat < E).sum())
    z, wts, h, d = torch.randn(tiles * align, W, generator=g), torch.rand(n, top, generator=g), torch.randn(n, W, generator=g).to(dtype), torch.randn(n, W, generator=g)
    out = d.clone().cuda()
    kernels.moe_combine(out, z.cuda(), wts.cuda(), pair_row, top, h.cuda())
    want = d.double()
    for t in range(n):
        for j in range(top):
            row = pr[t * top + j]
            want[t] += wts[t, j].double() * (h[t].double() if row < 0 else z[row].double())
    assert torch.allclose(out.double().cpu(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,K,D,Vd", [(4, 2, 24, 16), (8, 2, 64, 48), (3, 1, 10, 13), (2, 2, 128, 128)])
def test_values_left_and_mixed_on_their_way_to_the_cache(dtype, H, K, D, Vd):
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(D + Vd)
    n, page, hd = 9, 8, -(-max(D, Vd) // 16) * 16
    cols = (H + K) * D + K * Vd
    pos, seg = list(range(n)), torch.zeros(n, dtype=torch.int32).cuda()
    bt = _i32([[1, 0] + [-1] * 6])
    qw, kw = _dev(1.0 + 0.2 * torch.randn(D, generator=g)), _dev(1.0 + 0.2 * torch.randn(D, generator=g))
    splits = 3
    first = torch.full((n, K * Vd), float("nan"), dtype=dtype).cuda()
    shared = None
    for lam in (None, 0.3):
        rows = torch.randn(n, cols, generator=g)
        parts = torch.randn(splits, n, cols, generator=g)
        parts[-1] = rows - parts[:-1].sum(0)
        for partial in (False, True):
            cache = torch.zeros(3, 1, 2, K, page, hd, dtype=dtype).cuda()
            q_out = torch.zeros(n, H * hd, dtype=dtype).cuda()
            inp = torch.zeros(n, -(-cols // 8) * 8, dtype=dtype).cuda()[:, :cols]
            if not partial:
                inp.copy_(rows)
            elif dtype == torch.float32:
                continue                                                       # (partial sums come from the tensor cores' products)
            kernels.qk_norm_rope_store(inp, q_out, _i32(pos), seg, bt, None, qw, kw, cache.data_ptr(), cache.stride(0), cache.stride(2), H, K, D, Vd, hd, 0, 8, page,
                                       False, 1e-6, partial=_dev(parts) if partial else None, splits=splits if partial else 0, v_first=first, v_lambda=lam)
            v = rows[:, (H + K) * D:].to(dtype).double()
            tol = dict(rtol=1e-6, atol=1e-6) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
            if lam is None:
                assert torch.allclose(first.double().cpu(), v, **tol)
                shared = first.double().cpu()
            want = v if lam is None else (1 - lam) * v + lam * shared
            got = torch.stack([cache[bt[0, p // page], 0, 1, :, p % page] for p in pos]).double().cpu()
            assert torch.allclose(got[:, :, :Vd].reshape(n, K * Vd), want, **tol) and got[:, :, Vd:].abs().sum() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [1, 7, 200])
def test_square_of_relu_in_the_products_epilogue(dtype, n):
    from xyntetik_runner_b200 import kernels
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(n, 264, generator=g).to(torch.bfloat16), (torch.randn(136, 264, generator=g) / 16).to(torch.bfloat16)
    want = torch.relu(x.double() @ w.double().T) ** 2
    if dtype == "bfloat16":
        for splits in (1, 3):
            out = torch.empty(n, 136, dtype=torch.bfloat16).cuda()
            kernels.gemm_tc(x.cuda(), w.cuda(), out, None, kernels.EPI_STORE, force_splits=splits, act=kernels.ACT_RELU2)
            assert torch.allclose(out.double().cpu(), want, rtol=1e-2, atol=1e-3)
    else:
        out = torch.empty(n, 136).cuda()
        kernels.gemm_simt(_dev(x), _dev(w), out)
        kernels.act_mul(out, out, kernels.ACT_RELU2, gated=False)
        assert torch.allclose(out.double().cpu(), want, rtol=1e-4, atol=1e-5)


# ---- keys that stand out ---------------------------------------------------------------------------------------------------
def _echo_model(size, keep, dim=16, vdim=24, heads=2, scale=1.2, bias_max=40, rel=8):
    """One layer of attention in which an odd token asks for the even one below it: queries read the first half of the embedding, keys
    the second half, by the same matrix, and an odd token's first half is the second half of its even one.  The score of that pair
    is about dim * scale, all others scatter around zero."""
    cfg = ts.model(700, 64, 1e-6, [ts.layer(_a(heads, heads, dim, vdim, scale, size, keep, bias_max, rel), None)])
    t = ts.draw(cfg, 50)
    t["embed"][1::2, :32] = t["embed"][0::2, 32:]
    t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
    t["l0.mix.q"][:, 32:] = 0
    t["l0.mix.k"] = torch.cat([torch.zeros_like(t["l0.mix.q"][:, :32]), t["l0.mix.q"][:, :32]], dim=1)
    t["l0.mix.k.norm"] = t["l0.mix.q.norm"] = torch.ones_like(t["l0.mix.q.norm"])
    t["l0.mix.v"] = t["l0.mix.v"] * 3.0
    return cfg, t


def _echo_tokens(n, at, seed):
    """n tokens, the last an odd one that asks for the one at position `at`; the rest are other tokens."""
    rng = np.random.RandomState(seed)
    pair = int(rng.randint(0, 350))
    toks = [int(v) for v in rng.permutation([v for v in range(700) if v // 2 != pair])[:n]]
    toks[at], toks[-1] = 2 * pair, 2 * pair + 1
    return toks


@pytest.mark.parametrize("size,keep,n", [(24, 5, 90), (70, 17, 150), (16, 0, 60)])
def test_a_key_that_stands_out_at_every_edge(size, keep, n):
    """The asking token is the last: places just inside and just outside its window, the last kept and the first not kept, and the
    borders of pages, in a prompt, decoded alone and behind portions of two."""
    page = 16
    cfg, t = _echo_model(size, keep)
    last = n - 1
    inside, outside = last - size + 1, last - size
    places = sorted({p for p in (0, keep - 1, keep, keep + 1, page - 1, page, 2 * page - 1, 2 * page, outside - 1, outside, inside, inside + 1, last - 1)
                     if 0 <= p < last})
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = ts.make_folder(tmp, None, t, cfg)
        reqs = {f"p{at}": _echo_tokens(n, at, at) for at in places}
        ref = {rid: ts.plain_logits(cfg, t, toks) for rid, toks in reqs.items()}
        for at in places:
            # the echo matters exactly where the place is visible
            other = list(reqs[f"p{at}"])
            other[at] = next(v for v in range(0, 700, 2) if v not in other)
            moved = np.abs(ts.plain_logits(cfg, t, other)[-1] - ref[f"p{at}"][-1]).max() / np.abs(ref[f"p{at}"]).max()
            assert (moved > 0.03) == (at >= inside or at < keep), (at, moved)
        for cut, dtype in (("whole", "float32"), ("tail", "float32"), ("pairs", "float32"), ("mixed", "float32"), ("whole", "bfloat16"), ("tail", "bfloat16")):
            steps = CUTS[cut](reqs)
            res, _ = run(path, dtype, steps, page)
            got = traces.collect(steps, res, cfg["vocab"])
            for rid in reqs:
                close(got[rid], ref[rid], dtype, f"echo {rid}/{cut}/{dtype}", cfg, t, reqs[rid], ("echo", size, rid))


@pytest.mark.parametrize("dim,vdim", [(64, 64), (128, 48)])
def test_edges_on_the_tensor_cores(dim, vdim):
    """The same with heads that the tcgen05 and bulk-copy kernels take, pages of 64, a window over several tiles, kept tokens over
    more than one: a far key among hundreds."""
    size, keep, n = 150, 70, 420
    cfg, t = _echo_model(size, keep, dim=dim, vdim=vdim, scale=0.25, bias_max=100, rel=16)
    last = n - 1
    places = [0, 5, 63, 64, keep - 1, keep, last - size, last - size + 1, last - 1, 200]
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = ts.make_folder(tmp, None, t, cfg)
        reqs = {f"p{at}": _echo_tokens(n, at, at) for at in places}
        ref = {rid: ts.plain_logits(cfg, t, toks) for rid, toks in reqs.items()}
        for cut, dtype in (("whole", "bfloat16"), ("tail", "bfloat16"), ("tail", "float32")):
            steps = CUTS[cut](reqs)
            res, _ = run(path, dtype, steps, 64)
            got = traces.collect(steps, res, cfg["vocab"])
            for rid in reqs:
                close(got[rid], ref[rid], dtype, f"echo {rid}/{cut}/{dtype}", cfg, t, reqs[rid], ("echo tc", dim, rid))


def test_slow_recurrences_remember_the_first_tokens_in_a_slot_used_before():
    """Decays near one: changing the FIRST token changes the logits 200 tokens later, and the engine follows, in a slot that another
    request used before and across decoded tokens."""
    cfg = ts.CONFIGS["rec"]
    t = ts.draw(cfg, 61, slow=True)
    a = traces.random_tokens(1, 230, cfg["vocab"])
    b = [(a[0] + 1) % cfg["vocab"], (a[1] + 7) % cfg["vocab"]] + a[2:]
    ra, rb = ts.plain_logits(cfg, t, a), ts.plain_logits(cfg, t, b)
    assert np.abs(ra[-1] - rb[-1]).max() > 1e-3 * np.abs(ra).max()
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = ts.make_folder(tmp, None, t, cfg)
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
    shared = int(pick(1, 2, 3)) * (int(pick(32, 64)) if layer_sizes else int(pick(4, 12, 16)))        # value elements of the mixing layers
    layers = []
    for _ in range(rng.randint(1, 6)):
        if rng.rand() < 0.6:
            mixes = bool(rng.rand() < 0.6)
            G = int(pick(*[g for g in (1, 2, 3) if shared % g == 0 and shared // g <= 128])) if mixes else int(pick(1, 2, 3))
            Vd = shared // G if mixes else (int(pick(64, 128)) if layer_sizes else int(pick(4, 12, 16, 30)))
            H = G * int(pick(1, 2, 8 if layer_sizes else 4))
            D = int(pick(64, 128)) if layer_sizes else int(pick(6, 10, 16, 24, 34))
            rel = int(pick(4, 8, 16, 32))
            size = int(pick(1, 8, 30, 64, 65, 128, 500))
            mixer = ts.attention(H, G, D, Vd, float(pick(0.1, 0.3, D ** -0.5)), size, int(pick(0, 1, 4, 20, 64, 70)), int(rel // 2 + pick(1, 9, 60, 300)), rel, mixes)
        else:
            G = int(pick(1, 2, 3))
            H, V = G * int(pick(1, 2, 3)), int(pick(4, 8, 30))
            parts = [p for p in (1, 2, 3, 4) if (H * V) % p == 0]
            mixer = ts.mamba2(H, V, int(pick(4, 16, 33, 64)), G, int(pick(1, 2, 4, 5)), int(pick(*parts)))
        k = rng.randint(3)
        if k == 0:
            mlp = None
        elif k == 1:
            mlp = ts.dense(int(pick(24, 40, 64, 100)))
        else:
            count = int(pick(1, 2, 3, 4))
            R = count * int(pick(2, 3, 5))
            identity = int(rng.randint(0, R))
            keep = int(rng.randint(1, count + 1))
            mlp = ts.moe(R - identity, int(rng.randint(1, min(keep * R // count, 5) + 1)), int(pick(8, 24, 64)), float(pick(0.5, 1.5, 7.0)), identity,
                         (count, keep), float(pick(0.5, 1.0, 2.5)))
        layers.append(ts.layer(mixer, mlp))
    return ts.model(int(pick(61, 128, 333)), W, float(pick(1e-6, 1e-5)), layers)


@pytest.mark.parametrize("seed", range(16))
def test_drawn_configurations(seed):
    rng = np.random.RandomState(4000 + seed)
    cfg = _drawn_config(rng, layer_sizes=seed >= 10)
    t = ts.draw(cfg, 90 + seed)
    page = int(rng.choice([4, 8, 16, 64])) if seed < 10 else 64
    reqs = {f"r{i}": traces.random_tokens(11 * seed + i, n, cfg["vocab"]) for i, n in enumerate((3, 90, 17, 140, 1, 45))}
    ref = {rid: ts.plain_logits(cfg, t, toks) for rid, toks in reqs.items()}
    with tempfile.TemporaryDirectory() as tmp:
        path, _, _ = ts.make_folder(tmp, None, t, cfg)
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
            assert g.tokens == ts.plain_greedy(cfg, tensors, p, 12)
        else:
            # teacher-forced: every token is the plain argmax for the engine's own prefix, or within rounding of it
            for i, tok in enumerate(g.tokens):
                lg = ts.plain_logits(cfg, tensors, list(p) + list(g.tokens[:i]))[-1]
                assert lg.max() - lg[tok] <= 0.06 * np.abs(lg).max()


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
    want = "ids:" + ",".join(str(t) for t in ts.plain_greedy(cfg, tensors, prompt, 6))
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
