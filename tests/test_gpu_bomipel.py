"""The Bomipel design on the GPU against the plain implementation (tests/plain/plain_bomipel.py): every mechanism alone, then
whole models replayed whole, token by token, in portions down to two tokens and mixed with other requests on a pool so
small that pages and slots are used again; generation through the scheduler.

Where random weights would hide a fault the inputs are made so that it shows: one key that stands out just inside and just
outside a window and among the kept first ones, pages between them that are gone, shares of mixed values far from 0 and 1,
experts whose weight would show on the wrong side of them."""

import json
import math
import subprocess
import sys
import tempfile
from pathlib import Path
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from bomipel_tools import CONFIGS, PAGE_SIZES, attention, draw_weights, latent, layer, make, model, plain_rows, rotation, write_folder
from helpers import random_tokens
from plain import plain_bomipel as plain
from trace_tools import ROOT, collect, mixed_trace, portions_trace, round64, run_trace_engine, tail_trace, whole_trace

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

# |engine - plain float64| on logits of a few units. float32: the order of sums and the device's exp, sin, cos. bfloat16: most
# rows within a few times the median, a few of a hundred beyond it.
TOL_F32 = 6e-5
TOL_BF16 = {"P": 0.2, "Q": 0.25, "R": 0.2}
BF16_ROWS_BEYOND, BF16_WORST = 0.04, 1.0
LENGTHS = {"P": [70, 45, 100, 33, 2, 64, 17, 1], "Q": [130, 64, 97, 33, 210, 5], "R": [50, 33, 80, 17, 64, 9]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bomipel")
    return {name: make(root / name, name) for name in CONFIGS}


def _requests(name):
    v = CONFIGS[name]["vocab"]
    return {f"{name}{i}": random_tokens(n, v, seed=41 * i + n) for i, n in enumerate(LENGTHS[name])}


_expected = {}


def _expect(models, name):
    if name not in _expected:
        _, cfg, w = models[name]
        _expected[name] = plain_rows(cfg, w, _requests(name))
    return _expected[name]


def _compare(got, expect, name, dtype, what=""):
    assert set(got) == set(expect)
    errs = {k: float(np.abs(got[k].astype(np.float64) - expect[k].astype(np.float64)).max()) for k in expect}
    worst = max(errs, key=errs.get)
    beyond = [k for k in errs if errs[k] > TOL_BF16[name]]
    print(f"measured {name} {dtype} {what}: median {np.median(list(errs.values())):.3g}, worst {errs[worst]:.3g} at {worst}, {len(beyond)} of {len(errs)} beyond")
    if dtype == "float32":
        assert errs[worst] <= TOL_F32, f"worst difference {errs[worst]} at (request, position) {worst}"
        return
    assert len(beyond) <= max(1, BF16_ROWS_BEYOND * len(errs)) and errs[worst] <= BF16_WORST, (len(beyond), len(errs), errs[worst], worst)


def _d(t):
    return t.to(DEV)


def _i(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _entries(lens, starts):
    """The step arrays of entries with these lengths and first positions, each in its own slot."""
    q0 = [0] + np.cumsum(lens).tolist()
    token_req = [e for e, n in enumerate(lens) for _ in range(n)]
    return _i(q0), _i(starts), _i(list(range(len(lens)))), _i(token_req)


# ---------------------------------------------------------------- small kernels against their formulas


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, d, dv, rot", [(6, 3, 10, 7, 4), (4, 1, 32, 16, 32), (2, 2, 64, 128, 12), (3, 3, 8, 8, 0), (2, 1, 128, 24, 128), (1, 1, 200, 40, 2)])
@pytest.mark.parametrize("mixes", [False, True])
def test_rotation_in_neighbouring_pairs_and_values_mixed_with_another_layers(dtype, H, G, d, dv, rot, mixes):
    """In 16-byte pieces where sizes allow it and element by element; part, all and none of a head turned; the other layer's
    values a block of columns of wider rows; pages in shuffled order."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(H * d + dv)
    page, lens, starts, share = 8, [5, 1, 9], [0, 13, 6], 0.3
    n, B = sum(lens), len(lens)
    cols = (H + G) * d + G * dv
    proj = (torch.randn(n, (cols + 7) // 8 * 8) * 1.5).to(dtype)
    other = torch.randn(n, (16 + G * dv + 7) // 8 * 8).to(dtype)
    blocks = 3
    table = torch.randperm(B * blocks + 2)[:B * blocks].view(B, blocks).to(torch.int32)
    kp = torch.zeros(B * blocks + 2, G, page, d, device=DEV, dtype=dtype)
    vp = torch.zeros(B * blocks + 2, G, page, dv, device=DEV, dtype=dtype)
    q_out = torch.empty(n, H * d, device=DEV, dtype=dtype)
    _, _, _, token_req = _entries(lens, starts)
    positions = [s0 + i for s0, ln in zip(starts, lens) for i in range(ln)]
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    inv = plain.pair_frequencies(rot, 300.0, {"factor": 3.0, "low": 1.0, "high": 3.0, "original": 60})
    k.bias_rope_kv(_d(proj), None, q_out, _d(inv.float()) if rot else None, rot, True, _i(positions), token_req, _d(table), page, kp, vp, H, G, d,
                   dv, status, v_first=_d(other)[:, 16:16 + G * dv] if mixes else None, v_share=share)
    assert int(status.item()) == 0
    x = proj.double()
    full = torch.zeros(max(positions) + 1, H + G, d, dtype=torch.float64)
    v = x[:, (H + G) * d:cols].reshape(n, G, dv)
    if mixes:
        v = plain.mix_values(v, other[:, 16:16 + G * dv].double().view(n, G, dv), share)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    for t, p in enumerate(positions):
        full.zero_()
        full[p] = x[t, :(H + G) * d].view(H + G, d)
        turned = plain.rotate(full, rot, inv, "interleaved")[p]
        assert float((q_out[t].cpu().double().view(H, d) - turned[:H]).abs().max()) < tol
        pg = int(table[int(token_req[t]), p // page])
        assert float((kp[pg, :, p % page].cpu().double() - turned[H:]).abs().max()) < tol
        assert float((vp[pg, :, p % page].cpu().double() - v[t]).abs().max()) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Q, R, r, rot, parts", [(13, 12, 6, 4, 1), (48, 32, 16, 16, 3), (200, 64, 0, 0, 1), (24, 9, 32, 32, 5), (1, 1, 2, 2, 1)])
def test_both_latents_normalised_and_the_cache_row(dtype, Q, R, r, rot, parts):
    """A projection's rows whole or as partial sums; half-split pairs; a rotated part of no coordinates, of part and of all."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(Q + R)
    page, lens, starts, eps = 8, [5, 1, 9], [0, 13, 6], 3e-6
    n, B, width = sum(lens), len(lens), Q + R + r
    z = torch.randn(parts, n, width) if parts > 1 else torch.randn(n, width).to(dtype)
    qg, cg = 1.0 + 0.3 * torch.randn(Q), 1.0 + 0.3 * torch.randn(R)
    table = torch.randperm(B * 3 + 2)[:B * 3].view(B, 3).to(torch.int32)
    cache = torch.full((B * 3 + 2, page, R + r), 9.0, device=DEV, dtype=dtype)
    cq = torch.empty(n, Q, device=DEV, dtype=dtype)
    _, _, _, token_req = _entries(lens, starts)
    positions = [s0 + i for s0, ln in zip(starts, lens) for i in range(ln)]
    inv = plain.pair_frequencies(rot, 300.0)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    k.latent_down(_d(z), Q, _d(qg), cq, _d(cg), eps, _d(inv.float()) if rot else None, rot, _i(positions), token_req, _d(table), cache, r, R, status,
                  half_split=True)
    assert int(status.item()) == 0
    row = z.double().sum(0) if parts > 1 else z.double()
    tol = 3e-6 if dtype == torch.float32 else 0.02
    assert float((cq.cpu().double() - plain.rms_norm(row[:, :Q], qg, eps)).abs().max()) < tol
    c = plain.rms_norm(row[:, Q:Q + R], cg, eps)
    for t, p in enumerate(positions):
        got = cache[int(table[int(token_req[t]), p // page]), p % page].cpu().double()
        assert float((got[:R] - c[t]).abs().max()) < tol
        if r:
            full = torch.zeros(p + 1, 1, r, dtype=torch.float64)
            full[p, 0] = row[t, Q + R:]
            assert float((got[R:] - plain.rotate(full, rot, inv, "half")[p, 0]).abs().max()) < 4 * tol


@pytest.mark.parametrize("E, top", [(5, 3), (8, 1), (64, 6), (33, 33), (1, 1), (200, 4), (1000, 2)])
@pytest.mark.parametrize("correction, normalize, scale", [(False, False, 1.0), (True, True, 1.7), (True, False, 0.5)])
def test_a_router_with_sigmoid_scores(E, top, correction, normalize, scale):
    """Each logit's own sigmoid; weights as they are, or over their sum; a correction steers the choice alone."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(E)
    n = 50
    logits = torch.randn(n, E) * 2.0
    corr = torch.randn(E) * 0.2 if correction else None
    s = torch.sigmoid(logits.double())
    idx = torch.topk(s + (corr.double() if correction else 0.0), top, dim=-1).indices
    ref = torch.gather(s, 1, idx)
    ref = ref / (ref.sum(1, keepdim=True) + 1e-20) * scale if normalize else ref * scale
    ids, weights = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, dtype=torch.float32, device=DEV)
    k.moe_route(_d(logits), _d(corr) if correction else None, ids, weights, scale, "sigmoid", normalize)
    assert torch.equal(ids.cpu().long(), idx)
    assert float((weights.cpu().double() - ref).abs().max()) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n, E, top, width, ff", [(1, 3, 2, 24, 10), (37, 5, 3, 44, 20), (130, 4, 1, 64, 40), (70, 8, 8, 72, 36), (9, 40, 2, 16, 8)])
def test_experts_whose_weight_multiplies_their_input(dtype, n, E, top, width, ff):
    """The grouped products with activation and weight in the epilogue, the rows scaled as they are gathered, the sum of the
    experts' outputs and another sublayer's output (none, whole, partial sums); experts that get nothing."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(n + E)
    x = torch.randn(n, width).to(dtype)
    gu, down = (torch.randn(E, 2 * ff, width) * 1.5 / math.sqrt(width)).to(dtype), (torch.randn(E, width, ff) / math.sqrt(ff)).to(dtype)
    ids = torch.stack([torch.randperm(max(top, E - 1))[:top] for _ in range(n)]).to(torch.int32)
    weights = torch.rand(n, top)
    pairs = n * top
    offsets, order, place = _i([0] * (E + 1)), _i([0] * pairs), _i([0] * pairs)
    tiles = torch.empty(min(pairs, pairs // k.moe_tile_rows() + E), 3, dtype=torch.int32, device=DEV)
    k.moe_group(_d(ids), E, offsets, order, place, tiles)
    a = torch.empty(pairs, ff, dtype=dtype, device=DEV)
    k.moe_gemm(_d(x), _d(gu), a, tiles, order, top, gather=True, epilogue="silu_mul", pair_scale=_d(weights))
    flat_e, flat_t = ids.flatten().long(), torch.arange(n).repeat_interleave(top)
    scaled = weights.flatten()[:, None].double() * x.double()[flat_t]
    both = torch.einsum("pk,pnk->pn", scaled, gu.double()[flat_e])
    ref_a = plain.silu(both[:, 0::2]) * both[:, 1::2]
    o = order.cpu().long()
    tol = 2e-5 if dtype == torch.float32 else 0.06
    assert float((a.cpu().double() - ref_a[o]).abs().max()) < tol
    xs = torch.empty(pairs, width, dtype=dtype, device=DEV)
    k.moe_gather(_d(x), order, top, xs, pair_scale=_d(weights))
    assert float((xs.cpu().double() - scaled[o]).abs().max()) < (1e-6 if dtype == torch.float32 else 0.02)
    y = torch.empty(pairs, width, dtype=dtype, device=DEV)
    k.moe_gemm(a, _d(down), y, tiles, order, top, gather=False)
    total = torch.zeros(n, width, dtype=torch.float64).index_add_(0, flat_t, torch.einsum("pf,pwf->pw", ref_a, down.double()[flat_e]))
    for other in (None, torch.randn(n, width).to(dtype), torch.randn(4, n, width)):
        out = torch.empty(n, width, dtype=torch.float32, device=DEV)
        k.moe_combine(y, place, None, None, out, add=_d(other) if other is not None else None, top=top)
        want = total + (0.0 if other is None else other.double().sum(0) if other.dim() == 3 else other.double())
        assert float((out.cpu().double() - want).abs().max()) < tol * max(1.0, float(total.abs().max()))


def _attention_case(H, G, d, dv, page, lens, starts, window, keep, seed):
    """Queries, shuffled pages of which those behind the window that hold no kept key are gone, and the float64 result."""
    torch.manual_seed(seed)
    B, n = len(lens), sum(lens)
    ctx = [s + l for s, l in zip(starts, lens)]
    blocks = max(-(-c // page) for c in ctx)
    table = torch.randperm(B * blocks + 3)[:B * blocks].view(B, blocks).to(torch.int32)
    kp = torch.full((B * blocks + 3, G, page, d), 30.0)
    vp = torch.full((B * blocks + 3, G, page, dv), -30.0)
    keys = [(torch.randn(c, G, d) * 1.2).to(torch.bfloat16).float() for c in ctx]
    vals = [torch.randn(c, G, dv).to(torch.bfloat16).float() for c in ctx]
    q = (torch.randn(n, H, d) * 1.2).to(torch.bfloat16).float()
    scale = 1.0 / math.sqrt(d)
    ref = torch.zeros(n, H, dv, dtype=torch.float64)
    a, kept_share = 0, []
    for e in range(B):
        for j in range(ctx[e]):
            kp[table[e, j // page], :, j % page] = keys[e][j]
            vp[table[e, j // page], :, j % page] = vals[e][j]
        for b in range(blocks):         # what the cache manager has given back before this step
            if (b + 1) * page <= starts[e] - (window or 1 << 30) + 1 and b * page >= keep:
                kp[table[e, b]], vp[table[e, b]], table[e, b] = 30.0, -30.0, -1
        K, V = keys[e].double().repeat_interleave(H // G, 1), vals[e].double().repeat_interleave(H // G, 1)
        ok = plain.visible(ctx[e], window, keep)
        for t in range(lens[e]):
            pos = starts[e] + t
            w = torch.softmax((torch.einsum("jhd,hd->hj", K, q[a + t].double()) * scale).masked_fill(~ok[pos], -math.inf), dim=-1)
            if window and pos - window >= keep:
                kept_share += w[:, :keep].sum(-1).tolist()
            ref[a + t] = torch.einsum("hj,jhe->he", w, V)
        a += lens[e]
    if keep and kept_share:
        assert np.median(kept_share) > 0.005         # the premise: leaving the kept keys out changes most rows
    return q, kp, vp, table, scale, ref, ctx


def _batch(lens, starts, ctx, decode):
    q0, sp, _, token_req = _entries(lens, starts)
    return SimpleNamespace(q_start=q0, start_pos=sp, n_requests=len(lens), token_req=token_req, all_decode=decode, n_lead_decode=1,
                           positions=_i([s0 + i for s0, ln in zip(starts, lens) for i in range(ln)]), max_kv_len=max(ctx),
                           tile_req=_i([]), tile_q0=_i([]))


WINDOWS = [(40, 6), (40, 64), (17, 65), (64, 63), (1, 1), (9, 130), (65, 8), (300, 5), (None, 7), (33, 0)]


@pytest.mark.parametrize("impl, dtype", [("generic", torch.float32), ("generic", torch.bfloat16), ("mma", torch.bfloat16)])
@pytest.mark.parametrize("H, G, d, dv, page", [(4, 2, 16, 24, 8), (2, 1, 64, 64, 16), (3, 3, 40, 8, 10)])
@pytest.mark.parametrize("window, keep", WINDOWS)
def test_kept_first_keys_behind_a_window(impl, dtype, H, G, d, dv, page, window, keep):
    """Kept keys that end inside, at and behind a key tile, as many as the context or none; a decode token in front of two
    portions, one that starts inside a page; the pages between the kept keys and the window are gone."""
    from quantinfer_b200 import kernels as k

    lens, starts = [1, 150, 20], [270, 0, 199]
    q, kp, vp, table, scale, ref, ctx = _attention_case(H, G, d, dv, page, lens, starts, window, keep, H * d + keep)
    n = sum(lens)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * dv), float("nan"), dtype=dtype, device=DEV)
    k.gated_attention(_d(q.view(n, H * d).to(dtype)), out, _d(kp.to(dtype)), _d(vp.to(dtype)), _d(table), _batch(lens, starts, ctx, False), H, G, d,
                      dv, scale, window or 0, 0, None, status, impl=impl, keep_first=keep)
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, dv) - ref).abs()
    assert float(err.max()) < (1e-4 if dtype == torch.float32 else 0.04), (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


@pytest.mark.parametrize("grouped", [False, True])
@pytest.mark.parametrize("H, G, d, dv, ranges", [(4, 2, 16, 24, 3), (6, 2, 128, 128, None), (8, 1, 32, 40, 1), (2, 2, 128, 64, 4)])
@pytest.mark.parametrize("window, keep", WINDOWS)
def test_single_tokens_with_kept_first_keys(grouped, H, G, d, dv, ranges, window, keep):
    """Contexts of 1 to 300 in one or several ranges of keys over separate CTAs, more of them than some tokens have key tiles."""
    from quantinfer_b200 import kernels as k

    page, lens, starts, bf = 8, [1] * 6, [299, 0, 63, 64, 150, 45], torch.bfloat16
    q, kp, vp, table, scale, ref, ctx = _attention_case(H, G, d, dv, page, lens, starts, window, keep, H * d + keep + 1)
    n = sum(lens)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * dv), float("nan"), dtype=bf, device=DEV)
    k.gated_attention(_d(q.view(n, H * d).to(bf)), out, _d(kp.to(bf)), _d(vp.to(bf)), _d(table), _batch(lens, starts, ctx, True), H, G, d, dv, scale,
                      window or 0, 0, None, status, impl="mma", key_ranges=ranges, grouped_heads=grouped, keep_first=keep)
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, dv) - ref).abs()
    assert float(err.max()) < 0.04, (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


@pytest.mark.parametrize("H, G, page, ranges", [(4, 2, 16, 1), (2, 1, 64, 1), (2, 2, 8, 3), (3, 3, 8, 2)])
@pytest.mark.parametrize("window, keep", WINDOWS)
def test_kept_first_keys_in_the_tcgen05_attention_kernel(H, G, page, ranges, window, keep):
    """Heads of 128; the kept keys' tiles before the window's, in one range of keys and in several (a range may hold tiles of both
    kinds, or of one); tiles in which the window begins behind kept keys."""
    from quantinfer_b200 import kernels as k

    d, bf = 128, torch.bfloat16
    lens, starts = [280, 70], [0, 345]
    q, kp, vp, table, scale, ref, ctx = _attention_case(H, G, d, d, page, lens, starts, window, keep, H + keep)
    n = sum(lens)
    q0, sp, _, _ = _entries(lens, starts)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * d), float("nan"), dtype=bf, device=DEV)
    k.attention_prefill(_d(q.view(n, H * d).to(bf)), out, _d(kp.to(bf)), _d(vp.to(bf)), _d(table), q0, sp, _i([0, 0, 0, 1]), _i([0, 128, 256, 280]),
                        H, G, d, scale, window or 0, status, impl="tcgen05", max_kv_len=max(ctx), key_ranges=ranges, keep_first=keep)
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, d) - ref).abs()
    assert float(err.max()) < 0.04, (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


# ---------------------------------------------------------------- one sublayer alone, in an engine of one layer


def _one_layer(tmp_path, entry, width, dtype, page_size=8, seed=77, eps=1e-6, max_tokens=512, edit=None):
    from quantinfer_b200.engine import Engine

    cfg = model(16, width, eps, [entry])
    w = draw_weights(cfg, seed)
    if edit is not None:
        edit(w)
    folder = write_folder(tmp_path / f"one{dtype}{seed}", cfg, w)
    eng = Engine.from_folder(folder, dtype=dtype, page_size=page_size, max_tokens=max_tokens, max_requests=4, use_graphs=False)
    return eng, cfg, w


def _run(eng, inputs, cuts, rid="r"):
    """Feeds `inputs` [T, width] through the layer's mixer in portions `cuts` for one request."""
    from quantinfer_b200.engine import StepEntry

    eng.open(rid)
    outs, a = [], 0
    mixer = eng.model.blocks[0].mixer
    for n in cuts:
        eng.cache.prepare(rid, n)
        batch = eng.make_batch([StepEntry(rid, [0] * n, [])])
        y = mixer.forward(inputs[a:a + n].to(DEV, eng.dtype).contiguous(), batch, eng._views[0]).float()
        if y.dim() == 3:            # the partial sums of a projection cut along K
            y = y.sum(dim=0)
        outs.append(y.cpu())
        eng.raise_on_status()
        eng.cache.commit(rid)
        eng.cache.check_invariants()
        a += n
    eng.close(rid)
    return torch.cat(outs)


def _portions(T, sizes):
    out, i = [], 0
    while sum(out) < T:
        out.append(min(sizes[i % len(sizes)], T - sum(out)))
        i += 1
    return out


CUTS = {
    "whole": lambda T: [T],
    "one by one": lambda T: [1] * T,
    "portions": lambda T: _portions(T, (7, 2, 16, 3, 2, 31, 5)),
    "prompt then decode": lambda T: [T - 20] + [1] * 20,
}


def _loud(H, G, d, col):
    """Makes input coordinate 0 a long query and a long key in coordinate `col` of every head (one that no rotation turns)."""
    def edit(w):
        for name, heads in (("q", H), ("k", G)):
            t = w[f"l0.mix.{name}"].clone()
            t[:, 0] = 0.0
            t[col::d] = 0.0
            t[col::d, 0] = 1.0
            w[f"l0.mix.{name}"] = t
    return edit


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, keep, page", [(9, 3, 8), (24, 8, 8), (10, 17, 16), (16, 1, 16)])
def test_which_queries_see_a_loud_key(tmp_path, cut, dtype, window, keep, page):
    """One key far louder than the rest at the first position, at the last kept one, at the first that is not kept, at a
    page's last and first place: the engine agrees with the plain rule, whose rows change exactly where the rule lets that
    key in: behind the kept ones in `window` rows, else in every later row."""
    H, G, d, W, T = 4, 2, 12, 24, 75
    entry = layer(attention(H, G, d, 7, rotation(8), (window, keep), True))
    eng, cfg, w = _one_layer(tmp_path, entry, W, dtype, page_size=page, seed=25, edit=_loud(H, G, d, d - 1))
    m = cfg["layers"][0]["mixer"]
    torch.manual_seed(7)
    base = torch.randn(T, W)
    base[:, 0] = 1.0                    # every query asks for it
    exact = lambda t: plain.attention(t.to(torch.bfloat16).double() if dtype == "bfloat16" else t.double(), m, w, "l0.mix.")[0]
    quiet = exact(base)
    for far in sorted({0, keep - 1, keep, page - 1, page, 30}):
        x = base.clone()
        x[far, 0] = 40.0
        ref = exact(x)
        changed = (ref - quiet).abs().max(dim=1).values > 1e-9
        sees = torch.tensor([i >= far and (i - far < window or far < keep) for i in range(T)])
        assert torch.equal(changed, sees)
        got = _run(eng, x, CUTS[cut](T))
        err = (got.double() - ref).abs().max(dim=1).values
        tol = 1e-4 if dtype == "float32" else 0.05
        assert float(err.max()) < tol * max(1.0, float(ref.abs().max())), (far, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("heads, dim, rot_dim, vdim, q_rank, kv_rank, dims, bands, page", [
    (3, 10, 6, 7, 13, 12, 6, None, 8), (2, 16, 16, 24, 40, 64, 16, (4.0, 1.0, 2.0, 40), 16), (1, 8, 4, 8, 5, 9, 2, None, 8), (4, 8, 0, 16, 16, 24, 0, None, 8)])
def test_the_latent_mixer_however_the_sequence_is_cut(tmp_path, cut, heads, dim, rot_dim, vdim, q_rank, kv_rank, dims, bands, page):
    rot = rotation(dims, 50.0, bands) if dims else None
    entry = layer(latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, rot))
    eng, cfg, w = _one_layer(tmp_path, entry, 24, "float32", page_size=page, seed=26)
    torch.manual_seed(8)
    x = torch.randn(95, 24)
    ref = plain.latent_attention(x.double(), cfg["layers"][0]["mixer"], w, "l0.mix.", 1e-6)
    got = _run(eng, x, CUTS[cut](95))
    err = (got.double() - ref).abs().max(dim=1).values
    assert float(err.max()) < 1e-4 * max(1.0, float(ref.abs().max())), (int(err.argmax()), float(err.max()))
    # the premises: the first position still weighs in the last row; the norm of the query latent shows
    x2 = x.clone()
    x2[0] *= -1.0
    assert float((plain.latent_attention(x2.double(), cfg["layers"][0]["mixer"], w, "l0.mix.", 1e-6) - ref)[-1].abs().max()) > 1e-5
    w2 = dict(w, **{"l0.mix.dq.norm": w["l0.mix.dq.norm"] * 1.5})
    assert float((plain.latent_attention(x.double(), cfg["layers"][0]["mixer"], w2, "l0.mix.", 1e-6) - ref).abs().max()) > 1e-2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_latent_row_hundreds_of_positions_back(tmp_path, dtype):
    """What the last queries look for lies six hundred positions behind them: prompt portions, then single tokens over key
    ranges (a latent of 32 with a rotated part of 16: the tensor-core kernel in bfloat16)."""
    def edit(w):      # input coordinate 0 fills one coordinate of the latent, and of every query's plain part
        for name, row in (("dkv", 0), ("dq", 0)):
            t = w["l0.mix." + name].clone()
            t[:, 0] = 0.0
            t[row] = 0.0
            t[row, 0] = 1.0
            w["l0.mix." + name] = t
        uq, uk = w["l0.mix.uq"].clone(), w["l0.mix.uk"].clone()
        uq[:, 0], uk[:, 0] = 0.0, 0.0
        uq[0::32, 0] = 3.0
        uk[0::16, 0] = 3.0
        w["l0.mix.uq"], w["l0.mix.uk"] = uq, uk
        w["l0.mix.uv"] = w["l0.mix.uv"] * 4.0
        w["l0.mix.uv"][:, 0] = 0.0          # (all loud rows have that coordinate in common)

    entry = layer(latent(2, 16, 16, 16, 24, 32, rotation(16, 1000.0)))
    eng, cfg, w = _one_layer(tmp_path, entry, 32, dtype, page_size=16, seed=23, max_tokens=1024, edit=edit)
    T, m = 600, cfg["layers"][0]["mixer"]
    torch.manual_seed(9)
    x = torch.randn(T, 32)
    x[:, 0] = 0.0
    x[1, 0] = 20.0                      # what is looked for
    x[-40:, 0] = 20.0                   # the queries
    xq = x.to(torch.bfloat16).double() if dtype == "bfloat16" else x.double()
    ref = plain.latent_attention(xq, m, w, "l0.mix.", 1e-6)
    got = _run(eng, x, [300, 150, 110] + [1] * 40)
    tol = 1e-4 if dtype == "float32" else 0.06
    assert float((got.double() - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))
    x2 = xq.clone()
    x2[1, 0] = 0.0
    assert float((plain.latent_attention(x2, m, w, "l0.mix.", 1e-6) - ref)[-40].abs().max()) > 0.05


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts, top, ff", [(5, 2, 20), (8, 1, 32), (3, 3, 12), (1, 1, 8), (40, 6, 16)])
def test_the_mixture_alone_and_a_token_in_any_company(tmp_path, dtype, experts, top, ff):
    """Against the plain rule (rows whose choice is close left aside in bfloat16); a token alone gives the row it gives among
    fifty, bit for bit."""
    entry = layer(attention(2, 1, 8, 8), (experts, top, ff))
    eng, cfg, w = _one_layer(tmp_path, entry, 32, dtype, seed=31)
    torch.manual_seed(5)
    x = torch.randn(50, 32).to(torch.bfloat16)
    ffn = eng.model.blocks[0].ffn
    xd = _d(x.to(eng.dtype))
    other = torch.randn(50, 32)
    got, added = ffn.forward(xd).float().cpu(), ffn.forward_add(xd, _d(other)).cpu()
    h = x.double()
    ref = plain.mixture(h, cfg["layers"][0]["mlp"], w, "l0.mlp.")
    tol = (2e-5 if dtype == "float32" else 0.05) * max(1.0, float(ref.abs().max()))
    assert float((got.double() - ref).abs().max()) < tol and float((added.double() - ref - other.double()).abs().max()) < tol
    for t in (0, 17, 49):
        assert torch.equal(ffn.forward(xd[t:t + 1].contiguous()).float().cpu()[0], got[t])
    # the premise: the weight on the output, and renormalised weights, are other numbers
    scores, chosen = plain.route(h, w["l0.mlp.router"], top)
    wrong = torch.stack([sum(s * plain.expert(h[t], w, f"l0.mlp.e{int(e)}.") for s, e in zip(scores[t], chosen[t])) for t in range(50)])
    assert float((wrong - ref).abs().max(dim=1).values.median()) > 0.1


def test_a_step_of_many_tokens_runs_the_experts_one_by_one(tmp_path, monkeypatch):
    """From 128 rows an expert on a prompt step gathers scaled rows and takes each expert through the tcgen05 product; the
    grouped kernels give the same within bfloat16."""
    entry = layer(attention(2, 1, 8, 8), (4, 2, 64))
    eng, cfg, w = _one_layer(tmp_path, entry, 64, "bfloat16", seed=33)
    torch.manual_seed(6)
    x = torch.randn(400, 64).to(torch.bfloat16)
    ffn = eng.model.blocks[0].ffn
    assert ffn._by_expert(_d(x), 800)
    many = ffn.forward(_d(x)).float().cpu()
    monkeypatch.setattr(type(ffn), "ROWS_AN_EXPERT", 10 ** 9)
    grouped = ffn.forward(_d(x)).float().cpu()
    ref = plain.mixture(x.double(), cfg["layers"][0]["mlp"], w, "l0.mlp.")
    tol = 0.05 * max(1.0, float(ref.abs().max()) / 4)
    assert float((many.double() - ref).abs().max()) < tol and float((grouped.double() - ref).abs().max()) < tol
    eng.raise_on_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("moe", [None, (3, 2, 20)])
@pytest.mark.parametrize("mixer", [attention(2, 1, 8, 8, rotation(8), (5, 2), True), latent(2, 8, 4, 8, 12, 16, rotation(4))])
def test_one_norm_and_both_sublayers_side_by_side(tmp_path, dtype, moe, mixer):
    """One layer as a whole through the step function in portions; the stream after the layer against the plain one, with and
    without a feed-forward."""
    from quantinfer_b200.engine import StepEntry

    eng, cfg, w = _one_layer(tmp_path, layer(mixer, moe), 24, dtype, seed=35)
    toks, taken = random_tokens(40, 16, seed=2), []
    _, kept = plain.forward(cfg, w, toks, keep_layers=True)
    eng.model.tap = lambda call, resid, delta: taken.append((resid + (delta.float().sum(0) if delta.dim() == 3 else delta.float())).cpu())
    eng.open("r")
    for a, b in ((0, 9), (9, 10), (10, 12), (12, 40)):
        eng.step([StepEntry("r", toks[a:b], [])])
    got = torch.cat(taken)
    assert float((got.double() - kept[0]).abs().max()) < (2e-5 if dtype == "float32" else 0.05) * max(1.0, float(kept.abs().max()))


# ---------------------------------------------------------------- whole models, replayed


def _family(name, reqs, family):
    longest = round64(max(LENGTHS[name]))
    if family == "whole":
        return whole_trace(reqs), longest
    if family == "tail":
        return tail_trace(reqs, 48), longest
    if family == "portions":
        return portions_trace(reqs), longest
    steps, peak = mixed_trace(reqs, seed=5, max_live=4, max_tokens=longest + 2 * 64)
    assert sum(round64(n) for n in LENGTHS[name]) > peak and max(len(s["entries"]) for s in steps) >= 3
    return steps, peak


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("family", ["whole", "tail", "portions", "mixed"])
def test_replay_family(models, name, dtype, family):
    folder, cfg, w = models[name]
    steps, max_tokens = _family(name, _requests(name), family)
    got = run_trace_engine(folder, dtype, steps, max_tokens, PAGE_SIZES[name])
    _compare(got, _expect(models, name), name, dtype, family)


@pytest.mark.parametrize("dtype, family", [("bfloat16", "whole"), ("bfloat16", "mixed"), ("bfloat16", "tail"), ("float32", "portions")])
def test_sizes_of_the_tensor_core_kernels(tmp_path, dtype, family):
    """Heads of 128 (prompt portions on the tcgen05 kernel, single tokens over key ranges) behind a window with kept keys, a
    latent of 256 with a rotated part of 64, prompts whose experts run one by one, pages of 64, requests of several query tiles."""
    rot = rotation(128, 10000.0, (8.0, 1.0, 4.0, 256))
    cfg = model(300, 256, 1e-5, [
        layer(attention(4, 2, 128, 128, rot, (90, 70), True), (2, 1, 128)),
        layer(latent(4, 64, 64, 64, 96, 256, rotation(64)), (4, 2, 72)),
        layer(attention(2, 2, 128, 128, rotation(64), (64, 4), True), (3, 2, 64))], 12.0)
    w = draw_weights(cfg, 91)
    folder = write_folder(tmp_path / "wide", cfg, w)
    reqs = {f"w{i}": random_tokens(n, 300, seed=90 + i) for i, n in enumerate([300, 150, 70, 200, 40])}
    expect = plain_rows(cfg, w, reqs)
    if family == "whole":
        steps, max_tokens = whole_trace(reqs), 320
    elif family == "tail":
        steps, max_tokens = tail_trace(reqs, 30), 320
    elif family == "portions":
        steps, max_tokens = portions_trace(reqs, sizes=(70, 2, 130, 3, 64, 1)), 320
    else:
        steps, max_tokens = mixed_trace(reqs, seed=4, max_live=4, max_tokens=320 + 256, sizes=(2, 30, 64, 129, 17), decode_tail=12)
    got = run_trace_engine(folder, dtype, steps, max_tokens, 64)
    errs = np.array([float(np.abs(got[k].astype(np.float64) - expect[k].astype(np.float64)).max()) for k in expect])
    print(f"measured wide {dtype} {family}: median {np.median(errs):.3g}, worst {errs.max():.3g}, beyond 0.25 {(errs > 0.25).mean():.3g}")
    if dtype == "float32":
        assert errs.max() <= TOL_F32
    else:
        assert np.median(errs) < 0.12 and (errs > 0.25).mean() <= BF16_ROWS_BEYOND and errs.max() <= BF16_WORST


def test_the_cuts_agree_with_one_another_in_float32(models):
    """What a position's logits are must not depend on how its prompt was cut or on its company in the batch."""
    folder, cfg, w = models["P"]
    reqs = _requests("P")
    runs = []
    for family in ("whole", "tail", "portions", "mixed"):
        steps, max_tokens = _family("P", reqs, family)
        runs.append(run_trace_engine(folder, "float32", steps, max_tokens, PAGE_SIZES["P"]))
    for other in runs[1:]:
        worst = max(float(np.abs(other[k] - runs[0][k]).max()) for k in runs[0])
        assert worst <= 3e-5, worst


def test_what_the_replays_would_miss_if_it_did_not_show(models):
    """The premises: kept keys left out, values not mixed, mixed with the layer before instead of the first, bands left out, the
    cap left out, each moves the plain logits of the drawn models far beyond the bound."""
    _, cfg, w = models["P"]
    toks = random_tokens(60, cfg["vocab"], 4)
    ref = plain.forward(cfg, w, toks)

    def moved(edit, weights=w):
        d = json.loads(json.dumps(cfg))
        edit(d)
        return float((plain.forward(d, weights, toks) - ref).abs().max(dim=1).values[30:].median())

    def no_keep(d):
        for e in d["layers"]:
            if "mask" in e["mixer"]:
                e["mixer"]["mask"]["keep_first"] = 0

    def no_mix(d):
        for e in d["layers"]:
            e["mixer"].pop("v_mix", None)

    assert moved(no_keep) > 0.05 and moved(no_mix) > 0.05
    assert moved(lambda d: d["layers"][1]["mixer"].update(v_mix=False)) > 0.05          # layer 4 would be the first
    assert moved(lambda d: d["layers"][1]["mixer"]["rot"].pop("scaling")) > 0.01
    assert moved(lambda d: d.pop("logit_softcap")) > 0.05
    wide = lambda d: d["layers"][1]["mixer"]["mask"].update(size=10)
    assert moved(wide) > 0.01


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(models, dtype):
    """bin/trace_run as a child process, the default page size, four slots, a mixed trace in which pages and slots are
    used again."""
    folder, cfg, w = models["Q"]
    reqs = _requests("Q")
    steps, peak = mixed_trace(reqs, seed=9, max_live=4, max_tokens=round64(max(LENGTHS["Q"])) + 128)
    with tempfile.TemporaryDirectory() as out:
        cmd = [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", out,
               "--max-tokens", str(peak)]
        r = subprocess.run(cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-3000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
        outputs = {}
        for s in steps:
            wanted = sum(len(e["want"]) for e in s["entries"])
            if wanted:
                outputs[s["step"]] = np.fromfile(Path(out) / f"{s['step']}.f32", dtype="<f4").reshape(wanted, cfg["vocab"])
    _compare(collect(steps, outputs), _expect(models, "Q"), "Q", dtype, "trace_run")


# ---------------------------------------------------------------- generation through the scheduler


def _plain_greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(plain.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name, run_ahead, graphs", [("P", True, True), ("R", False, True), ("Q", True, False), ("Q", True, True)])
def test_greedy_generation_through_the_scheduler(models, name, run_ahead, graphs):
    """Three prompts of unequal length taken in portions of five tokens while earlier ones already decode, decode steps
    replayed from CUDA graphs and launched ahead of the host: the plain implementation's tokens."""
    import quantinfer_b200 as q
    from quantinfer_b200.engine import Engine

    folder, cfg, w = models[name]
    prompts = [random_tokens(n, cfg["vocab"], seed=n) for n in (13, 1, 27)]
    eng = Engine.from_folder(folder, dtype="float32", page_size=PAGE_SIZES[name], max_tokens=512, max_requests=4, use_graphs=graphs)
    model_ = q.Model.from_engine(eng, max_batch_tokens=16, chunk_size=5, run_ahead=run_ahead)
    got = model_.generate_batch(prompts, max_new_tokens=12, eos_token_id=None)
    for p, g in zip(prompts, got):
        assert g == _plain_greedy(cfg, w, p, 12), (name, len(p))
    # again on the same engine: slots and pages of the first call are used again
    assert model_.generate_batch(prompts[::-1], max_new_tokens=12, eos_token_id=None) == got[::-1]
    assert model_.generate_tokens(prompts[2], max_new_tokens=12, eos_token_id=None) == got[2]


def test_command_line_generates_the_same_tokens(models):
    folder, cfg, w = models["R"]
    prompt = random_tokens(9, cfg["vocab"], seed=1)
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "quantinfer"), "generate", "--input", str(folder), "--tokens",
                        ",".join(map(str, prompt)), "--max-new-tokens", "10", "--dtype", "float32", "--page-size", "8"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    line = [l for l in r.stdout.splitlines() if l.startswith("generated_tokens=")][0]
    assert json.loads(line.split("=", 1)[1]) == _plain_greedy(cfg, w, prompt, 10)


def test_random_weights_from_the_command_line(tmp_path):
    """`--random-weights` draws a model of this design from its config.json alone."""
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(CONFIGS["P"]))
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "quantinfer"), "generate", "--input", str(cfg), "--random-weights", "--tokens",
                        "1,2,3", "--max-new-tokens", "5", "--page-size", "8"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert len(json.loads([l for l in r.stdout.splitlines() if l.startswith("generated_tokens=")][0].split("=", 1)[1])) == 5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_past_windows_and_pages(models, dtype):
    """Three tokens of prompt, then a hundred and fifty decoded one by one with given ids: every window passes over decoded
    tokens while the first ones stay, pages in between go back."""
    folder, cfg, w = models["P"]
    toks = random_tokens(153, cfg["vocab"], seed=8)
    seen = []

    def look(eng):
        g = next(g for g in eng.cache.groups if getattr(g.need, "keep_first", 0) == 3)
        seen.append(g.allocator.num_pages - g.allocator.free_pages)

    got = run_trace_engine(folder, dtype, tail_trace({"long": toks}, 150), 192, PAGE_SIZES["P"], after_step=look)
    assert max(seen) <= 5          # one kept page, two or three of the window, and never the whole sequence's twenty
    _compare(got, plain_rows(cfg, w, {"long": toks}), "P", dtype, "long decode")
