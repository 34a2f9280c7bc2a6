"""The Siditar design on the GPU against the plain implementation (tests/plain/plain_siditar.py): every mechanism
alone, then whole models replayed whole, token by token, in portions down to two tokens and mixed with other
requests on a pool so small that pages and slots are used again; generation through the scheduler.

Where random weights would hide a fault the inputs are made so that it shows: distance biases that differ by units from one
row of the table to the next, a key far back that stands out, sinks that take a good part of a row's weight, stream mixes
far from symmetric, a recurrent state carried over hundreds of steps, a slot whose earlier owner left its state."""

import json
import math
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from helpers import random_tokens
from plain import plain_siditar as plain
from siditar_tools import CONFIGS, PAGE_SIZES, clean, draw_weights, layer, left, make, model, plain_rows, right, write_folder
from trace_tools import ROOT, collect, mixed_trace, portions_trace, round64, run_trace_engine, tail_trace, whole_trace

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

# |engine - plain float64| on logits of a few units. float32: the order of sums and the device's exp, log, sin, cos (measured:
# median 2e-6 to 1e-5, worst 2.4e-5).
# bfloat16: most rows within three times the median, a few of a hundred beyond it, none beyond 1.5.
TOL_F32 = 6e-5
TOL_BF16 = {"P": 0.15, "Q": 0.12, "R": 0.15, "S": 0.1}
BF16_ROWS_BEYOND, BF16_WORST = 0.04, 1.5
LENGTHS = {"P": [70, 45, 100, 33, 2, 64, 17, 1], "Q": [130, 64, 97, 33, 210, 5], "R": [50, 33, 80, 17, 64, 9], "S": [40, 21, 66, 3]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("siditar")
    return {name: make(root / name, name) for name in CONFIGS}


def _requests(name):
    v = CONFIGS[name]["vocab"]
    return {f"{name}{i}": random_tokens(n, v, seed=37 * i + n) for i, n in enumerate(LENGTHS[name])}


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
    print(f"measured {name} {dtype} {what}: median {np.median(list(errs.values())):.3g}, worst {errs[worst]:.3g} at {worst}")
    if dtype == "float32":
        assert errs[worst] <= TOL_F32, f"worst difference {errs[worst]} at (request, position) {worst}"
        return
    beyond = sorted(k for k in errs if errs[k] > TOL_BF16[name])
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
@pytest.mark.parametrize("width, copies", [(44, 3), (33, 1), (256, 2)])
def test_the_embedding_with_sinusoidal_positions(dtype, width, copies):
    """Positions up to a hundred thousand, an odd width, a factor on the row, copies side by side; a token outside the
    vocabulary leaves zeros and sets the status."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(width)
    table = torch.randn(50, width).to(dtype)
    ids, positions = [3, 49, 0, 3, 77], [0, 1, 4097, 99999, 5]
    freq = 10000.0 ** (-2.0 * torch.arange((width + 1) // 2, dtype=torch.float64) / width)
    out = torch.full((5, copies * width), float("nan"), dtype=torch.float32, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    k.embedding_sinusoid(_d(table), _i(ids), _i(positions), _d(freq), out, status, copies, 0.7)
    assert int(status.item()) == k.STATUS_BAD_TOKEN
    got = out.cpu().double().view(5, copies, width)
    for t in range(4):
        angle = positions[t] * freq[torch.arange(width) // 2]
        ref = table[ids[t]].double() * 0.7 + torch.where(torch.arange(width) % 2 == 0, torch.sin(angle), torch.cos(angle))
        assert float((got[t] - ref).abs().max()) < 1e-6
    assert float(got[4].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [44, 64, 1000, 2048, 4104])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("parts", [None, 1, 3])
def test_streams_between_two_sublayers(dtype, width, streams, parts):
    """The streams receive a sublayer's result (none, whole, or as partial sums) and are read through a norm; both forms of
    the kernel; the gathered form that writes nothing back; the form that only moves the streams on; an RMS norm."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(width + streams)
    n, eps = 5, 3e-6
    x = torch.randn(n, streams, width) * 2.0 + 0.5
    mix, share, read = torch.randn(streams, streams), torch.randn(streams), torch.randn(streams)
    gain, bias = 1.0 + 0.2 * torch.randn(width), torch.randn(width)
    y = None if parts is None else (torch.randn(n, width).to(dtype) if parts == 1 else torch.randn(parts, n, width))
    new = x.double()
    if y is not None:
        total = y.double() if parts == 1 else y.double().sum(0)
        new = torch.einsum("st,nsw->ntw", mix.double(), new) + share.double()[None, :, None] * total[:, None, :]
    tol = 2e-5 if dtype == torch.float32 else 0.05

    def normed(u, center, b):
        v = u - u.mean(-1, keepdim=True) if center else u
        return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * gain.double() + (b.double() if b is not None else 0.0)

    args = (None if y is None else _d(y), _d(mix), _d(share))
    for center, b, r in ((True, None, read), (True, bias, None), (False, None, read)):
        s, out = _d(x.reshape(n, -1).clone()), torch.empty(n, width, dtype=dtype, device=DEV)
        k.hyper_norm(s, streams, *args, _d(r) if r is not None else None, _d(gain), _d(b) if b is not None else None, eps, center, out)
        u = (new * (r.double() if r is not None else torch.ones(streams, dtype=torch.float64))[None, :, None]).sum(1)
        assert float((out.cpu().double() - normed(u, center, b)).abs().max()) < tol * max(1.0, float(u.abs().max()) / 4)
        assert float((s.cpu().double().view(n, streams, width) - new).abs().max()) < 2e-5
    s, rows = _d(x.reshape(n, -1).clone()), [3, 0, 3]
    out = torch.empty(3, width, dtype=dtype, device=DEV)
    k.hyper_norm(s, streams, *args, None, _d(gain), None, eps, True, out, rows=_i(rows))
    assert float((out.cpu().double() - normed(new.sum(1), True, None)[rows]).abs().max()) < tol
    assert torch.equal(s.cpu(), x.reshape(n, -1))
    if y is not None:
        k.hyper_norm(s, streams, *args)
        assert float((s.cpu().double().view(n, streams, width) - new).abs().max()) < 2e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, d, dv, rot", [(6, 3, 10, 7, 0), (4, 1, 32, 16, 0), (2, 2, 64, 128, 0), (3, 3, 8, 8, 0), (2, 1, 128, 24, 0),
                                              (1, 1, 200, 40, 0), (4, 2, 16, 16, 8)])
def test_norms_of_every_head_and_queries_that_grow_warmer(dtype, H, G, d, dv, rot):
    """Every head of q and k by its own root mean square, a gain that the heads share, q times 1 + c ln(floor((p + 1) / e) +
    1) on both sides of a step, values as projected; in 16-byte pieces where sizes allow it and element by element (with a
    rotation, too); columns beyond q | k | v are left alone; pages in shuffled order."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(H * d + dv)
    page, lens, starts, eps, temp = 8, [5, 1, 9], [0, 13, 6], 3e-6, (0.6, 7)
    n, B = sum(lens), len(lens)
    cols = (H + G) * d + G * dv
    proj = (torch.randn(n, (cols + 15) // 8 * 8) * 1.5).to(dtype)
    qg, kg = 1.0 + 0.3 * torch.randn(d), 1.0 + 0.3 * torch.randn(d)
    blocks = 3
    table = torch.randperm(B * blocks + 2)[:B * blocks].view(B, blocks).to(torch.int32)
    kp = torch.zeros(B * blocks + 2, G, page, d, device=DEV, dtype=dtype)
    vp = torch.zeros(B * blocks + 2, G, page, dv, device=DEV, dtype=dtype)
    q_out = torch.empty(n, H * d, device=DEV, dtype=dtype)
    q0, sp, _, token_req = _entries(lens, starts)
    positions = [s0 + i for s0, ln in zip(starts, lens) for i in range(ln)]
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    inv = 300.0 ** (-2.0 * torch.arange(rot // 2).double() / rot) if rot else None
    k.bias_rope_kv(_d(proj), None, q_out, _d(inv.float()) if rot else None, rot, True, _i(positions), token_req, _d(table), page, kp, vp, H, G, d,
                   dv, status, q_gain=_d(qg), k_gain=_d(kg), norm_eps=eps, head_norm=True, q_temp=temp)
    assert int(status.item()) == 0
    x = proj.double()
    qn = plain.unit_rms(x[:, :H * d].view(n, H, d), eps) * qg.double()
    kn = plain.unit_rms(x[:, H * d:(H + G) * d].view(n, G, d), eps) * kg.double()
    if rot:
        ang = torch.tensor(positions).double()[:, None] * inv[None]
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        for h in (qn, kn):
            a, b = h[..., 0:rot:2].clone(), h[..., 1:rot:2].clone()
            h[..., 0:rot:2], h[..., 1:rot:2] = a * c - b * s, a * s + b * c
    factor = plain.query_temperature(max(positions) + 1, *temp)[positions]
    assert float(factor.max()) > 1.6 and float(factor.min()) == 1.0
    qn = qn * factor[:, None, None]
    tol = 2e-5 if dtype == torch.float32 else 0.03
    assert float((q_out.cpu().double().view(n, H, d) - qn).abs().max()) < tol * max(1.0, float(qn.abs().max()) / 2)
    for t in range(n):
        e, p = int(token_req[t]), positions[t]
        pg = int(table[e, p // page])
        assert float((kp[pg, :, p % page].cpu().double() - kn[t]).abs().max()) < tol * 2
        assert torch.equal(vp[pg, :, p % page].cpu(), proj[t, (H + G) * d:cols].view(G, dv))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads, dk, dv", [(4, 6, 6), (2, 32, 32), (2, 40, 70), (2, 100, 8), (1, 130, 20), (4, 16, 130), (3, 64, 128)])
@pytest.mark.parametrize("long", [False, True])
def test_the_recurrence_with_a_gated_decay_per_channel(dtype, heads, dk, dv, long):
    """Keys of 6 to 130 numbers, more value columns than a block takes, entries of 1, 2, 19 and 45 tokens, slots with and
    without an earlier state; with `long`, entries that are cut into segments beside single tokens."""
    from quantinfer_b200 import kernels as k
    from quantinfer_b200.parts import segments

    torch.manual_seed(dk + dv)
    lens, starts = ([1, 300, 2, 193, 1], [3, 0, 0, 11, 0]) if long else ([1, 19, 2, 45], [3, 0, 0, 11])
    n, B, rate, qs = sum(lens), len(lens), 1.0 / 6.0, 0.37
    q = (torch.randn(n, heads * dk + 3) * 0.7).to(dtype)
    kk = (torch.randn(n, heads * dk) * 0.7).to(dtype)
    v = (torch.randn(n, heads * dv + 1) * 0.7).to(dtype)
    z = torch.randn(n, heads * dk + 2) * 2.0
    zb = 1.0 + torch.randn(heads * dk)
    zb[0] = -30.0                # a channel that forgets almost everything at once
    state = torch.randn(B, heads * dv * dk + 4) * 0.3
    q0, sp, slots, token_req = _entries(lens, starts)
    o = torch.empty(n, heads * dv, dtype=torch.float32, device=DEV)
    st = _d(state.clone())
    S_dev = st[:, :heads * dv * dk].unflatten(1, (heads, dv, dk))
    h_q = [0] + np.cumsum(lens).tolist()
    batch = SimpleNamespace(extra={}, max_q_len=max(lens), h_q_start=h_q, q_start=q0, start_pos=sp, slot_ids=slots)
    segments.matrix_state_scan("channel_gate", _d(q)[:, 3:], _d(kk), _d(v)[:, :heads * dv], S_dev, o, batch, heads, dk, dv,
                               log_decay=_d(z)[:, :heads * dk], decay_bias=_d(zb), rate=rate, q_scale=qs)
    assert any(key[0] == "segments" for key in batch.extra) == long
    a = 0
    for e, ln in enumerate(lens):
        S = state[e, :heads * dv * dk].double().view(heads, dv, dk).transpose(1, 2).clone() if starts[e] > 0 else torch.zeros(heads, dk, dv, dtype=torch.float64)
        for t in range(a, a + ln):
            w = torch.sigmoid(z[t, :heads * dk].double() + zb.double()) ** rate
            S = w.view(heads, dk)[:, :, None] * S + kk[t].double().view(heads, dk)[:, :, None] * v[t, :heads * dv].double().view(heads, dv)[:, None, :]
            ref = torch.einsum("hkv,hk->hv", S, q[t, 3:].double().view(heads, dk) * qs).reshape(-1)
            assert float((o[t].cpu().double() - ref).abs().max()) < 1e-4 * max(1.0, float(ref.abs().max())), (e, t)
        got_S = st[e, :heads * dv * dk].cpu().double().view(heads, dv, dk).transpose(1, 2)
        assert float((got_S - S).abs().max()) < 1e-4 * max(1.0, float(S.abs().max()))
        assert torch.equal(st[e, heads * dv * dk:].cpu(), state[e, heads * dv * dk:])
        a += ln


def _attention_case(H, G, d, dv, page, lens, starts, rows, reach, seed):
    """Queries, shuffled pages, a distance bias whose rows differ by units, sinks, and the float64 result."""
    from quantinfer_b200.parts.position import distance_buckets

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
    rel, sink, scale = torch.randn(rows, H) * 2.0, torch.randn(H) + 3.5, 0.8 / math.sqrt(d)
    ref = torch.zeros(n, H, dv, dtype=torch.float64)
    a, sink_share = 0, []
    for e in range(B):
        for j in range(ctx[e]):
            kp[table[e, j // page], :, j % page] = keys[e][j]
            vp[table[e, j // page], :, j % page] = vals[e][j]
        K, V = keys[e].double().repeat_interleave(H // G, 1), vals[e].double().repeat_interleave(H // G, 1)
        bias = plain.distance_bias(rel, ctx[e], reach)
        for t in range(lens[e]):
            pos = starts[e] + t
            s = torch.einsum("jhd,hd->hj", K[:pos + 1], q[a + t].double()) * scale + bias[:, pos, :pos + 1]
            m = torch.maximum(s.max(-1).values, sink.double())
            w, tail = torch.exp(s - m[:, None]), torch.exp(sink.double() - m)
            sink_share += (tail / (w.sum(-1) + tail)).tolist()
            ref[a + t] = torch.einsum("hj,jhe->he", w / (w.sum(-1) + tail)[:, None], V[:pos + 1])
        a += lens[e]
    assert np.median(sink_share) > 0.01         # the premise: leaving the sink out changes every row
    spread = rel[torch.tensor(distance_buckets(rows, reach))].t().contiguous()
    return q, kp, vp, table, spread, sink, scale, ref, ctx


def _batch(lens, starts, ctx, decode):
    q0, sp, _, token_req = _entries(lens, starts)
    return SimpleNamespace(q_start=q0, start_pos=sp, n_requests=len(lens), token_req=token_req, all_decode=decode, n_lead_decode=1,
                           positions=_i([s0 + i for s0, ln in zip(starts, lens) for i in range(ln)]), max_kv_len=max(ctx),
                           tile_req=_i([]), tile_q0=_i([]))


@pytest.mark.parametrize("impl, dtype", [("generic", torch.float32), ("generic", torch.bfloat16), ("mma", torch.bfloat16)])
@pytest.mark.parametrize("H, G, d, dv, rows, reach", [(4, 2, 16, 24, 8, 40), (2, 1, 64, 64, 16, 128), (3, 3, 40, 8, 2, 5), (2, 2, 8, 96, 6, 200)])
def test_a_distance_bias_and_a_sink(impl, dtype, H, G, d, dv, rows, reach):
    """Distances below and beyond the table's reach and on its edges, within a key tile and over several; a decode token in
    front of two portions, one that starts inside a page; pages in shuffled order with large numbers where nothing lies."""
    from quantinfer_b200 import kernels as k

    page, lens, starts = 8, [1, 137, 20], [150, 0, 99]
    q, kp, vp, table, bias, sink, scale, ref, ctx = _attention_case(H, G, d, dv, page, lens, starts, rows, reach, H * d + rows)
    n = sum(lens)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * dv), float("nan"), dtype=dtype, device=DEV)
    k.gated_attention(_d(q.view(n, H * d).to(dtype)), out, _d(kp.to(dtype)), _d(vp.to(dtype)), _d(table), _batch(lens, starts, ctx, False), H, G, d,
                      dv, scale, 0, 0, None, status, impl=impl, sink=_d(sink), bias=_d(bias))
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, dv) - ref).abs()
    assert float(err.max()) < (1e-4 if dtype == torch.float32 else 0.04), (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


@pytest.mark.parametrize("H, G, d, dv, rows, reach, ranges", [(4, 2, 16, 24, 8, 40, 3), (2, 1, 64, 64, 16, 128, 5), (3, 3, 40, 8, 2, 5, 1), (6, 2, 128, 128, 12, 90, None),
                                                              (8, 1, 32, 40, 6, 300, 2), (2, 2, 128, 64, 4, 17, 4)])
def test_single_tokens_with_a_distance_bias(H, G, d, dv, rows, reach, ranges):
    """Steps of single tokens at contexts of 1 to 300, each token's keys in one or several ranges over separate CTAs (more
    ranges than some tokens have key tiles)."""
    from quantinfer_b200 import kernels as k

    page, lens, starts = 8, [1, 1, 1, 1, 1], [299, 0, 63, 64, 150]
    q, kp, vp, table, bias, sink, scale, ref, ctx = _attention_case(H, G, d, dv, page, lens, starts, rows, reach, H * d + rows + 1)
    n, bf = sum(lens), torch.bfloat16
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * dv), float("nan"), dtype=bf, device=DEV)
    k.gated_attention(_d(q.view(n, H * d).to(bf)), out, _d(kp.to(bf)), _d(vp.to(bf)), _d(table), _batch(lens, starts, ctx, True), H, G, d, dv, scale, 0,
                      0, None, status, impl="mma", sink=_d(sink), key_ranges=ranges, bias=_d(bias))
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, dv) - ref).abs()
    assert float(err.max()) < 0.04, (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


@pytest.mark.parametrize("H, G, page, rows, reach, ranges", [(4, 2, 16, 16, 128, 1), (2, 1, 64, 8, 40, 1), (2, 2, 8, 6, 400, 3), (3, 3, 8, 2, 5, 2)])
def test_a_distance_bias_in_the_tcgen05_attention_kernel(H, G, page, rows, reach, ranges):
    """Heads of 128: warps whose rows all lie beyond the bias's reach of a key tile, warps that read an entry a score, and
    tiles on the boundary; with one range of keys and with several."""
    from quantinfer_b200 import kernels as k

    d, bf = 128, torch.bfloat16
    lens, starts = [280, 70], [0, 145]
    q, kp, vp, table, bias, sink, scale, ref, ctx = _attention_case(H, G, d, d, page, lens, starts, rows, reach, H + rows)
    n = sum(lens)
    q0, sp, _, token_req = _entries(lens, starts)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((n, H * d), float("nan"), dtype=bf, device=DEV)
    k.attention_prefill(_d(q.view(n, H * d).to(bf)), out, _d(kp.to(bf)), _d(vp.to(bf)), _d(table), q0, sp, _i([0, 0, 0, 1]), _i([0, 128, 256, 280]),
                        H, G, d, scale, 0, status, impl="tcgen05", max_kv_len=max(ctx), key_ranges=ranges, sink=_d(sink), bias=_d(bias))
    assert int(status.item()) == 0
    err = (out.cpu().double().view(n, H, d) - ref).abs()
    assert float(err.max()) < 0.04, (float(err.max()), np.unravel_index(int(err.argmax()), err.shape))


@pytest.mark.parametrize("K", [8256, 8320, 2112, 1096])
def test_a_product_whose_contraction_does_not_divide_into_the_usual_parts(K):
    """Few tokens, K cut into parts: every part must have work (129 blocks of 64 do not divide into 16 parts of 9)."""
    from quantinfer_b200 import kernels as k

    torch.manual_seed(K)
    x, w = (torch.randn(m, K) / math.sqrt(K) for m in (8, 256))
    x, w = x.to(torch.bfloat16), w.to(torch.bfloat16)
    out = torch.empty(8, 256, dtype=torch.float32, device=DEV)
    k.gemm_bf16(_d(x), _d(w), out)
    assert float((out.cpu().double() - x.double() @ w.double().t()).abs().max()) < 1e-5


# ---------------------------------------------------------------- one mixer alone, in an engine of one layer


def _one_layer(tmp_path, entry, width, dtype, page_size=8, seed=77, eps=1e-6, max_tokens=512, streams=2, edit=None):
    from quantinfer_b200.engine import Engine

    cfg = model(16, width, streams, eps, [entry])
    w = draw_weights(cfg, seed)
    if edit is not None:
        edit(w)
    folder = write_folder(tmp_path / f"one{dtype}{seed}", cfg, w)
    eng = Engine.from_folder(folder, dtype=dtype, page_size=page_size, max_tokens=max_tokens, max_requests=4, use_graphs=False)
    return eng, clean(cfg), {k: v.double() for k, v in w.items()}


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


def _ref(x, cfg, w):
    return plain.two_branches(w, "l0.mix.", cfg["layers"][0]["mixer"], x, cfg["norm"]["eps"])


@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("rows, reach, temp, page, kv", [(8, 40, (0.4, 16), 8, 2), (16, 60, (0.9, 7), 8, 4), (2, 9, None, 16, 1), (6, 300, (0.3, 50), 8, 2)])
def test_the_two_branches_however_the_sequence_is_cut(tmp_path, cut, rows, reach, temp, page, kv):
    """Distances on every row of the table and beyond its reach; temperatures that step inside and at the cuts; a slot
    whose earlier owner left a state."""
    far, T = 31, 95
    entry = layer(left(4, kv, 10, 7, reach, temp), right(3, 5, 9, 8.0), (0.8, 1.3), rows=rows, rank=5)
    eng, cfg, w = _one_layer(tmp_path, entry, 24, "float32", page_size=page, seed=25)
    torch.manual_seed(7)
    x = torch.randn(T, 24)
    m = cfg["layers"][0]["mixer"]
    _run(eng, torch.randn(40, 24) * 3.0, [40], rid="earlier")
    ref = _ref(x.double(), cfg, w)
    got = _run(eng, x, CUTS[cut](T))
    err = (got.double() - ref).abs().max(dim=1).values
    assert float(err.max()) < 1e-4 * max(1.0, float(ref.abs().max())), (int(err.argmax()), float(err.max()))
    # the premises: another row of the table at one distance, the temperature and the state thirty positions back all show
    w2 = dict(w)
    w2["l0.mix.left.rel"] = w["l0.mix.left.rel"].clone()
    w2["l0.mix.left.rel"][-1] += 3.0
    changed = (_ref(x.double(), cfg, w2) - ref).abs().max(dim=1).values
    if T > reach:
        assert float(changed[reach + 2:].median()) > 1e-2
    x2 = x.clone()
    x2[far] += 1.0
    lin = lambda t: plain.linear_attention(w, "l0.mix.right.", m["right"], t.double(), 1e-6)
    assert float((lin(x2) - lin(x)).abs().max(dim=1).values[far + 30]) > 1e-3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_hundreds_of_positions_back(tmp_path, dtype):
    """The second position's key is what the queries look for, six hundred positions behind it: prompt portions, then single tokens
    over key ranges."""
    def edit(w):      # one direction of the input makes a long query and a long key in the same direction
        w["l0.mix.left.q"][:, 0] = w["l0.mix.left.k"][:, 0]
        w["l0.mix.left.q.norm"].fill_(3.0)
        w["l0.mix.left.k.norm"].fill_(3.0)

    entry = layer(left(4, 4, 16, 16, 100, (0.3, 64)), right(2, 16, 16, 16.0), rows=8, rank=4)
    eng, cfg, w = _one_layer(tmp_path, entry, 32, dtype, page_size=16, seed=23, max_tokens=1024, edit=edit)
    T = 600
    torch.manual_seed(8)
    x = torch.randn(T, 32)
    x[:, 0] = 0.0
    x[1, 0] = 20.0                      # the key
    x[-40:, 0] = 20.0                   # the queries
    x[-40:, 1:] *= 0.3
    xq = x.to(torch.bfloat16).double() if dtype == "bfloat16" else x.double()
    ref = _ref(xq, cfg, w)
    got = _run(eng, x, [300, 150, 110] + [1] * 40)
    tol = 1e-4 if dtype == "float32" else 0.06
    assert float((got.double() - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))
    x2 = xq.clone()
    x2[1, 0] = 0.0
    assert float((_ref(x2, cfg, w) - ref)[-40].abs().max()) > 0.05        # the premise: the first of those queries sees that key


@pytest.mark.parametrize("heads, dk, dv", [(3, 72, 8), (2, 130, 20), (4, 16, 70)])
def test_the_linear_branch_with_wide_keys_and_values(tmp_path, heads, dk, dv):
    entry = layer(left(2, 2, 8, 8, 20), right(heads, dk, dv, 5.0), rank=6)
    eng, cfg, w = _one_layer(tmp_path, entry, 32, "float32", seed=27)
    torch.manual_seed(9)
    x = torch.randn(250, 32)
    ref = _ref(x.double(), cfg, w)
    got = _run(eng, x, [13, 2, 1, 1, 200, 30, 3])
    assert float((got.double() - ref).abs().max()) < 1e-4 * max(1.0, float(ref.abs().max()))


def test_three_hundred_single_steps_in_bfloat16(tmp_path):
    """A state carried through three hundred steps of one token stays where the whole sequence in one step puts it."""
    entry = layer(left(4, 2, 16, 16, 50, (0.3, 32)), right(2, 16, 16, 16.0), rows=8, rank=8)
    eng, cfg, w = _one_layer(tmp_path, entry, 32, "bfloat16", page_size=16, seed=29, max_tokens=512)
    T = 303
    torch.manual_seed(10)
    x = torch.randn(T, 32)
    ref = _ref(x.to(torch.bfloat16).double(), cfg, w)
    got = _run(eng, x, [3] + [1] * (T - 3))
    whole = _run(eng, x, [T])
    tol = 0.08 * max(1.0, float(ref.abs().max()) / 4)
    assert float((got.double() - ref).abs().max()) < tol and float((whole.double() - ref).abs().max()) < tol
    assert float((got[-50:] - whole[-50:]).abs().max()) < tol


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff, streams", [(None, 2), (36, 3), (36, 1), (24, 6)])
def test_the_block_over_residual_streams(tmp_path, dtype, ff, streams):
    """One layer as a whole through the step function in portions; the sum of the streams after the layer against the plain
    implementation, with and without a feed-forward."""
    from quantinfer_b200.engine import StepEntry

    entry = layer(left(2, 1, 8, 8, 12, (0.4, 6)), right(2, 6, 5, 7.0), ff=ff, limit=1.1 if ff else None, rows=6)
    eng, cfg, w = _one_layer(tmp_path, entry, 24, dtype, seed=31, streams=streams)
    toks, taps, taken = random_tokens(40, 16, seed=2), [], []
    plain.forward(cfg, w, toks, taps)

    def tap(call, resid, delta):
        r = resid.clone()
        delta.apply(r)
        taken.append(r.view(r.shape[0], streams, -1).sum(1).cpu())

    eng.model.tap = tap
    eng.open("r")
    for a, b in ((0, 9), (9, 10), (10, 12), (12, 40)):
        eng.step([StepEntry("r", toks[a:b], [])])
    got = torch.cat(taken)
    assert float((got.double() - taps[0]).abs().max()) < (2e-5 if dtype == "float32" else 0.04) * max(1.0, float(taps[0].abs().max()))


def test_the_clamps_of_the_feed_forward_bite():
    """The premise of the tests of whole models: without the clamps the drawn models' feed-forwards give other numbers."""
    cfg, w = clean(CONFIGS["P"]), draw_weights(CONFIGS["P"], 61)
    torch.manual_seed(3)
    h = torch.randn(20, cfg["width"]).double()
    a = plain.feed_forward(w, "l0.mlp.", cfg["layers"][0]["mlp"]["limit"], h)
    assert float((plain.feed_forward(w, "l0.mlp.", 1e9, h) - a).abs().max(dim=1).values.min()) > 0.05


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
    """Softmax heads of 128 (prompt portions on the tcgen05 kernel, single tokens over key ranges), states of 64 x 128 whose
    prompts run in segments, pages of 64, requests of several query tiles, a looped layer."""
    cfg = model(300, 256, 2, 1e-5, [
        layer(left(4, 2, 128, 128, 90, (0.3, 50)), right(2, 64, 128, 16.0), (1.0, 0.8), 384, 2.0, rows=12, rank=16),
        layer(left(2, 2, 64, 128, 200, (0.2, 128)), right(4, 32, 64, 8.0), (0.9, 1.1), 320, 1.5, rows=16, rank=8)], loop=(1, 2, 2))
    w = draw_weights(cfg, 71)
    folder = write_folder(tmp_path / "wide", cfg, w)
    reqs = {f"w{i}": random_tokens(n, 300, seed=90 + i) for i, n in enumerate([300, 150, 70, 200, 40])}
    expect = plain_rows(clean(cfg), w, reqs)
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
    print(f"measured wide {dtype} {family}: median {np.median(errs):.3g}, worst {errs.max():.3g}")
    if dtype == "float32":
        assert errs.max() <= TOL_F32
    else:
        assert np.median(errs) < 0.12 and (errs > 0.35).mean() <= BF16_ROWS_BEYOND and errs.max() <= BF16_WORST


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


def test_every_pass_of_a_loop_has_its_own_cache_and_state(models):
    """The premise of the replays of looped models: passes that shared a state would give other logits (the plain
    implementation with the loop run once differs)."""
    _, cfg, w = models["P"]
    once = json.loads(json.dumps(cfg))
    once["loop"]["times"] = 1
    toks = random_tokens(30, cfg["vocab"], 4)
    assert float((plain.forward(cfg, w, toks) - plain.forward(once, w, toks)).abs().max(dim=1).values.min()) > 0.1
    from quantinfer_b200.engine import Engine

    eng = Engine.from_folder(models["P"][0], dtype="float32", page_size=8, max_tokens=256, max_requests=1)
    assert len(eng.model.cache_needs) == 12 and len({v.mixer_state.data_ptr() for v in eng._views[:6]}) == 6
    assert len({v.k_pages.data_ptr() for v in eng._views[:6]}) == 6


def test_a_stale_state_shows(models):
    """The premise of the replay tests: a request that takes over a slot without its state being cleared (the manager's
    zeroing switched off, and the kernels told that the sequence goes on) gives other logits, far beyond the bound."""
    from quantinfer_b200.engine import Engine, StepEntry

    folder, cfg, w = models["P"]
    eng = Engine.from_folder(folder, dtype="float32", page_size=8, max_tokens=256, max_requests=1)
    a, b = random_tokens(40, cfg["vocab"], 1), random_tokens(30, cfg["vocab"], 2)
    eng.open("a")
    eng.step([StepEntry("a", a, [])])
    eng.close("a")
    eng.open("b")
    clean_run = eng.step([StepEntry("b", b, [29])]).cpu().clone()
    eng.close("b")
    eng.open("a")
    eng.step([StepEntry("a", a, [])])
    stale = eng.cache._state_rows.clone()
    eng.close("a")
    eng.open("b")
    eng.step([StepEntry("b", b[:1], [])])
    eng.cache._state_rows.copy_(stale)             # as if the slot had not been cleared
    dirty = eng.step([StepEntry("b", b[1:], [28])]).cpu()
    assert float((dirty - clean_run).abs().max()) > 50 * TOL_F32


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(models, dtype):
    """bin/trace_run as a child process, the default page size, four slots, a mixed trace in which pages and slots are
    used again."""
    import tempfile
    from pathlib import Path

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


@pytest.mark.parametrize("name, run_ahead, graphs", [("P", True, True), ("R", False, True), ("Q", True, False), ("S", True, True)])
def test_greedy_generation_through_the_scheduler(models, name, run_ahead, graphs):
    """Three prompts of unequal length taken in portions of five tokens while earlier ones already decode, decode
    steps replayed from CUDA graphs and launched ahead of the host: the plain implementation's tokens."""
    import quantinfer_b200 as q
    from quantinfer_b200.engine import Engine

    folder, cfg, w = models[name]
    prompts = [random_tokens(n, cfg["vocab"], seed=n) for n in (13, 1, 27)]
    eng = Engine.from_folder(folder, dtype="float32", page_size=PAGE_SIZES[name], max_tokens=512, max_requests=4, use_graphs=graphs)
    model_ = q.Model.from_engine(eng, max_batch_tokens=16, chunk_size=5, run_ahead=run_ahead)
    got = model_.generate_batch(prompts, max_new_tokens=10, eos_token_id=None)
    for p, g in zip(prompts, got):
        assert g == _plain_greedy(cfg, w, p, 10), (name, len(p))
    # again on the same engine: slots and pages of the first call are used again, state must start afresh
    assert model_.generate_batch(prompts[::-1], max_new_tokens=10, eos_token_id=None) == got[::-1]
    assert model_.generate_tokens(prompts[2], max_new_tokens=10, eos_token_id=None) == got[2]


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
    """`--random-weights` draws a model of this design from its config.json alone (the table's rows and the rank are free there)."""
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(clean(CONFIGS["P"])))
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "quantinfer"), "generate", "--input", str(cfg), "--random-weights", "--tokens",
                        "1,2,3", "--max-new-tokens", "5", "--page-size", "8"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert len(json.loads([l for l in r.stdout.splitlines() if l.startswith("generated_tokens=")][0].split("=", 1)[1])) == 5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_past_pages_and_the_reach_of_the_bias(models, dtype):
    """Three tokens of prompt, then a hundred and fifty decoded one by one with given ids: distances pass the reach of every
    table, temperatures step, pages fill, the states are carried through every step."""
    folder, cfg, w = models["P"]
    toks = random_tokens(153, cfg["vocab"], seed=8)
    steps = tail_trace({"long": toks}, 150)
    got = run_trace_engine(folder, dtype, steps, 192, PAGE_SIZES["P"])
    _compare(got, plain_rows(cfg, w, {"long": toks}), "P", dtype, "long decode")


@pytest.mark.parametrize("grouped", [False, True])
@pytest.mark.parametrize("H, G, d, dv, ranges", [(8, 2, 40, 24, 1), (16, 1, 64, 128, 3), (3, 3, 128, 32, 2), (12, 1, 96, 96, 1)])
def test_both_forms_of_the_single_token_attention(grouped, H, G, d, dv, ranges):
    """Query heads of a group as the rows of one tile, or a tile a query head: window, chunk, cap, gate, factor, bias and sink at once,
    the output a block of columns of wider rows."""
    from quantinfer_b200 import kernels as k

    page, lens, starts, rows, reach, window, chunk, cap, factor = 8, [1, 1, 1, 1], [299, 0, 64, 150], 8, 50, 90, 128, 3.0, 0.7
    q, kp, vp, table, bias, sink, scale, _, ctx = _attention_case(H, G, d, dv, page, lens, starts, rows, reach, H * d)
    bf, n = torch.bfloat16, 4
    gate = torch.randn(n, H * dv).to(bf)
    wide = torch.full((n, 16 + H * dv + 8), 7.0, dtype=bf, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    k.gated_attention(_d(q.view(n, H * d).to(bf)), wide[:, 16:16 + H * dv], _d(kp.to(bf)), _d(vp.to(bf)), _d(table), _batch(lens, starts, ctx, True), H, G,
                      d, dv, scale, window, chunk, _d(gate), status, impl="mma", softcap=cap, out_scale=factor, sink=_d(sink), key_ranges=ranges,
                      bias=_d(bias), grouped_heads=grouped)
    assert int(status.item()) == 0
    assert float((wide[:, :16].float() - 7.0).abs().max()) == 0.0 and float((wide[:, 16 + H * dv:].float() - 7.0).abs().max()) == 0.0
    for t in range(n):
        pos = starts[t]
        lo = max(0, pos - window + 1, pos // chunk * chunk)
        pages = table[t][torch.arange(lo, pos + 1) // page]
        K, V = (p[pages, :, torch.arange(lo, pos + 1) % page].double().repeat_interleave(H // G, 1) for p in (kp, vp))
        s = cap * torch.tanh(torch.einsum("jhd,hd->hj", K, q[t].double()) * scale / cap)
        back = torch.clamp(pos - torch.arange(lo, pos + 1), max=bias.shape[1] - 1)
        s = s + bias.double()[:, back]
        e, tail = torch.exp(s), torch.exp(sink.double())
        a = torch.einsum("hj,jhe->he", e / (e.sum(-1) + tail)[:, None], V).reshape(-1)
        ref = a * torch.sigmoid(gate[t].double()) * factor
        err = (wide[t, 16:16 + H * dv].cpu().double() - ref).abs()
        assert float(err.max()) < 0.03, (t, float(err.max()))


@pytest.mark.parametrize("rows, width, inter", [(1, 64, 24), (40, 64, 24), (300, 128, 200), (520, 256, 512), (7, 44, 20)])
def test_the_clamped_activation_in_the_products_epilogue(rows, width, inter):
    """g sigmoid(1.702 g) (u + 1) of clamped pairs, by the tensor-core product's epilogue in its three shapes (few tokens,
    single CTAs, pairs of CTAs) and by the kernel of its own where the product cannot."""
    from quantinfer_b200.parts import Runtime
    from quantinfer_b200.parts.linear import Linear

    torch.manual_seed(rows)
    x, w = torch.randn(rows, width).to(torch.bfloat16), (torch.randn(2 * inter, width) * 2.0 / math.sqrt(width)).to(torch.bfloat16)
    lin = Linear(Runtime(torch.bfloat16, DEV), 2 * inter, width)
    lin.load(w)
    got = lin.forward_glu_clamped(_d(x), 1.3, 1.702).cpu().double()
    both = x.double() @ w.double().t()
    g, u = torch.clamp(both[:, 0::2], max=1.3), torch.clamp(both[:, 1::2], min=-1.3, max=1.3)
    assert float((g == 1.3).double().mean()) > 0.1          # the premise: the clamps bite
    assert float((got - g * torch.sigmoid(1.702 * g) * (u + 1.0)).abs().max()) < 0.03


def test_merged_projections_are_the_separate_ones(tmp_path):
    """The two branches through one product in and one product out, against each branch by itself and their weighted sum."""
    from quantinfer_b200.config import ParallelMixersSpec, config_from_dict
    from quantinfer_b200.engine import Engine
    import dataclasses

    entry = layer(left(3, 1, 10, 7, 40, (0.4, 16)), right(3, 5, 9, 8.0), (0.8, 1.3), rows=8, rank=5)
    eng, cfg, w = _one_layer(tmp_path, entry, 24, "float32", seed=33)
    spec = config_from_dict(cfg).to_model_spec()
    mixer = dataclasses.replace(spec.layers[0].mixer, merged=False)
    assert isinstance(mixer, ParallelMixersSpec) and spec.layers[0].mixer.merged
    plain_spec = dataclasses.replace(spec, layers=(dataclasses.replace(spec.layers[0], mixer=mixer),))
    other = Engine(plain_spec, {k: v.to(torch.bfloat16) for k, v in w.items()}, dtype="float32", page_size=8, max_tokens=512, max_requests=4,
                   use_graphs=False)
    torch.manual_seed(1)
    x = torch.randn(50, 24)
    a, b = _run(eng, x, [20, 2, 1, 27]), _run(other, x, [20, 2, 1, 27])
    assert eng.model.blocks[0].mixer.merged and not other.model.blocks[0].mixer.merged
    assert float((a - b).abs().max()) < 1e-5 * max(1.0, float(a.abs().max()))
