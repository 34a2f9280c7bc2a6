"""Shared by the Bomipel tests: small configurations that differ from one another in every size and option, weights drawn so
that activations are of order one (attention far from uniform, router scores spread over (0, 1), shares of mixed values away
from 0 and 1, logits that reach their cap), model folders, and the plain implementation's logits.

No choice of experts is close: the first CODE coordinates of the stream hold a code of the token that no sublayer writes to and
that alone the routers read, and a token's code is drawn until every router's last chosen and first unchosen expert lie well
apart. So bfloat16 takes the experts that float64 takes, and differences are those of the arithmetic."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch


def rotation(dims, base=300.0, bands=None):
    r = {"base": base, "dims": dims}
    if bands is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    return r


def attention(heads, kv_heads, dim, vdim, rot=None, mask=None, v_mix=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 / math.sqrt(dim)}
    if rot is not None:
        m["rot"] = rot
    if mask is not None:
        m["mask"] = dict(zip(("size", "keep_first"), mask))
    if v_mix is not None:
        m["v_mix"] = v_mix
    return m


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, rot=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": scale if scale is not None else 1.5 / math.sqrt(dim + rot_dim)}
    if rot is not None:
        m["rot"] = rot
    return m


def layer(mixer, moe=None):
    """`moe`: (experts, top, ff) or None."""
    return {"type": "latent_attention" if "kv_rank" in mixer else "attention", "mixer": mixer,
            "mlp": {"kind": "moe", "router": {"experts": moe[0], "top": moe[1]}, "expert": {"ff": moe[2]}} if moe is not None else None}


def model(vocab, width, eps, layers, cap=None):
    cfg = {"architecture": "Bomipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


CONFIGS = {
    # no size a power of two or a multiple of eight; three kv heads; kept keys that end inside the first page, behind it
    # and none; a window longer than most requests; a layer that mixes nothing between layers that do; a layer without
    # feed-forward; values narrower and wider than keys
    "P": model(131, 44, 3e-6, [
        layer(latent(3, 10, 6, 7, 13, 12, rotation(6)), (5, 2, 20)),
        layer(attention(6, 3, 10, 7, rotation(4, bands=(3.0, 1.0, 3.0, 60)), (9, 3), True), (3, 1, 28)),
        layer(attention(2, 2, 6, 11, rotation(6, 50.0), (13, 11), False)),
        layer(latent(2, 6, 4, 9, 10, 20, rotation(4, 900.0)), (7, 3, 12)),
        layer(attention(3, 3, 14, 7, rotation(2), (17, 0), True), (4, 4, 20)),
        layer(attention(3, 3, 6, 7, None, (70, 2), True), (5, 1, 36))], 9.0),
    # multiples of 16 (the tensor-core kernels' sizes); one kv head; whole heads turned; windows of one page and of three;
    # kept keys of a page and a bit; no cap
    "Q": model(200, 64, 1e-5, [
        layer(attention(4, 1, 32, 16, rotation(32, 10000.0, (8.0, 1.0, 4.0, 128)), (16, 20), True), (8, 1, 32)),
        layer(latent(4, 32, 16, 32, 48, 32, rotation(16, 10000.0)), (4, 2, 64)),
        layer(attention(2, 1, 64, 16, rotation(16, 5000.0, (2.0, 2.0, 2.0, 64)), (48, 4), True), (6, 2, 16)),
        layer(latent(2, 16, 16, 64, 16, 64, rotation(16, 1000.0)), (8, 3, 32))]),
    # a rotated part of 32 of which all turns in bands; no rotation at all; every earlier key; a window of one; one expert
    "R": model(97, 48, 1e-6, [
        layer(latent(2, 16, 32, 24, 24, 64, rotation(32, 1000.0, (4.0, 1.0, 2.0, 100))), (3, 3, 40)),
        layer(attention(4, 2, 64, 64, None, None, None), (2, 1, 24)),
        layer(latent(1, 8, 0, 8, 7, 9), (1, 1, 16)),
        layer(attention(2, 2, 16, 40, rotation(16), (1, 1), True), (6, 5, 8))], 30.0),
}
CODE, APART = 6, 0.12
PAGE_SIZES = {"P": 8, "Q": 16, "R": 8}
SEEDS = {"P": 81, "Q": 82, "R": 83}


def draw_weights(cfg: dict, seed: int, dtype=torch.bfloat16) -> dict:
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(out, inp, gain=1.0):
        return (torch.randn(out, inp, generator=g) * gain / math.sqrt(inp)).to(dtype)

    def vec(n, std, mean=0.0):
        return (mean + std * torch.randn(n, generator=g)).to(dtype)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(dtype), "final.norm": (vec(W, 0.2, 1.0).float() * 3.0 / math.sqrt(W)).to(dtype)}
    for i, entry in enumerate(cfg["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        q = p + "mix."
        w[p + "norm1"] = vec(W, 0.2, 1.0)
        if entry["type"] == "latent_attention":
            H, d, r, e, Q, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(Q, W, 1.5), vec(Q, 0.2, 1.0), mat(H * (d + r), Q, 1.5)
            w[q + "dkv"], w[q + "dkv.norm"] = mat(R + r, W, 1.5), vec(R, 0.2, 1.0)
            w[q + "uk"], w[q + "uv"] = mat(H * d, R, 1.2), mat(H * e, R, 1.5)
        else:
            H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w[q + "q"], w[q + "k"], w[q + "v"] = mat(H * d, W, 1.2), mat(G * d, W, 1.2), mat(G * e, W, 1.5)
            if m.get("v_mix"):
                w[q + "vmix"] = (0.25 + 0.5 * torch.rand((), generator=g)).to(dtype)
        w[q + "o"] = mat(W, H * e)
        w[q + "o"][:CODE] = 0.0
        if entry["mlp"] is not None:
            E, ff = entry["mlp"]["router"]["experts"], entry["mlp"]["expert"]["ff"]
            w[p + "mlp.router"] = mat(E, W, 1.5 * math.sqrt(W / CODE))
            w[p + "mlp.router"][:, CODE:] = 0.0
            for k in range(E):
                w[f"{p}mlp.e{k}.gate"], w[f"{p}mlp.e{k}.up"], w[f"{p}mlp.e{k}.down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), mat(W, ff)
                w[f"{p}mlp.e{k}.down"][:CODE] = 0.0
    for t in range(cfg["vocab"]):
        for _ in range(10000):
            code = torch.randn(CODE, generator=g)
            code = (1.5 * code / code.norm() * math.sqrt(CODE)).to(dtype)
            if all(_apart(code, w[f"l{i}.norm1"], w[f"l{i}.mlp.router"], e["mlp"]["router"]) for i, e in enumerate(cfg["layers"]) if e["mlp"]):
                break
        else:
            raise AssertionError("no code keeps the experts apart")
        w["embed"][t, :CODE] = code
    return w


def _apart(code, gain, router, sizes) -> bool:
    z = torch.sort(router[:, :CODE].double() @ (gain[:CODE].double() * code.double()), descending=True).values
    return sizes["top"] == sizes["experts"] or float(z[sizes["top"] - 1] - z[sizes["top"]]) > APART


def write_folder(path, cfg: dict, weights: dict) -> Path:
    from quantinfer_b200.weights import write_safetensors

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg, indent=1))
    write_safetensors(path / "model.safetensors", {k: v.contiguous() for k, v in weights.items()})
    return path


def make(path, name: str):
    """(folder, config, weights) of the named configuration."""
    cfg = CONFIGS[name]
    w = draw_weights(cfg, SEEDS[name])
    return write_folder(path, cfg, w), cfg, w


def plain_rows(cfg: dict, weights: dict, requests: dict) -> dict:
    """{(request, position): logits row} from the plain implementation."""
    from plain import plain_bomipel

    rows = {}
    for rid, toks in requests.items():
        logits = plain_bomipel.forward(cfg, weights, toks).to(torch.float32).numpy()
        for p in range(len(toks)):
            rows[(rid, p)] = logits[p]
    return rows
