"""Shared by the Siditar tests: small configurations that differ from one another in every size and option, weights drawn
so that activations are of order one (attention far from uniform, sinks and distance biases in reach, decays slow enough
for a state to last, clamps that bite), model folders, and the plain implementation's logits."""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch


def left(heads, kv_heads, dim, vdim, bias_max, temp=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.0 / math.sqrt(dim),
         "bias_max": bias_max}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def right(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def layer(l, r, scales=(1.0, 1.0), ff=None, limit=None, rows=8, rank=5):
    """`_rows` and `_rank` are not keys of the design: the tests' weights are drawn with that many rows of the distance
    bias and that rank of the decay's pair."""
    return {"type": "parallel", "mixer": {"left": l, "left_scale": scales[0], "right": r, "right_scale": scales[1]},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff is not None else None, "_rows": rows, "_rank": rank}


def model(vocab, width, streams, eps, layers, loop=None):
    cfg = {"architecture": "Siditar", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIGS = {
    # no size a power of two or a multiple of eight; three streams; a loop over the middle, run twice, that holds a
    # layer without feed-forward; values narrower and wider than keys; temperatures that step inside the requests
    "P": model(131, 44, 3, 3e-6, [
        layer(left(6, 3, 10, 7, 40, (0.4, 16)), right(4, 5, 7, 8.0), (0.8, 1.3), 56, 1.5, rows=8, rank=5),
        layer(left(2, 2, 6, 12, 19, (0.2, 7)), right(3, 6, 4, 3.0), (1.4, 0.6), rows=6, rank=2),
        layer(left(3, 1, 14, 10, 33, (0.9, 50)), right(2, 9, 5, 20.0), (1.0, 0.7), 20, 0.8, rows=10, rank=7),
        layer(left(4, 2, 8, 8, 25), right(1, 3, 11, 1.0), (0.5, 1.0), 36, 3.0, rows=4, rank=1)], loop=(1, 3, 2)),
    # multiples of 16 (the tensor-core kernels' sizes); one kv head; one stream; no loop; a table whose edges fall on powers of two
    "Q": model(200, 64, 1, 1e-5, [
        layer(left(4, 1, 32, 32, 128, (0.3, 32)), right(2, 16, 32, 16.0), (1.2, 0.9), 96, 2.5, rows=16, rank=8),
        layer(left(2, 2, 64, 16, 64, (0.5, 24)), right(4, 32, 16, 4.0), (0.7, 1.1), 64, 1.0, rows=12, rank=16)]),
    # keys of the recurrence wider than a warp and wider than 64; four streams; a loop that runs once; a loop-free tail
    "R": model(97, 48, 4, 1e-6, [
        layer(left(2, 1, 64, 24, 60, (0.6, 11), scale=0.2), right(2, 40, 24, 12.0), (0.9, 0.8), 40, 1.2, rows=14, rank=3),
        layer(left(4, 4, 16, 40, 9, (0.3, 64)), right(3, 72, 8, 6.0), (1.1, 1.2), 24, 2.0, rows=2, rank=6)], loop=(0, 1, 1)),
    # five streams (beyond the kernel that keeps a row in registers), the whole model a loop
    "S": model(70, 40, 5, 1e-5, [
        layer(left(2, 1, 8, 16, 30, (0.5, 5)), right(2, 16, 8, 9.0), (1.0, 1.0), 24, 1.7, rows=6, rank=4)], loop=(0, 1, 3)),
}
PAGE_SIZES = {"P": 8, "Q": 16, "R": 8, "S": 8}
SEEDS = {"P": 69, "Q": 62, "R": 63, "S": 64}


def clean(cfg: dict) -> dict:
    """The configuration as the design's config.json holds it (without the tests' own keys)."""
    out = json.loads(json.dumps(cfg))
    for e in out["layers"]:
        e.pop("_rows", None)
        e.pop("_rank", None)
    return out


def draw_weights(cfg: dict, seed: int, dtype=torch.bfloat16) -> dict:
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def mat(out, inp, gain=1.0):
        return (torch.randn(out, inp, generator=g) * gain / math.sqrt(inp)).to(dtype)

    def vec(n, std, mean=0.0):
        return (mean + std * torch.randn(n, generator=g)).to(dtype)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g).to(dtype), "head": mat(cfg["vocab"], W, 2.0), "final.norm": vec(W, 0.2, 1.0)}
    for i, entry in enumerate(cfg["layers"]):
        p, l, r = f"l{i}.", entry["mixer"]["left"], entry["mixer"]["right"]
        subs = (1, 2) if entry["mlp"] is not None else (1,)
        for q in subs:
            w[f"{p}norm{q}"] = vec(W, 0.2, 1.0)
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = vec(S, 0.3, 1.0 / S), vec(S, 0.4, 1.0)
            mix = 0.75 * torch.eye(S) + 0.25 / S + 0.15 * torch.randn(S, S, generator=g)      # far from symmetric
            w[f"{p}hc{q}.mix"] = mix.to(dtype)
        a, H, G, d, e = p + "mix.left.", l["heads"], l["kv_heads"], l["dim"], l["vdim"]
        w[a + "q"], w[a + "k"], w[a + "v"], w[a + "o"] = mat(H * d, W), mat(G * d, W), mat(G * e, W), mat(W, H * e)
        w[a + "q.norm"], w[a + "k.norm"] = vec(d, 0.3, 1.4), vec(d, 0.3, 1.4)       # scores of several units
        w[a + "rel"], w[a + "sink"] = torch.randn(entry["_rows"], H, generator=g).to(dtype), vec(H, 1.0, 1.5)
        b, H, d, e, rank = p + "mix.right.", r["heads"], r["dim"], r["vdim"], entry["_rank"]
        w[b + "q"], w[b + "k"], w[b + "v"], w[b + "g"], w[b + "o"] = mat(H * d, W), mat(H * d, W), mat(H * e, W), mat(H * e, W, 1.5), mat(W, H * e)
        w[b + "a1"], w[b + "a2"], w[b + "a2.b"] = mat(rank, W, 1.5), mat(H * d, rank, 1.5), vec(H * d, 1.5, 2.0)
        w[b + "norm"] = vec(e, 0.2, 1.0)
        if entry["mlp"] is not None:
            ff = entry["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, W, 1.5), mat(ff, W, 1.5), mat(W, ff)
    return w


def write_folder(path, cfg: dict, weights: dict) -> Path:
    from quantinfer_b200.weights import write_safetensors

    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(clean(cfg), indent=1))
    write_safetensors(path / "model.safetensors", {k: v.contiguous() for k, v in weights.items()})
    return path


def make(path, name: str):
    """(folder, config, weights) of the named configuration."""
    cfg = CONFIGS[name]
    w = draw_weights(cfg, SEEDS[name])
    return write_folder(path, cfg, w), clean(cfg), w


def plain_rows(cfg: dict, weights: dict, requests: dict) -> dict:
    """{(request, position): logits row} from the plain implementation."""
    from plain import plain_siditar

    rows = {}
    for rid, toks in requests.items():
        logits = plain_siditar.forward(cfg, weights, toks).to(torch.float32).numpy()
        for p in range(len(toks)):
            rows[(rid, p)] = logits[p]
    return rows
