"""A plain, slow restatement of the Siditar design in float64, one function per mechanism, for whole
sequences at once (no cache, no state carried between calls, no batching). It reads the design's config
dictionary and a dictionary of tensors by name and shares nothing with the engine.

Notation: T tokens, positions 0 .. T - 1; matrices are stored [out, in] and applied as x @ W.T.
"""

from __future__ import annotations

import math
from fractions import Fraction

import torch

F = torch.float64


def f64(t):
    return t.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    """Deviations from the mean over their root mean square, times a gain; there is no offset."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * f64(w)


def sinusoid(T, width):
    """[T, width]: coordinates 2i and 2i + 1 are the sine and the cosine of p / 10000^(2i / width)."""
    p = torch.arange(T, dtype=F)[:, None]
    out = torch.zeros(T, width, dtype=F)
    for c in range(width):
        angle = p[:, 0] * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(angle) if c % 2 else torch.sin(angle)
    return out


def embedding(w, tokens, width):
    return f64(w["embed"])[torch.as_tensor(tokens)] + sinusoid(len(tokens), width)


def distance_bucket(n, rows, reach):
    """Which of `rows` numbers a distance of n positions reads: the first half of them one a distance, the others over
    distances that grow geometrically up to `reach`. A distance n lies at least m steps into the second half when
    (n / h)^(rows - h) >= (reach / h)^m with h = rows / 2: compared exactly, in whole numbers."""
    h = Fraction(rows, 2)
    if n < h:
        return n
    steps, left, ratio = 0, (Fraction(n) / h) ** int(rows - h), Fraction(reach) / h
    while h + steps < rows - 1 and left >= ratio ** (steps + 1):
        steps += 1
    return int(h) + steps


def distance_bias(table, T, reach):
    """[heads, T, T]: the number that head h adds to the score of query i and key j <= i."""
    rows, heads = table.shape
    bucket = [distance_bucket(n, rows, reach) for n in range(T)]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    index = torch.tensor(bucket)[(i - j).clamp(min=0)]
    return f64(table)[index].permute(2, 0, 1)


def query_temperature(T, coef, every):
    return torch.tensor([1.0 + coef * math.log((p + 1) // every + 1) for p in range(T)], dtype=F)


def softmax_with_sink(s, ok, sink):
    """Weights over the visible keys of [heads, T, T] scores; exp(sink) stands once more in the denominator."""
    s = s.masked_fill(~ok, -math.inf)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def attention(w, p, m, h, eps):
    """The left branch."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ f64(w[p + "q"]).T).reshape(T, H, d)
    k = (h @ f64(w[p + "k"]).T).reshape(T, G, d)
    v = (h @ f64(w[p + "v"]).T).reshape(T, G, dv)
    q = unit_rms(q, eps) * f64(w[p + "q.norm"])
    k = unit_rms(k, eps) * f64(w[p + "k.norm"])
    if m.get("q_temp"):
        q = q * query_temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] + distance_bias(w[p + "rel"], T, m["bias_max"])
    ok = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    a = torch.einsum("hij,jhe->ihe", softmax_with_sink(s, ok, f64(w[p + "sink"])), v)
    return a.reshape(T, H * dv) @ f64(w[p + "o"]).T


def decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def gated_linear_scan(q, k, v, alpha):
    """q, k, alpha [T, heads, d], v [T, heads, e]: S = diag(alpha_t) S + k_t v_t^T; o_t = S^T q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F)
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", S, q[t])
    return out


def linear_attention(w, p, m, h, eps):
    """The right branch."""
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ f64(w[p + "q"]).T).reshape(T, H, d) / math.sqrt(d)
    k = (h @ f64(w[p + "k"]).T).reshape(T, H, d)
    v = (h @ f64(w[p + "v"]).T).reshape(T, H, e)
    z = h @ f64(w[p + "a1"]).T @ f64(w[p + "a2"]).T + f64(w[p + "a2.b"])
    o = gated_linear_scan(q, k, v, decay(z, m["tau"]).reshape(T, H, d))
    o = unit_rms(o, eps) * f64(w[p + "norm"])
    return (o.reshape(T, H * e) * silu(h @ f64(w[p + "g"]).T)) @ f64(w[p + "o"]).T


def two_branches(w, p, m, h, eps):
    return m["left_scale"] * attention(w, p + "left.", m["left"], h, eps) + m["right_scale"] * linear_attention(
        w, p + "right.", m["right"], h, eps)


def feed_forward(w, p, limit, h):
    g = torch.clamp(h @ f64(w[p + "gate"]).T, max=limit)
    u = torch.clamp(h @ f64(w[p + "up"]).T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ f64(w[p + "down"]).T


def hyper_step(w, p, streams, sublayer):
    """streams [s, T, width]: the sublayer reads their weighted sum, and every new stream is a mix of all the old
    ones (`mix` indexed [from, to]) plus its share of the sublayer's result."""
    into, out, mix = f64(w[p + "in"]), f64(w[p + "out"]), f64(w[p + "mix"])
    y = sublayer((into[:, None, None] * streams).sum(0))
    return torch.stack([(mix[:, t, None, None] * streams).sum(0) + out[t] * y for t in range(streams.shape[0])])


def run_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, w, tokens, taps=None):
    """Logits [T, vocab]; the sum of the streams after every layer run goes into `taps` when that is a list."""
    eps = cfg["norm"]["eps"]
    x = embedding(w, tokens, cfg["width"]).repeat(cfg["streams"], 1, 1)
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        x = hyper_step(w, p + "hc1.", x, lambda u: two_branches(w, p + "mix.", layer["mixer"], layer_norm(u, w[p + "norm1"], eps), eps))
        if layer["mlp"] is not None:
            x = hyper_step(w, p + "hc2.", x, lambda u: feed_forward(w, p + "mlp.", layer["mlp"]["limit"], layer_norm(u, w[p + "norm2"], eps)))
        if taps is not None:
            taps.append(x.sum(0))
    return layer_norm(x.sum(0), w["final.norm"], eps) @ f64(w["head"]).T
