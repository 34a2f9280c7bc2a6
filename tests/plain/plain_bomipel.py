"""A plain, slow restatement of the Bomipel design in float64, one function per mechanism, for whole sequences at once
(no cache, no batching, keys and values formed per head). It reads the design's config dictionary and a dictionary of
tensors by name and shares nothing with the engine.

Notation: T tokens, positions 0 .. T - 1; matrices are stored [out, in] and applied as x @ W.T.
"""

from __future__ import annotations

import math

import torch

F = torch.float64


def f64(t):
    return t.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def rms_norm(x, gain, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * f64(gain)


def pair_frequencies(dims, base, scaling=None):
    """One frequency a pair: base^(-2i / dims). With `scaling` (factor, low, high, original): a pair whose wavelength is
    above original / low turns `factor` times slower, one below original / high as it is, between the two a blend."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / f
            factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            if length > original / low:
                f = f / factor
            elif length >= original / high:
                s = (original / length - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate(x, dims, freqs, layout):
    """x [T, heads, d]: the first `dims` coordinates turn by position * frequency; pair i is (2i, 2i + 1) for layout
    "interleaved" and (i, i + dims / 2) for "half"."""
    if not dims:
        return x
    ang = torch.arange(x.shape[0], dtype=F)[:, None, None] * freqs
    c, s = torch.cos(ang), torch.sin(ang)
    first = slice(0, dims, 2) if layout == "interleaved" else slice(0, dims // 2)
    second = slice(1, dims, 2) if layout == "interleaved" else slice(dims // 2, dims)
    u, v = x[..., first], x[..., second]
    out = x.clone()
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


def visible(T, size=None, keep_first=0):
    """[T, T] True where query i sees key j: j <= i, and i - j < size or j < keep_first (size None: every earlier key)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size is None else (i - j) < size
    return (j <= i) & (near | (j < keep_first))


def softmax_over(scores, ok):
    return torch.softmax(scores.masked_fill(~ok, -math.inf), dim=-1)


def mix_values(v, v_first, share):
    return (1.0 - share) * v + share * v_first


def attention(h, m, w, p, v_first=None):
    """Returns (output, values of this layer before any mixing). `v_first`: another layer's values to mix in, or None."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ f64(w[p + "q"]).T).view(T, H, d)
    k = (h @ f64(w[p + "k"]).T).view(T, G, d)
    v = own = (h @ f64(w[p + "v"]).T).view(T, G, e)
    if v_first is not None:
        v = mix_values(v, v_first, float(w[p + "vmix"]))
    rot = m.get("rot")
    if rot and rot["dims"]:
        freqs = pair_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate(q, rot["dims"], freqs, "interleaved"), rotate(k, rot["dims"], freqs, "interleaved")
    mask = m.get("mask") or {}
    ok = visible(T, mask.get("size"), mask.get("keep_first", 0))
    heads = []
    for head in range(H):
        g = head // (H // G)
        heads.append(softmax_over(q[:, head] @ k[:, g].T * m["scale"], ok) @ v[:, g])
    return torch.cat(heads, dim=-1) @ f64(w[p + "o"]).T, own


def latent_attention(h, m, w, p, eps):
    T = h.shape[0]
    H, d, r, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_norm(h @ f64(w[p + "dq"]).T, w[p + "dq.norm"], eps)
    q = (cq @ f64(w[p + "uq"]).T).view(T, H, d + r)
    z = h @ f64(w[p + "dkv"]).T
    c, kr = rms_norm(z[:, :R], w[p + "dkv.norm"], eps), z[:, R:].reshape(T, 1, r)
    qp, qr = q[..., :d], q[..., d:]
    rot = m.get("rot")
    if rot and rot["dims"]:
        freqs = pair_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        qr, kr = rotate(qr, rot["dims"], freqs, "half"), rotate(kr, rot["dims"], freqs, "half")
    k = (c @ f64(w[p + "uk"]).T).view(T, H, d)
    v = (c @ f64(w[p + "uv"]).T).view(T, H, e)
    ok = visible(T)
    heads = []
    for head in range(H):
        scores = (qp[:, head] @ k[:, head].T + qr[:, head] @ kr[:, 0].T) * m["scale"]
        heads.append(softmax_over(scores, ok) @ v[:, head])
    return torch.cat(heads, dim=-1) @ f64(w[p + "o"]).T


def route(h, w_router, top):
    """Per token the `top` experts with the largest sigmoid score, and those scores as they are."""
    scores = torch.sigmoid(h @ f64(w_router).T)
    return torch.topk(scores, top, dim=-1)


def expert(x, w, p):
    return (silu(x @ f64(w[p + "gate"]).T) * (x @ f64(w[p + "up"]).T)) @ f64(w[p + "down"]).T


def mixture(h, mlp, w, p):
    """The score multiplies what an expert reads."""
    scores, chosen = route(h, w[p + "router"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for s, e in zip(scores[t], chosen[t]):
            out[t] += expert(s * h[t], w, f"{p}e{int(e)}.")
    return out


def cap(z, c):
    return c * torch.tanh(z / c) if c else z


def forward(cfg, w, tokens, keep_layers=False):
    """Logits [T, vocab] of a whole sequence; with keep_layers also the stream after every layer [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    x = f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
    v_first, kept = None, []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, m, w, p + "mix.", eps)
        elif layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, m, w, p + "mix.", v_first if mixes else None)
            if mixes and v_first is None:
                v_first = own
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            y = y + mixture(h, layer["mlp"], w, p + "mlp.")
        x = x + y
        if keep_layers:
            kept.append(x.clone())
    logits = cap(rms_norm(x, w["final.norm"], eps) @ f64(w["embed"]).T, cfg.get("logit_softcap"))
    return (logits, torch.stack(kept)) if keep_layers else logits
