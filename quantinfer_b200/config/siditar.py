"""Typed configuration of the Siditar design, read from the keys of its config.json.

A small decoder-only model with several residual streams that every sublayer mixes (hyper-connections), a sinusoidal
position vector on the embedding, pre-norm layer norms without bias, and a stretch of layers that may run several times
with the same weights. Every mixer is two branches side by side on one input: softmax attention over grouped heads (an
RMS norm over every head of q and k, queries that grow warmer with the position, a learned bias by the key's distance, a
learned sink per head, no rotation) and gated linear attention (a matrix state per head, a decay per key channel that is a
gate of the token, an RMS norm per head, an output gate); the mixer is their weighted sum. The feed-forward is a clamped
gated one.

config.json keys (every size, and every constant that can differ between models):

    architecture            "Siditar"
    vocab, width
    streams                 residual streams
    norm.eps                eps of every norm
    loop                    {start, stop, times}: layers start .. stop - 1 run `times` times in a row (absent: once)
    layers[i]               {type: "parallel", mixer: {...}, mlp: {kind: "dense", ff, limit} or null}
      mixer                 {left: {heads, kv_heads, dim, vdim, scale, bias_max, q_temp: {coef, every}}, left_scale,
                             right: {heads, dim, vdim, tau}, right_scale}

Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.hc1|hc2.{in,out,mix}`, `l<i>.mix.left.{q,k,v,q.norm,k.norm,rel,sink,o}`,
`l<i>.mix.right.{q,k,v,g,a1,a2,a2.b,norm,o}`, `l<i>.mlp.{gate,up,down}`, `final.norm`, `head`. The rows of `rel` and the
rank of `a1` are read from the tensors. The design sets no limit on positions.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field

from ..errors import ConfigError
from .bebuvik import UNLIMITED_POSITIONS, _get
from .spec import (ClampedGLUSpec, EmbeddingSpec, GatedAttentionSpec, GatedLinearAttentionSpec, HeadSpec, HyperLayerSpec, LayerCall,
                   ModelSpec, NormSpec, ParallelMixersSpec, StreamSumNormSpec)

ARCHITECTURE = "Siditar"

# constants the design fixes
POSITION_BASE = 10000.0            # of the sinusoidal position vector
GLU_ALPHA = 1.702                  # inside the feed-forward's sigmoid
MAX_STREAMS = 16                   # what the streams' kernel takes


@dataclass(frozen=True)
class SiditarAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    temp_coef: float = 0.0
    temp_every: object = None      # None: the queries keep their length


@dataclass(frozen=True)
class SiditarLinearAttention:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class SiditarLayer:
    left: SiditarAttention
    right: SiditarLinearAttention
    left_scale: float
    right_scale: float
    ff: object = None              # the feed-forward's inner width; None: no feed-forward
    limit: float = 0.0


@dataclass(frozen=True)
class SiditarConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    layers: tuple
    loop: object = None            # (start, stop, times) or None
    raw: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, d: dict) -> "SiditarConfig":
        if not isinstance(d, dict):
            raise ConfigError("config.json must hold a JSON object")
        if d.get("architecture", ARCHITECTURE) != ARCHITECTURE and ARCHITECTURE not in (d.get("architectures") or []):
            raise ConfigError(f"this is not a {ARCHITECTURE} configuration")
        layers_in = d.get("layers")
        if not isinstance(layers_in, list) or not layers_in:
            raise ConfigError("config.json `layers` must be a non-empty list")
        layers = []
        for i, entry in enumerate(layers_in):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json `layers[{i}]` must be an object")
            if entry.get("type") != "parallel":
                raise ConfigError(f"config.json `{where}type` is {entry.get('type')!r}; this design's mixer is 'parallel'")
            m = _get(entry, "mixer", dict, where)
            mw = where + "mixer."
            l, r = _get(m, "left", dict, mw), _get(m, "right", dict, mw)
            lw, rw = mw + "left.", mw + "right."
            temp = _get(l, "q_temp", dict, lw, required=False)
            left = SiditarAttention(
                heads=_get(l, "heads", int, lw), kv_heads=_get(l, "kv_heads", int, lw), dim=_get(l, "dim", int, lw),
                vdim=_get(l, "vdim", int, lw), scale=_get(l, "scale", float, lw), bias_max=_get(l, "bias_max", float, lw),
                temp_coef=_get(temp, "coef", float, lw + "q_temp.") if temp is not None else 0.0,
                temp_every=_get(temp, "every", int, lw + "q_temp.") if temp is not None else None)
            right = SiditarLinearAttention(heads=_get(r, "heads", int, rw), dim=_get(r, "dim", int, rw), vdim=_get(r, "vdim", int, rw),
                                           tau=_get(r, "tau", float, rw))
            mlp, ff, limit = entry.get("mlp"), None, 0.0
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
                    raise ConfigError(f"config.json `{where}mlp` must be null or an object of kind 'dense'")
                ff, limit = _get(mlp, "ff", int, where + "mlp."), _get(mlp, "limit", float, where + "mlp.")
            layers.append(SiditarLayer(left, right, _get(m, "left_scale", float, mw), _get(m, "right_scale", float, mw), ff, limit))
        loop_in, loop = _get(d, "loop", dict, "", required=False), None
        if loop_in is not None:
            loop = tuple(_get(loop_in, k, int, "loop.") for k in ("start", "stop", "times"))
        cfg = cls(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""), streams=_get(d, "streams", int, ""),
                  norm_eps=_get(_get(d, "norm", dict, ""), "eps", float, "norm."), layers=tuple(layers), loop=loop, raw=copy.deepcopy(d))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        if self.raw:
            return copy.deepcopy(self.raw)
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "streams": self.streams,
             "norm": {"eps": self.norm_eps}, "layers": []}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        for layer in self.layers:
            l, r = layer.left, layer.right
            left = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale, "bias_max": l.bias_max}
            if l.temp_every is not None:
                left["q_temp"] = {"coef": l.temp_coef, "every": l.temp_every}
            d["layers"].append({
                "type": "parallel",
                "mixer": {"left": left, "left_scale": layer.left_scale,
                          "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "tau": r.tau}, "right_scale": layer.right_scale},
                "mlp": {"kind": "dense", "ff": layer.ff, "limit": layer.limit} if layer.ff is not None else None})
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("Siditar `vocab` and `width` must be greater than zero")
        if not 1 <= self.streams <= MAX_STREAMS:
            raise ConfigError(f"Siditar `streams` ({self.streams}) must lie in 1..{MAX_STREAMS}")
        if self.norm_eps <= 0.0:
            raise ConfigError("Siditar `norm.eps` must be positive")
        if self.loop is not None:
            a, b, times = self.loop
            if not 0 <= a < b <= len(self.layers) or times < 1:
                raise ConfigError(f"Siditar `loop` {self.loop} must name a stretch of the {len(self.layers)} layers and run it at least once")
        for i, layer in enumerate(self.layers):
            l, r = layer.left, layer.right
            if min(l.heads, l.kv_heads, l.dim, l.vdim) <= 0 or l.heads % l.kv_heads:
                raise ConfigError(f"Siditar layer {i}: left.heads must be a positive multiple of left.kv_heads, dim and vdim positive")
            if l.dim > 256 or l.vdim > 256:
                raise ConfigError(f"Siditar layer {i}: left.dim and left.vdim must not exceed 256 (the attention kernels' limit)")
            if l.scale <= 0.0 or l.bias_max <= 0.0:
                raise ConfigError(f"Siditar layer {i}: left.scale and left.bias_max must be positive")
            if l.temp_every is not None and l.temp_every < 1:
                raise ConfigError(f"Siditar layer {i}: left.q_temp.every must be at least one")
            if min(r.heads, r.dim, r.vdim) <= 0 or r.dim > 256:
                raise ConfigError(f"Siditar layer {i}: right.heads, dim and vdim must be greater than zero, dim at most 256")
            if r.tau <= 0.0:
                raise ConfigError(f"Siditar layer {i}: right.tau must be positive")
            if layer.ff is not None and (layer.ff <= 0 or layer.limit <= 0.0):
                raise ConfigError(f"Siditar layer {i}: mlp.ff and mlp.limit must be greater than zero")

    # ---- the model as data --------------------------------------------------

    def run_order(self) -> list:
        """The layers in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def to_model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps

        def norm(name):
            return NormSpec(w, eps, name, "layernorm_nobias")

        layers = []
        for i, layer in enumerate(self.layers):
            p, l, r = f"l{i}.", layer.left, layer.right
            left = GatedAttentionSpec(
                hidden_size=w, num_heads=l.heads, num_kv_heads=l.kv_heads, head_dim=l.dim, value_dim=l.vdim, position=None,
                scale=l.scale, bias=False, out_gate=False, prefix=p + "mix.left.", sink="learned", qk_norm="head", qk_norm_eps=eps,
                q_temp=(l.temp_coef, l.temp_every) if l.temp_every is not None else None, distance_bias=l.bias_max)
            right = GatedLinearAttentionSpec(hidden_size=w, heads=r.heads, head_dim=r.dim, value_dim=r.vdim, tau=r.tau, norm_eps=eps,
                                             prefix=p + "mix.right.")
            mixer = ParallelMixersSpec(left, right, prefix=p + "mix.", branch_scales=(layer.left_scale, layer.right_scale), hidden_size=w,
                                       merged=True)
            ffn = ClampedGLUSpec(w, layer.ff, layer.limit, GLU_ALPHA, p + "mlp.") if layer.ff is not None else None
            layers.append(HyperLayerSpec(mixer_norm=norm(p + "norm1"), mixer=mixer, ffn_norm=norm(p + "norm2") if ffn is not None else None,
                                         ffn=ffn, streams=self.streams,
                                         names=(p + "hc1", p + "hc2") if ffn is not None else (p + "hc1",)))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=w, max_positions=UNLIMITED_POSITIONS,
            embedding=EmbeddingSpec(self.vocab, w, "", weight_name="embed", sinusoid_base=POSITION_BASE, copies=self.streams),
            layers=tuple(layers), order=tuple(LayerCall(i, entry) for entry, i in enumerate(self.run_order())),
            final_norm=StreamSumNormSpec(norm("final.norm"), self.streams),
            head=HeadSpec(self.vocab, w, False, "", weight_name="head"), eos_token_id=None)
        spec.validate()
        return spec
