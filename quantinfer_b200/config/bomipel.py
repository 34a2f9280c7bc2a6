"""Typed configuration of the Bomipel design, read from the keys of its config.json.

A small decoder-only model whose layers have ONE RMS norm (gain per coordinate) that feeds a mixer and a feed-forward side
by side: x <- x + (mixer(h) + ff(h)). Two mixers. (1) Grouped-query softmax attention without biases: separate key and value
sizes, rotation in neighbouring pairs over the first coordinates of each head whose frequencies may be scaled in bands of
wavelength, a sliding window behind which the sequence's first tokens stay visible, and values that are mixed with those
of the first layer that does so. (2) Attention over a cached latent whose queries come through a latent of their own, with a
rotated part in half-split pairs, over every earlier position. The feed-forward is a mixture of small gated experts (silu):
the `top` experts with the largest sigmoid scores, whose scores, as they are, multiply the experts' inputs. The output head is
the embedding table, its logits soft-capped.

config.json keys (every size, and every constant that can differ between models):

    architecture            "Bomipel"
    vocab, width
    norm.eps                eps of every RMS norm
    logit_softcap           c in c tanh(logits / c) (absent or null: none)
    layers[i]               {type: "attention" | "latent_attention", mixer: {...}, mlp: {...} or null}
      attention             {heads, kv_heads, dim, vdim, scale, v_mix (optional), rot: {base, dims, scaling: {factor, low, high,
                             original} (optional)} (optional), mask: {size, keep_first (optional)} (optional)}
      latent_attention      {heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot: {base, dims, scaling (optional)} (optional)}
      mlp                   {kind: "moe", router: {experts, top}, expert: {ff}}

Tensor names: `embed`, `l<i>.norm1`, `l<i>.mix.{q,k,v,vmix,o}` or `l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}`,
`l<i>.mlp.{router,e<k>.gate|up|down}`, `final.norm`. The design sets no limit on positions.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field

from ..errors import ConfigError
from .bebuvik import UNLIMITED_POSITIONS, _get
from .spec import (EmbeddingSpec, FeedForwardSpec, GatedAttentionSpec, HeadSpec, LatentAttentionSpec, LayerCall, ModelSpec, MoESpec,
                   NormSpec, ParallelLayerSpec, RotarySpec)

ARCHITECTURE = "Bomipel"

# constants the design fixes
EXPERT_ACTIVATION = "silu"
ROUTER_SCORES = "sigmoid"
ATTENTION_PAIRING = "interleaved"  # coordinate 2i turns with coordinate 2i + 1
LATENT_PAIRING = "half_split"      # coordinate i turns with coordinate i + dims / 2


@dataclass(frozen=True)
class BomipelRotation:
    base: float
    dims: int
    bands: object = None           # (factor, low, high, original) or None


@dataclass(frozen=True)
class BomipelAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: object = None             # BomipelRotation or None
    window: object = None          # None: every earlier position
    keep_first: int = 0
    v_mix: bool = False


@dataclass(frozen=True)
class BomipelLatent:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: object = None


@dataclass(frozen=True)
class BomipelMoE:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class BomipelLayer:
    mixer: object                  # BomipelAttention or BomipelLatent
    mlp: object = None             # BomipelMoE or None


def _rotation(m, where):
    rot = _get(m, "rot", dict, where, required=False)
    if rot is None:
        return None
    rw = where + "rot."
    sc = _get(rot, "scaling", dict, rw, required=False)
    bands = tuple(_get(sc, k, float, rw + "scaling.") for k in ("factor", "low", "high", "original")) if sc is not None else None
    r = BomipelRotation(_get(rot, "base", float, rw), _get(rot, "dims", int, rw), bands)
    return r if r.dims else None


def _rotation_dict(r):
    d = {"base": r.base, "dims": r.dims}
    if r.bands is not None:
        d["scaling"] = dict(zip(("factor", "low", "high", "original"), r.bands))
    return d


@dataclass(frozen=True)
class BomipelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple
    logit_softcap: object = None
    raw: dict = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, d: dict) -> "BomipelConfig":
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
            m, mw, kind = _get(entry, "mixer", dict, where), where + "mixer.", entry.get("type")
            if kind == "attention":
                mask = _get(m, "mask", dict, mw, required=False)
                mix = m.get("v_mix", False)
                if mix not in (True, False, None):
                    raise ConfigError(f"config.json `{mw}v_mix` must be true or false")
                mixer = BomipelAttention(
                    heads=_get(m, "heads", int, mw), kv_heads=_get(m, "kv_heads", int, mw), dim=_get(m, "dim", int, mw),
                    vdim=_get(m, "vdim", int, mw), scale=_get(m, "scale", float, mw), rot=_rotation(m, mw),
                    window=_get(mask, "size", int, mw + "mask.", required=False) if mask is not None else None,
                    keep_first=_get(mask, "keep_first", int, mw + "mask.", required=False, default=0) if mask is not None else 0,
                    v_mix=bool(mix))
            elif kind == "latent_attention":
                mixer = BomipelLatent(
                    heads=_get(m, "heads", int, mw), dim=_get(m, "dim", int, mw), rot_dim=_get(m, "rot_dim", int, mw),
                    vdim=_get(m, "vdim", int, mw), q_rank=_get(m, "q_rank", int, mw), kv_rank=_get(m, "kv_rank", int, mw),
                    scale=_get(m, "scale", float, mw), rot=_rotation(m, mw))
            else:
                raise ConfigError(f"config.json `{where}type` is {kind!r}; this design's mixers are 'attention' and 'latent_attention'")
            mlp_in, mlp = entry.get("mlp"), None
            if mlp_in is not None:
                lw = where + "mlp."
                if not isinstance(mlp_in, dict) or mlp_in.get("kind") != "moe":
                    raise ConfigError(f"config.json `{where}mlp` must be null or an object of kind 'moe'")
                r, e = _get(mlp_in, "router", dict, lw), _get(mlp_in, "expert", dict, lw)
                mlp = BomipelMoE(_get(r, "experts", int, lw + "router."), _get(r, "top", int, lw + "router."), _get(e, "ff", int, lw + "expert."))
            layers.append(BomipelLayer(mixer, mlp))
        cfg = cls(vocab=_get(d, "vocab", int, ""), width=_get(d, "width", int, ""),
                  norm_eps=_get(_get(d, "norm", dict, ""), "eps", float, "norm."), layers=tuple(layers),
                  logit_softcap=_get(d, "logit_softcap", float, "", required=False), raw=copy.deepcopy(d))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        if self.raw:
            return copy.deepcopy(self.raw)
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "layers": []}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        for layer in self.layers:
            m = layer.mixer
            if isinstance(m, BomipelAttention):
                kind = "attention"
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window, "keep_first": m.keep_first}
                if m.v_mix:
                    mixer["v_mix"] = True
            else:
                kind = "latent_attention"
                mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank,
                         "scale": m.scale}
            if m.rot is not None:
                mixer["rot"] = _rotation_dict(m.rot)
            f = layer.mlp
            d["layers"].append({"type": kind, "mixer": mixer, "mlp": None if f is None else
                                {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.ff}}})
        return d

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("Bomipel `vocab` and `width` must be greater than zero")
        if self.norm_eps <= 0.0:
            raise ConfigError("Bomipel `norm.eps` must be positive")
        if self.logit_softcap is not None and self.logit_softcap <= 0.0:
            raise ConfigError("Bomipel `logit_softcap` must be positive (or absent)")
        first = None
        for i, layer in enumerate(self.layers):
            m, f = layer.mixer, layer.mlp
            if m.scale <= 0.0:
                raise ConfigError(f"Bomipel layer {i}: scale must be positive")
            if isinstance(m, BomipelAttention):
                turned = m.dim
                if min(m.heads, m.kv_heads, m.dim, m.vdim) <= 0 or m.heads % m.kv_heads:
                    raise ConfigError(f"Bomipel layer {i}: heads must be a positive multiple of kv_heads, dim and vdim positive")
                if max(m.dim, m.vdim) > 256:
                    raise ConfigError(f"Bomipel layer {i}: dim and vdim are at most 256 (the attention kernels' limit)")
                if m.window is not None and m.window <= 0:
                    raise ConfigError(f"Bomipel layer {i}: mask.size must be positive")
                if m.v_mix:
                    if first is None:
                        first = (i, m)
                    elif (m.kv_heads, m.vdim) != (first[1].kv_heads, first[1].vdim):
                        raise ConfigError(f"Bomipel layer {i}: it mixes in the values of layer {first[0]}, so kv_heads and vdim must be equal")
            else:
                turned = m.rot_dim
                if min(m.heads, m.dim, m.vdim, m.q_rank, m.kv_rank) <= 0:
                    raise ConfigError(f"Bomipel layer {i}: heads, dim, vdim, q_rank and kv_rank must be greater than zero")
                if m.kv_rank > 512:
                    raise ConfigError(f"Bomipel layer {i}: kv_rank is at most 512 (the attention kernels' limit)")
            if m.rot is not None:
                if m.rot.dims % 2 or m.rot.dims > turned:
                    raise ConfigError(f"Bomipel layer {i}: rot.dims ({m.rot.dims}) must be even and within the {turned} coordinates it turns")
                if m.rot.base <= 0.0:
                    raise ConfigError(f"Bomipel layer {i}: rot.base must be positive")
                if m.rot.bands is not None and (min(m.rot.bands) <= 0.0 or m.rot.bands[2] < m.rot.bands[1]):
                    raise ConfigError(f"Bomipel layer {i}: rot.scaling needs positive factor, low, high and original, high at least low")
            if f is not None and (not 0 < f.top <= f.experts or f.ff <= 0 or f.experts > 1024):
                raise ConfigError(f"Bomipel layer {i}: a mixture needs 0 < top <= experts <= 1024 and ff > 0")

    # ---- the model as data --------------------------------------------------

    def to_model_spec(self) -> ModelSpec:
        w, eps = self.width, self.norm_eps
        layers, mixed = [], False
        for i, layer in enumerate(self.layers):
            p, m, f = f"l{i}.", layer.mixer, layer.mlp
            if isinstance(m, BomipelAttention):
                role = None
                if m.v_mix:
                    role, mixed = ("mix" if mixed else "first"), True
                mixer = GatedAttentionSpec(
                    hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                    position=RotarySpec(m.rot.dims, m.rot.base, ATTENTION_PAIRING, bands=m.rot.bands) if m.rot is not None else None,
                    scale=m.scale, window=m.window, bias=False, out_gate=False, prefix=p + "mix.",
                    keep_first=m.keep_first if m.window is not None else 0, value_mix=role)
            else:
                mixer = LatentAttentionSpec(
                    hidden_size=w, num_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, value_dim=m.vdim, kv_rank=m.kv_rank,
                    position=RotarySpec(m.rot.dims, m.rot.base, LATENT_PAIRING, bands=m.rot.bands) if m.rot is not None else None,
                    norm_eps=eps, scale=m.scale, prefix=p + "mix.", q_rank=m.q_rank)
            ffn = MoESpec(hidden_size=w, experts=f.experts, top=f.top, router_scale=1.0,
                          expert=FeedForwardSpec(w, f.ff, EXPERT_ACTIVATION, p + "mlp."), prefix=p + "mlp.", scoring=ROUTER_SCORES,
                          has_correction=False, normalize=False, weight_on="input") if f is not None else None
            layers.append(ParallelLayerSpec(norm=NormSpec(w, eps, p + "norm1", "rmsnorm_named"), mixer=mixer, ffn=ffn, kind="parallel"))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=w, max_positions=UNLIMITED_POSITIONS,
            embedding=EmbeddingSpec(self.vocab, w, "", weight_name="embed"), layers=tuple(layers),
            order=tuple(LayerCall(i, i, True) for i in range(len(layers))), final_norm=NormSpec(w, eps, "final.norm", "rmsnorm_named"),
            head=HeadSpec(self.vocab, w, True, softcap=self.logit_softcap), eos_token_id=None)
        spec.validate()
        return spec
