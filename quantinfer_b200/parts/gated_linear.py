"""Linear attention over a matrix state per head whose decay per key channel is a gate of the token (gated linear attention).

    [q | k | v | g] = x . W^T                 (the four projections stacked at load: one product)
    z = W_a2 (W_a1 x) + b                     (the second product's output stays 32-bit)
    w = sigmoid(z)^(1 / tau)                  per head and key channel, as exp(-softplus(-z) / tau), 32-bit
    S_t = diag(w_t) S_(t-1) + k_t v_t^T       o_t = S_t^T q_t head_dim^(-1/2)                       (32-bit, per head)
    y = (o / rms(o) per head * norm * silu(g)) . Wo^T

A request's state of fixed size is S for every head, one row of 32-bit numbers in its slot, zero at a sequence's start. The
rank of the decay's two projections is read from `a1`.
"""

from __future__ import annotations

import torch

from .. import kernels
from . import segments
from ..cache.needs import StateNeed
from ..errors import ConfigError, WeightError
from ..weights.loader import TensorNeed
from .base import Part, register_part
from .linear import Linear


class GatedLinearAttention(Part):
    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        s = spec
        if min(s.heads, s.head_dim, s.value_dim) <= 0 or s.tau <= 0.0:
            raise ConfigError("gated_linear_attention: sizes and tau must be greater than zero")
        if s.head_dim > 256:
            raise ConfigError(f"gated_linear_attention: keys of {s.head_dim} are beyond the recurrence kernel (256)")
        self.qk, self.inner = s.heads * s.head_dim, s.heads * s.value_dim
        self.proj = Linear(runtime, 2 * self.qk + 2 * self.inner, s.hidden_size, s.prefix + "q+k+v+g")
        self.o = Linear(runtime, s.hidden_size, self.inner, s.prefix + "o")
        self.a1 = self.a2 = None            # built at load: their rank comes from the tensors
        self.gain = self.decay_bias = None

    @classmethod
    def needs_of_spec(cls, s):
        p, h, qk, inner = s.prefix, s.hidden_size, s.heads * s.head_dim, s.heads * s.value_dim
        return {p + "q": TensorNeed((qk, h)), p + "k": TensorNeed((qk, h)), p + "v": TensorNeed((inner, h)), p + "g": TensorNeed((inner, h)),
                p + "a1": TensorNeed((None, h)), p + "a2": TensorNeed((qk, None)), p + "a2.b": TensorNeed((qk,), "matrix", "zeros"),
                p + "norm": TensorNeed((s.value_dim,), "gain", "gain"), p + "o": TensorNeed((h, inner))}

    def load(self, tensors):
        p, s = self.spec.prefix, self.spec
        ws = [tensors[p + n] for n in ("q", "k", "v", "g")]
        if len({t.dtype for t in ws}) > 1:
            ws = [t.to(torch.float32) for t in ws]
        self.proj.load(torch.cat(ws, dim=0))
        rank = tensors[p + "a1"].shape[0]
        if tensors[p + "a2"].shape[1] != rank:
            raise WeightError(f"{p}a1 has {rank} rows, {p}a2 has {tensors[p + 'a2'].shape[1]} columns: the decay's rank must be one number")
        self.a1 = Linear(self.runtime, rank, s.hidden_size, p + "a1")
        self.a2 = Linear(self.runtime, self.qk, rank, p + "a2")
        self.a1.load(tensors[p + "a1"])
        self.a2.load(tensors[p + "a2"])
        self.o.load(tensors[p + "o"])
        self.decay_bias = self._gain(tensors[p + "a2.b"])
        self.gain = self._gain(tensors[p + "norm"].to(torch.float32).repeat(s.heads))

    def cache_need(self):
        s = self.spec
        return StateNeed((s.heads * s.value_dim * s.head_dim,), torch.float32)

    def forward(self, x, batch, cache):
        s = self.spec
        n = x.shape[0]
        qk, inner = self.qk, self.inner
        proj = self.proj(x)
        z = self.a2(self.a1(x), out_dtype=torch.float32)
        S = cache.state.unflatten(1, (s.heads, s.value_dim, s.head_dim))
        o = torch.empty((n, inner), dtype=torch.float32, device=x.device)
        segments.matrix_state_scan("channel_gate", proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + inner], S, o, batch,
                                   s.heads, s.head_dim, s.value_dim, log_decay=z, decay_bias=self.decay_bias, rate=1.0 / s.tau,
                                   q_scale=float(s.head_dim) ** -0.5)
        y = torch.empty((n, inner), dtype=x.dtype, device=x.device)
        kernels.gated_group_rmsnorm(o, proj[:, 2 * qk + inner:], self.gain, s.norm_eps, y, s.heads, gate="silu")
        return self.o(y, keep_partials=True)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
