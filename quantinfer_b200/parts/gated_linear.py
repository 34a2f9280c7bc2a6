"""Linear attention over a matrix state per head whose decay per key channel is a gate of the token (gated linear attention).

    [q | k | v | g | a] = x . W^T             (the four projections and the decay's first, W_a1, stacked at load: one product)
    z = W_a2 a + b                            (this product's output stays 32-bit)
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
        self.o = Linear(runtime, s.hidden_size, self.inner, s.prefix + "o")
        self.proj = self.a2 = None          # built at load: the decay's rank comes from the tensors
        self.gain = self.decay_bias = None

    @classmethod
    def needs_of_spec(cls, s):
        p, h, qk, inner = s.prefix, s.hidden_size, s.heads * s.head_dim, s.heads * s.value_dim
        return {p + "q": TensorNeed((qk, h)), p + "k": TensorNeed((qk, h)), p + "v": TensorNeed((inner, h)), p + "g": TensorNeed((inner, h)),
                p + "a1": TensorNeed((None, h)), p + "a2": TensorNeed((qk, None)), p + "a2.b": TensorNeed((qk,), "matrix", "zeros"),
                p + "norm": TensorNeed((s.value_dim,), "gain", "gain"), p + "o": TensorNeed((h, inner))}

    def load(self, tensors):
        p, s = self.spec.prefix, self.spec
        ws = [tensors[p + n] for n in ("q", "k", "v", "g", "a1")]
        if len({t.dtype for t in ws}) > 1:
            ws = [t.to(torch.float32) for t in ws]
        rank = tensors[p + "a1"].shape[0]
        if tensors[p + "a2"].shape[1] != rank:
            raise WeightError(f"{p}a1 has {rank} rows, {p}a2 has {tensors[p + 'a2'].shape[1]} columns: the decay's rank must be one number")
        # the rank's columns start and end on 16-byte boundaries (rows of zeros between and after them), so that the second
        # product reads them where they lie
        cols = 2 * self.qk + 2 * self.inner
        self.low_at, self.rank = (cols + 7) // 8 * 8, (rank + 7) // 8 * 8
        rows = torch.zeros((self.low_at + self.rank, s.hidden_size), dtype=ws[0].dtype)
        rows[:cols], rows[self.low_at:self.low_at + rank] = torch.cat(ws[:4], dim=0), ws[4]
        self.proj = Linear(self.runtime, rows.shape[0], s.hidden_size, p + "q+k+v+g+a1")
        self.proj.load(rows)
        high = torch.zeros((self.qk, self.rank), dtype=tensors[p + "a2"].dtype)
        high[:, :rank] = tensors[p + "a2"]
        self.a2 = Linear(self.runtime, self.qk, self.rank, p + "a2")
        self.a2.load(high)
        self.o.load(tensors[p + "o"])
        self.decay_bias = self._gain(tensors[p + "a2.b"])
        self.gain = self._gain(tensors[p + "norm"].to(torch.float32).repeat(s.heads))

    def cache_need(self):
        s = self.spec
        return StateNeed((s.heads * s.value_dim * s.head_dim,), torch.float32)

    def forward(self, x, batch, cache):
        y = torch.empty((x.shape[0], self.inner), dtype=x.dtype, device=x.device)
        self.mix(self.proj(x), batch, cache, y)
        return self.o(y, keep_partials=True)

    def mix(self, proj, batch, cache, out, out_scale: float = 1.0):
        """From the projected rows (`proj`, maybe a block of columns of wider rows) to what the output projection reads, times
        `out_scale`, written to `out` [n, heads value_dim] (likewise)."""
        s = self.spec
        n = proj.shape[0]
        qk, inner = self.qk, self.inner
        z = self.a2(proj[:, self.low_at:self.low_at + self.rank], out_dtype=torch.float32)
        S = cache.state.unflatten(1, (s.heads, s.value_dim, s.head_dim))
        o = torch.empty((n, inner), dtype=torch.float32, device=proj.device)
        segments.matrix_state_scan("channel_gate", proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + inner], S, o, batch,
                                   s.heads, s.head_dim, s.value_dim, log_decay=z, decay_bias=self.decay_bias, rate=1.0 / s.tau,
                                   q_scale=float(s.head_dim) ** -0.5)
        kernels.gated_group_rmsnorm(o, proj[:, 2 * qk + inner:2 * qk + 2 * inner], self.gain, s.norm_eps, out, s.heads, gate="silu",
                                    out_scale=out_scale)


register_part("mixer", "gated_linear_attention", GatedLinearAttention)
