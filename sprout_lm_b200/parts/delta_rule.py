"""A recurrence that corrects itself (the gated delta rule): a float32 state per request and head, no keys or values per token.

q = W_q h and k = W_k h (kv_heads x dim), v = W_v h (heads x value_dim); each passes a causal convolution per channel
(``taps`` taps, no bias, zeros before the start of the sequence) and silu; q and k are then divided per head by
sqrt(sum of squares + 1e-6), q also multiplied by dim^(-1/2).  Head h reads the q and k of head h // (heads // kv_heads).
beta = sigmoid(W_b h) and g = exp(-exp(A_log) softplus(W_a h + dt_bias)), one each per head.  Per head

    S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q

so what is written is the difference between the value and what the decayed state already returns for the key, and the
output sees the token's own write.  Each head's o is divided by its root mean square over value_dim (``eps``), multiplied by
a weight [value_dim] that the heads share and by silu(W_g h) (heads x value_dim), and the heads side by side are projected by
W_o.  ``out_scale`` multiplies the mixer's output (folded into the norm's weight).

The state has two tensors per request: the convolution's last taps - 1 inputs and S [heads, dim, value_dim]; both float32.
Everything from the unit norms to the outputs is float32 in both compute dtypes (``csrc/delta_rule.cu``).
"""
from __future__ import annotations

import torch

from .. import kernels
from .base import Part, StateSpec, StateView, TensorDecl, WeightSource, register_part
from .linear import Linear

UNIT_EPS = 1e-6              # inside the root of the unit norms


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Part):
    DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "g": "g", "b": "b", "a": "a", "a_log": "A_log", "dt_bias": "dt_bias", "norm": "norm",
                     "o": "o", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv"}

    def __init__(self, prefix: str, hidden_size: int, heads: int, kv_heads: int, dim: int, value_dim: int, taps: int, eps: float,
                 out_scale: float = 1.0, names: dict | None = None):
        if hidden_size <= 0 or heads <= 0 or kv_heads <= 0 or heads % kv_heads or value_dim <= 0 or eps <= 0:
            raise ValueError("gated_delta_rule: sizes and eps must be positive, heads a multiple of kv_heads")
        if not 0 < dim <= 256:
            raise ValueError("gated_delta_rule: key vectors of up to 256 elements")
        if taps < 1:
            raise ValueError("gated_delta_rule: the convolution has at least one tap")
        self.hidden_size, self.heads, self.kv_heads, self.dim, self.value_dim = hidden_size, heads, kv_heads, dim, value_dim
        self.taps, self.eps, self.out_scale = taps, float(eps), float(out_scale)
        self.kept_taps = max(2, taps)                   # the kernel's least; a single tap gets a zero before it
        self.channels = 2 * kv_heads * dim + heads * value_dim
        self.names = {key: prefix + value for key, value in {**self.DEFAULT_NAMES, **(names or {})}.items()}
        self.runtime = None

    def cache_spec(self):
        return None

    def state_spec(self):
        return (StateSpec(shape=(self.kept_taps - 1, self.channels), dtype=torch.float32),
                StateSpec(shape=(self.heads, self.dim, self.value_dim), dtype=torch.float32))

    def tensor_decls(self):
        n, qk, vw = self.names, self.kv_heads * self.dim, self.heads * self.value_dim
        return [TensorDecl(n["q"], (qk, self.hidden_size)), TensorDecl(n["k"], (qk, self.hidden_size)),
                TensorDecl(n["v"], (vw, self.hidden_size)), TensorDecl(n["g"], (vw, self.hidden_size)),
                TensorDecl(n["q_conv"], (qk, self.taps), "conv"), TensorDecl(n["k_conv"], (qk, self.taps), "conv"),
                TensorDecl(n["v_conv"], (vw, self.taps), "conv"),
                TensorDecl(n["b"], (self.heads, self.hidden_size)), TensorDecl(n["a"], (self.heads, self.hidden_size)),
                TensorDecl(n["a_log"], (self.heads,), "bias"), TensorDecl(n["dt_bias"], (self.heads,), "bias"),
                TensorDecl(n["norm"], (self.value_dim,), "gain"), TensorDecl(n["o"], (self.hidden_size, vw))]

    def load(self, source: WeightSource):
        n, status = self.names, source.runtime.status
        self.runtime = source.runtime
        # one product for everything that reads h: [q | k | v | g | b | a]
        fused = torch.cat([source.raw(n[key]) for key in ("q", "k", "v", "g", "b", "a")], dim=0)
        self.proj = Linear(source.to_device_matrix(fused), None, status, any_inner_size=True)
        taps = torch.cat([source.vector(n[key]) for key in ("q_conv", "k_conv", "v_conv")], dim=0)
        self.conv = torch.nn.functional.pad(taps, (self.kept_taps - self.taps, 0)).contiguous()
        self.a_log, self.dt_bias = source.vector(n["a_log"]), source.vector(n["dt_bias"])
        self.gain = (source.vector(n["norm"]) * self.out_scale).contiguous()
        self.out = Linear(source.matrix(n["o"]), None, status, any_inner_size=True)

    def forward(self, h, x, ctx, cache, state: StateView):
        """x (float32) += out_scale * W_o (rmsnorm_per_head(o) * w * silu(W_g h)); the requests' states advance."""
        if state is None:
            raise RuntimeError("gated_delta_rule: the layer needs a state slot per request")
        status = self.runtime.status
        rows = self.proj.forward(h)
        qk, vw, heads = self.kv_heads * self.dim, self.heads * self.value_dim, self.heads
        conv = torch.empty((rows.shape[0], self.channels), dtype=rows.dtype, device=rows.device)
        kernels.causal_conv(rows[:, :self.channels], self.conv, None, conv, ctx, state.part(0), status, silu=True)
        at = self.channels + vw
        o = torch.empty((rows.shape[0], vw), dtype=torch.float32, device=rows.device)
        kernels.delta_rule(conv[:, :qk], conv[:, qk:2 * qk], conv[:, 2 * qk:], rows[:, at:at + heads], rows[:, at + heads:at + 2 * heads],
                           self.a_log, self.dt_bias, ctx, state.part(1), o, heads, self.kv_heads, self.dim, self.value_dim, status,
                           q_scale=self.dim ** -0.5, unit_eps=UNIT_EPS)
        gated = torch.empty((rows.shape[0], vw), dtype=rows.dtype, device=rows.device)
        kernels.gated_group_norm(o, rows[:, self.channels:at], self.gain, gated, self.eps, groups=heads, gate_first=False, silu=True)
        self.out.forward(gated, residual=x)
