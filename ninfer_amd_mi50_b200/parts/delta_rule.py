"""The gated delta rule: a recurrence that corrects what its state would answer, with its state in the request's slot.

Per head, with q_t, k_t of size D (several heads may share them), v_t of size V and the layer's input x_t:

    q, k, v = silu(conv(W_q x)), silu(conv(W_k x)), silu(conv(W_v x))     a short causal convolution per channel
    q_t <- q_t / sqrt(sum(q_t^2) + 1e-6) * scale,   k_t <- k_t / sqrt(sum(k_t^2) + 1e-6)      scale: D^-1/2
    g_t = exp(-exp(A_log) softplus(w_a . x + dt_bias)),   beta_t = sigmoid(w_b . x)
    S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t          S is D x V

Each head's o over its own root mean square, times a weight of size V that the heads share, times
``silu(W_g x)``; out-projection.

What a request keeps between steps is of fixed size: the convolutions' last ``taps - 1`` inputs and S of
every head, float32, side by side in one slot (`state_spec`), so prompts cut into portions, decoded tokens
and mixed batches continue from the slot and leave it updated (``csrc/ssm.cu`` for the convolution,
``csrc/delta_rule.cu`` for the rest).  Unit norms, decays, step sizes, S and the sums are 32-bit in both
modes; the projections, the convolutions' outputs and the gate are in the engine's type.  The projections
that read x are one matrix, fused at load: ``[q | k | v | gate | a | b]``, padded with rows of zeros to a
multiple of 8.
"""

from __future__ import annotations

from typing import List, Optional

import torch

from .. import kernels
from ..registry import register_part
from .base import CacheView, Fetch, Mixer, StateSpec, StepContext, TensorSpec


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    graph_safe = True

    DEFAULT_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("q_conv", "q.conv"), ("k_conv", "k.conv"), ("v_conv", "v.conv"),
                     ("gate", "g"), ("a", "a"), ("b", "b"), ("A_log", "A_log"), ("dt_bias", "dt_bias"), ("norm", "norm"),
                     ("out", "o"))

    def __init__(self, hidden_size: int, heads: int, kv_heads: int, dim: int, value_dim: int, conv_taps: int, eps: float,
                 prefix: str, query_scale: Optional[float] = None, tensor_names=None):
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.dim, self.value_dim, self.taps = int(dim), int(value_dim), int(conv_taps)
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads do not share {self.kv_heads} query/key heads evenly")
        if not 1 <= self.dim <= kernels.DELTA_RULE_MAX_DIM:
            raise ValueError(f"dim {self.dim} outside 1..{kernels.DELTA_RULE_MAX_DIM}")
        if not 1 <= self.taps <= kernels.CONV_MAX_TAPS:
            raise ValueError(f"conv taps {self.taps} outside 1..{kernels.CONV_MAX_TAPS}")
        self.eps, self.prefix = float(eps), prefix
        self.query_scale = self.dim ** -0.5 if query_scale is None else float(query_scale)
        self.qk_width, self.v_width = self.kv_heads * self.dim, self.heads * self.value_dim
        self.conv_channels = 2 * self.qk_width + self.v_width
        # S starts on 16 bytes behind the convolution's inputs
        self.state_off = ((self.taps - 1) * self.conv_channels + 3) // 4 * 4
        self.names = dict(self.DEFAULT_NAMES)
        self.names.update(dict(tensor_names or ()))
        self.w_in = self.w_o = self.conv_w = self.A_log = self.dt_bias = self.norm_w = None

    def _n(self, what: str) -> str:
        return self.prefix + self.names[what]

    # ---- weights ----------------------------------------------------------------------
    def _projections(self):
        return (("q", self.qk_width), ("k", self.qk_width), ("v", self.v_width), ("gate", self.v_width), ("a", self.heads),
                ("b", self.heads))

    def tensor_specs(self) -> List[TensorSpec]:
        W, H = self.hidden_size, self.heads
        specs = [TensorSpec(self._n(n), (width, W)) for n, width in self._projections()]
        specs += [TensorSpec(self._n(n + "_conv"), (width, self.taps), role="vector") for n, width in self._projections()[:3]]
        return specs + [TensorSpec(self._n("A_log"), (H,), role="vector"), TensorSpec(self._n("dt_bias"), (H,), role="vector"),
                        TensorSpec(self._n("norm"), (self.value_dim,), role="vector", init="norm"),
                        TensorSpec(self._n("out"), (W, self.v_width))]

    def load(self, fetch: Fetch) -> None:
        rows = [fetch(self._n(n)) for n, _ in self._projections()]
        pad = -sum(r.shape[0] for r in rows) % 8
        if pad:
            rows.append(rows[0].new_zeros((pad, self.hidden_size)))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = fetch(self._n("out"))
        # the checkpoint's taps are [channels, taps]; the kernel reads them tap-major
        self.conv_w = torch.cat([fetch(self._n(n + "_conv")) for n in ("q", "k", "v")], dim=0).t().contiguous()
        self.A_log, self.dt_bias = fetch(self._n("A_log")).contiguous(), fetch(self._n("dt_bias")).contiguous()
        self.norm_w = fetch(self._n("norm")).repeat(self.heads)             # the heads share it

    def weight_bytes(self) -> int:
        n = (self.w_in.numel() + self.w_o.numel()) * self.w_in.element_size()
        return n + 4 * (self.conv_w.numel() + 2 * self.heads + self.value_dim)

    def state_spec(self) -> StateSpec:
        """[conv inputs: (taps - 1) x channels, padded | S: heads x value column x dim], float32."""
        return StateSpec((self.state_off + self.heads * self.value_dim * self.dim,), torch.float32)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[CacheView],
                state: Optional[torch.Tensor]) -> torch.Tensor:
        assert state is not None, "the delta rule needs a state slot"
        Q, C = self.qk_width, self.conv_channels
        proj = kernels.linear(x, self.w_in)                                    # [T, q | k | v | gate | a | b]
        qkv = kernels.causal_conv_silu(proj, 0, C, self.conv_w, None, state, ctx)
        a0 = C + self.v_width
        o = kernels.delta_rule(qkv, 0, Q, 2 * Q, proj, a0, a0 + self.heads, self.dt_bias, self.A_log, self.query_scale, state,
                               self.state_off, ctx, self.heads, self.kv_heads, self.dim, self.value_dim)
        g = kernels.group_rmsnorm_gate(o, proj, C, self.norm_w, self.eps, self.heads, kernels.GATE_SILU, x.dtype)
        return kernels.linear(g, self.w_o)
