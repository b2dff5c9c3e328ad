"""Attention through a latent: queries, keys and values are projected down to a narrow latent
first, and only the keys' and values' common latent is cached.

With H heads, per head ``dim`` unrotated and ``rot_dim`` rotated query/key dimensions, value size
``vdim`` and latent width ``kv_rank``:

    c_q = rms(W_dq h) * w_qn          q = W_uq c_q, head by head [dim | rot_dim]
    [c_raw | k_rot_raw] = W_dkv h     c = rms(c_raw) * w_kvn,  k_rot = rotate(k_rot_raw)   (one for all heads)
    k_h = W_uk[h] c,  v_h = W_uv[h] c
    s = (q_plain_h . k_h + rotate(q_rot_h) . k_rot) * scale      over positions j <= i
    p = softmax with exp(sink_h) added to the denominator (a learned number per head)
    out = W_o ( concat_h(sum_j p_j v_h,j) * sigmoid(W_g h) )

The cache keeps one row ``[c | k_rot]`` per token (`CacheSpec` with `row_width`).  The kernels
never materialise k_h or v_h: the key projection is folded into the query
(``q_abs_h = W_uk[h]^T q_plain_h``, so ``q_plain_h . k_h = q_abs_h . c``) and the value projection
is applied after the weighted sum (``sum_j p_j v_h,j = W_uv[h] sum_j p_j c_j``), which is the same
arithmetic regrouped.  Portions of few rows and decoded tokens run this form.  For a portion of many rows it
costs several times the arithmetic of plain attention (every score is as wide as the latent); without a rotated
part and a sink, and with sizes the tcgen05 kernel takes, such a portion gathers its cached latents, expands
them into keys and values by one product and runs that kernel over them.
Norms, rotation angles, scores and softmax are 32-bit in both modes.

Variants by parameter: `q_rank` None - the queries are one product of the layer's input, ``q = W_q h``, without
a latent of their own; `rot_dim` 0 - no rotated part; `sink` false - the plain softmax; `gate_per_head` - the
output gate is one number a head, ``sigmoid(W_g h)_head``.

The projections that read the layer's input (W_dq or W_q, W_dkv, W_g) are one matrix, fused at load.
"""

from __future__ import annotations

from typing import List, Optional

import torch

from .. import kernels
from ..config.model_config import PartSpec
from ..registry import build_part, register_part
from .base import CacheSpec, CacheView, Fetch, Mixer, StepContext, TensorSpec


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    graph_safe = True

    DEFAULT_NAMES = (("q", "q"), ("dq", "dq"), ("dq_norm", "dq.norm"), ("uq", "uq"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"),
                     ("uk", "uk"), ("uv", "uv"), ("sink", "sink"), ("gate", "g"), ("out", "o"))

    def __init__(self, hidden_size: int, heads: int, dim: int, rot_dim: int, value_dim: int, kv_rank: int,
                 q_rank: Optional[int], scale: float, eps: float, position: PartSpec, prefix: str, sink: bool = True,
                 output_gate: bool = True, window: Optional[int] = None, tensor_names=None, gate_per_head: bool = False):
        self.hidden_size, self.heads, self.dim, self.rot_dim = int(hidden_size), int(heads), int(dim), int(rot_dim)
        self.value_dim, self.kv_rank = int(value_dim), int(kv_rank)
        self.q_rank = int(q_rank) if q_rank else None
        self.gate_per_head = bool(gate_per_head)
        self.scale, self.eps, self.prefix = float(scale), float(eps), prefix
        self.has_sink, self.has_gate, self.window = bool(sink), bool(output_gate), window
        if not 1 <= self.kv_rank <= kernels.LATENT_MAX_RANK:
            raise ValueError(f"kv_rank {self.kv_rank} outside 1..{kernels.LATENT_MAX_RANK}")
        self.position = build_part("position", position)
        self.q_head = self.dim + self.rot_dim
        self.names = dict(self.DEFAULT_NAMES)
        self.names.update(dict(tensor_names or ()))
        self.w_in = self.w_uq = self.w_uk = self.w_uv = self.w_o = None
        self.q_norm = self.kv_norm = self.sink = None

    def _n(self, what: str) -> str:
        return self.prefix + self.names[what]

    # ---- weights ----------------------------------------------------------------------
    def tensor_specs(self) -> List[TensorSpec]:
        W, H = self.hidden_size, self.heads
        if self.q_rank:
            specs = [TensorSpec(self._n("dq"), (self.q_rank, W)),
                     TensorSpec(self._n("dq_norm"), (self.q_rank,), role="vector", init="norm"),
                     TensorSpec(self._n("uq"), (H * self.q_head, self.q_rank))]
        else:
            specs = [TensorSpec(self._n("q"), (H * self.q_head, W))]
        specs += [TensorSpec(self._n("dkv"), (self.kv_rank + self.rot_dim, W)),
                 TensorSpec(self._n("dkv_norm"), (self.kv_rank,), role="vector", init="norm"),
                 TensorSpec(self._n("uk"), (H * self.dim, self.kv_rank)),
                 TensorSpec(self._n("uv"), (H * self.value_dim, self.kv_rank)),
                 TensorSpec(self._n("out"), (W, H * self.value_dim))]
        if self.has_sink:
            specs.append(TensorSpec(self._n("sink"), (H,), role="vector"))
        if self.has_gate:
            specs.append(TensorSpec(self._n("gate"), (H if self.gate_per_head else H * self.value_dim, W)))
        return specs

    def load(self, fetch: Fetch) -> None:
        H = self.heads
        parts = [fetch(self._n("dq" if self.q_rank else "q")), fetch(self._n("dkv"))]
        if self.has_gate:
            parts.append(fetch(self._n("gate")))
        rows = sum(p.shape[0] for p in parts)
        if rows % 8:                            # rows of the product stay 16-byte aligned
            parts.append(parts[0].new_zeros((8 - rows % 8, self.hidden_size)))
        self.w_in = torch.cat(parts, dim=0).contiguous()            # rows: [c_q or q | c, k_rot | gate]
        self.w_uq = fetch(self._n("uq")) if self.q_rank else None
        self.w_o = fetch(self._n("out"))
        # one matrix, keys of all heads and then values, for expanding; its parts for the folded form
        self.w_kv = torch.cat([fetch(self._n("uk")), fetch(self._n("uv"))], dim=0).contiguous()
        self.w_uk = self.w_kv[:H * self.dim].view(H, self.dim, self.kv_rank)                               # q_plain_h @ W_uk[h]
        self.w_uv = self.w_kv[H * self.dim:].view(H, self.value_dim, self.kv_rank).transpose(1, 2)          # o_h @ W_uv[h]^T
        self.q_norm = fetch(self._n("dq_norm")) if self.q_rank else None
        self.kv_norm = fetch(self._n("dkv_norm"))
        self.sink = fetch(self._n("sink")) if self.has_sink else None

    def weight_bytes(self) -> int:
        el = self.w_in.element_size()
        n = sum(t.numel() for t in (self.w_in, self.w_uq, self.w_uk, self.w_uv, self.w_o) if t is not None) * el
        return n + 4 * ((self.q_rank or 0) + self.kv_rank + (self.heads if self.has_sink else 0))

    # ---- cache ------------------------------------------------------------------------
    def cache_spec(self) -> CacheSpec:
        return CacheSpec("window" if self.window else "full", window=self.window,
                         row_width=self.kv_rank + self.rot_dim)

    # ---- forward ----------------------------------------------------------------------
    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[CacheView],
                state: Optional[torch.Tensor]) -> torch.Tensor:
        assert cache is not None, "latent attention needs a cache slot"
        H, R, Dr, T = self.heads, self.kv_rank, self.rot_dim, x.shape[0]
        proj = kernels.linear(x, self.w_in)                                   # [T, c_q or q | R + Dr | gate]
        if self.q_rank:
            q_cols = self.q_rank
            cq = kernels.rms_norm_slice(proj, 0, self.q_rank, self.q_norm, self.eps)
            q = kernels.linear(cq, self.w_uq)                                 # [T, H * (dim + rot_dim)]
        else:
            q_cols = H * self.q_head
            q = proj                                                          # its first columns are the queries
        table = self.position.rotary_table(x.device)        # None: nothing is turned
        inv_freq, rot = table if table is not None else (None, 0)
        if rot:
            kernels.rope_head_slices(q, H, self.q_head, self.dim, rot, inv_freq, ctx.positions)
        if cache.append:
            kernels.latent_append(proj, q_cols, R, Dr, self.kv_norm, self.eps, inv_freq, rot, ctx,
                                  cache.pages, cache.block_table, cache.page_size)
        if (not Dr and not self.has_sink and not self.window and not (self.has_gate and not self.gate_per_head)
                and kernels.can_expand_latent(q, H, self.dim, self.value_dim, R, ctx)):
            return self._forward_expanded(q, proj, q_cols + R, ctx, cache)
        o = self._folded(q, proj, q_cols + R + Dr, ctx, cache.pages, cache.block_table, cache.page_size)
        return kernels.linear(o, self.w_o)

    def _forward_expanded(self, q, proj, gate_col0: int, ctx: StepContext, cache: CacheView) -> torch.Tensor:
        """The segments of several rows over expanded keys and values, those of one row in the folded form."""
        H = self.heads
        o = torch.empty((q.shape[0], H * self.value_dim), dtype=q.dtype, device=q.device)
        kernels.expanded_latent_attention(q, self.w_kv, H, self.dim, cache.pages, cache.block_table, cache.page_size, ctx,
                                          self.scale, o, proj if self.has_gate else None, gate_col0)
        sub = ctx.single_rows_context()
        if sub is not None:
            rows, _ = ctx.single_rows()
            own = proj is q
            q_s = q.index_select(0, rows)
            proj_s = q_s if own else proj.index_select(0, rows)
            table = cache.block_table.index_select(0, sub.scratch["segments"])
            o.index_copy_(0, rows.long(), self._folded(q_s, proj_s, gate_col0, sub, cache.pages, table, cache.page_size))
        return kernels.linear(o, self.w_o)

    def _folded(self, q, proj, gate_col0: int, ctx: StepContext, pages, block_table, page_size: int) -> torch.Tensor:
        """Gated outputs [T, H * vdim] with the key projection folded into the query and the value projection
        applied after the weighted sum."""
        H, T = self.heads, q.shape[0]
        # the key projection folded into the query: [H, T, dim] x [H, dim, R]
        q_heads = q[:, :H * self.q_head].unflatten(1, (H, self.q_head))
        q_abs = kernels.heads_linear(q_heads[:, :, :self.dim].transpose(0, 1), self.w_uk)
        o_lat = kernels.latent_attention(q_abs, q, self.q_head, self.dim, self.rot_dim, pages, block_table, page_size, ctx,
                                         self.sink, self.scale, self.window or 0)
        v = kernels.heads_linear(o_lat, self.w_uv)                            # [H, T, vdim]
        if self.has_gate:
            return kernels.heads_sigmoid_gate(v, proj, gate_col0, per_head=self.gate_per_head)
        return v.transpose(0, 1).reshape(T, H * self.value_dim)
