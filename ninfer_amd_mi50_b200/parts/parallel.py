"""Several mixers side by side on the same input.

`parallel_mean`: the mean of their outputs, each first over its own root mean square and times its own weight,

    out = (1 / n) * sum_m (y_m / rms(y_m)) * w_m,      y_m = mixer_m(x)

as float32 (a norm reads it next).  `parallel_scaled`: two mixers, their outputs added with fixed factors, which is
left to whoever reads them (`ScaledPair`).

At most one of the mixers may keep pages and at most one a fixed-size state: the layer's cache
slot and state slot go to those.
"""

from __future__ import annotations

from typing import List, Optional, Sequence, Tuple

import torch

from .. import kernels
from ..config.model_config import PartSpec
from ..registry import build_part, register_part
from .base import BiasedOutput, CacheSpec, CacheView, Fetch, Mixer, ScaledPair, StateSpec, StepContext, TensorSpec, summed


class SideBySide(Mixer):
    """What mixers on one input have in common: each one's tensors lie below ``prefix + name + "."``."""

    def _take(self, prefix: str, branches: Sequence[Tuple[str, PartSpec]]) -> None:
        self.prefix = prefix
        self.branch_names = [n for n, _ in branches]
        self.mixers: List[Mixer] = [build_part("mixer", spec, prefix=f"{prefix}{n}.") for n, spec in branches]
        if sum(m.cache_spec() is not None for m in self.mixers) > 1 or sum(m.state_spec() is not None for m in self.mixers) > 1:
            raise ValueError("at most one mixer with pages and one with a state may stand side by side")

    @property
    def graph_safe(self) -> bool:
        return all(m.graph_safe for m in self.mixers)

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for m in self.mixers for s in m.tensor_specs()]

    def load(self, fetch: Fetch) -> None:
        for m in self.mixers:
            m.load(fetch)

    def weight_bytes(self) -> int:
        return sum(m.weight_bytes() for m in self.mixers)

    def check_limits(self, dtype, max_context, page_size) -> None:
        for m in self.mixers:
            m.check_limits(dtype, max_context, page_size)

    def cache_spec(self) -> Optional[CacheSpec]:
        return next((s for s in (m.cache_spec() for m in self.mixers) if s is not None), None)

    def state_spec(self) -> Optional[StateSpec]:
        return next((s for s in (m.state_spec() for m in self.mixers) if s is not None), None)

    def _run(self, m: Mixer, x: torch.Tensor, ctx: StepContext, cache, state):
        return m.forward(x, ctx, cache if m.cache_spec() is not None else None, state if m.state_spec() is not None else None)


@register_part("mixer", "parallel_mean")
class ParallelMean(SideBySide):
    def __init__(self, hidden_size: int, eps: float, prefix: str, branches: Sequence[Tuple[str, PartSpec]],
                 weight_suffix: str = "out"):
        """`branches`: (name, mixer spec) pairs; branch `name`'s weight is ``prefix + name + "." + weight_suffix``."""
        if not 1 <= len(branches) <= 4:
            raise ValueError("one to four mixers side by side")
        self.hidden_size, self.eps = int(hidden_size), float(eps)
        self._take(prefix, branches)
        self.weight_names = [f"{prefix}{n}.{weight_suffix}" for n in self.branch_names]
        self.weights: List[torch.Tensor] = []

    def tensor_specs(self) -> List[TensorSpec]:
        return super().tensor_specs() + [TensorSpec(n, (self.hidden_size,), role="vector", init="norm") for n in self.weight_names]

    def load(self, fetch: Fetch) -> None:
        super().load(fetch)
        self.weights = [fetch(n) for n in self.weight_names]

    def weight_bytes(self) -> int:
        return super().weight_bytes() + 4 * self.hidden_size * len(self.mixers)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[CacheView],
                state: Optional[torch.Tensor]) -> torch.Tensor:
        return kernels.mean_of_rmsnorms([self._run(m, x, ctx, cache, state) for m in self.mixers], self.weights, self.eps)


@register_part("mixer", "parallel_scaled")
class ParallelScaled(SideBySide):
    """``scale_a * mixer_a(x) + scale_b * mixer_b(x)``.  In small steps, whose kernels do not fill the device, the second
    mixer runs beside the first on a second stream (a parallel branch of a captured graph)."""

    # steps of up to this many rows run the second mixer on the second stream; 0: never
    fork_max_rows = 64

    def __init__(self, prefix: str, branches: Sequence[Tuple[str, PartSpec]], scales: Sequence[float]):
        if len(branches) != 2 or len(scales) != 2:
            raise ValueError("two mixers side by side, a factor each")
        self.scales = (float(scales[0]), float(scales[1]))
        self._take(prefix, branches)
        self._bias = None

    def load(self, fetch: Fetch) -> None:
        super().load(fetch)
        self._bias = None

    def _pair(self, a, b) -> ScaledPair:
        """Both outputs with their factors; projection biases that were left pending become one vector, once."""
        if self._bias is None:
            parts = [y.bias * s for y, s in ((a, self.scales[0]), (b, self.scales[1])) if isinstance(y, BiasedOutput)]
            self._bias = sum(parts[1:], parts[0]).contiguous() if parts else None
        a, b = (y.y if isinstance(y, BiasedOutput) else summed(y) for y in (a, b))
        return ScaledPair(a, self.scales[0], b, self.scales[1], self._bias)

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: Optional[CacheView],
                state: Optional[torch.Tensor]) -> ScaledPair:
        from .feedforward import _side_stream
        first, second = self.mixers
        if not (x.is_cuda and x.shape[0] <= self.fork_max_rows):
            a = self._run(first, x, ctx, cache, state)
            return self._pair(a, self._run(second, x, ctx, cache, state))
        main, side = torch.cuda.current_stream(x.device), _side_stream(x.device)
        side.wait_stream(main)
        with torch.cuda.stream(side):
            kernels.chain_break()               # its input comes from the other stream
            b = self._run(second, x, ctx, cache, state)
        a = self._run(first, x, ctx, cache, state)
        main.wait_stream(side)
        kernels.chain_break()                   # the kernel that adds both up also reads what the other stream produced
        return self._pair(a, b)
