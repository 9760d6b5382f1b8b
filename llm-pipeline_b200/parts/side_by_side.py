"""Two mixers side by side: both read the same input, and the result is a weighted sum of theirs.

``side_by_side`` builds its two members from part specifications (kind, sizes, tensor-name prefix below its own), so
any two registered mixers can stand beside each other. What they ask of the cache manager is put together: at most one
member may keep pages (the layer has one page group), and the members' states lie one after the other in the request's
state vector, each member seeing its own column range. The sum ``left_scale * left + right_scale * right`` is float32. With
``out_norm_eps`` each member's result first passes an RMS norm over its row with a weight of its own (``out_norms``: the two
names). Where both members read their input through one product each and can go on from its rows (``Mixer.forward_from``), the
two products are one. A block that takes addends gets both results with their norms and leaves the work to the kernel that adds them."""

from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch

from ..cache.spec import StateSpec
from ..ops import kernels
from ..ops.linear import linear
from ..weights.source import ParamSpec
from .base import Addend, LayerCache, Mixer, TensorGetter
from .registry import lookup, register_mixer


@register_mixer("side_by_side")
class SideBySide(Mixer):
    def __init__(self, prefix: str, left: Dict[str, Any], right: Dict[str, Any], left_scale: float = 1.0, right_scale: float = 1.0,
                 out_norm_eps: Optional[float] = None, out_norms: Sequence[str] = (), hidden_size: int = 0):
        """``left`` / ``right``: {"kind": a registered mixer, "args": its sizes, "prefix": its tensors' prefix below this one's}. ``out_norms``: the full names of
        the norms' weights, of ``hidden_size`` entries."""
        self.prefix = prefix
        self.scales = (float(left_scale), float(right_scale))
        self.members = tuple(lookup("mixer", m["kind"])(f"{prefix}.{m['prefix']}" if m.get("prefix") else prefix, **m["args"])
                             for m in (left, right))
        if sum(m.cache_spec() is not None for m in self.members) > 1:
            raise ValueError("mixers side by side share one page group: only one of them may keep pages")
        self.graph_safe = all(getattr(m, "graph_safe", False) for m in self.members)
        self._state_at = []
        at = 0
        for m in self.members:
            spec = m.state_spec()
            if spec is None:
                self._state_at.append(None)
                continue
            if spec.dtype != torch.float32 or len(spec.shape) != 1:
                raise ValueError("mixers side by side keep their states as float32 vectors")
            self._state_at.append((at, at + spec.shape[0]))
            at += spec.shape[0]
        self._state_entries = at
        self.out_norm_eps = None if out_norm_eps is None else float(out_norm_eps)
        self.out_norms, self.hidden_size = tuple(out_norms), int(hidden_size)
        if (self.out_norm_eps is not None) != (len(self.out_norms) == 2 and self.hidden_size > 0):
            raise ValueError("norms on the members' results need an eps, two weights' names and the row's size")
        self.norm_weights: Optional[List[torch.Tensor]] = None
        self.w_in: Optional[torch.Tensor] = None

    def cache_spec(self):
        for m in self.members:
            if m.cache_spec() is not None:
                return m.cache_spec()
        return None

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self._state_entries,), torch.float32) if self._state_entries else None

    def graph_key_group(self):
        return ("side_by_side",) + tuple(m.graph_key_group() for m in self.members)

    def graph_key(self, shape):
        return tuple(m.graph_key(shape) for m in self.members)

    def captured_context_limit(self):
        limits = [n for n in (m.captured_context_limit() for m in self.members) if n is not None]
        return min(limits) if limits else None

    def param_specs(self):
        out = {}
        for m in self.members:
            out.update(m.param_specs())
        out.update({name: ParamSpec((self.hidden_size,), role="vector", init="norm") for name in self.out_norms})
        return out

    def copies(self):
        out = {}
        for m in self.members:
            out.update(m.copies())
        return out

    def load(self, get: TensorGetter) -> None:
        for m in self.members:
            m.load(get)
        if all(hasattr(m, "forward_from") and getattr(m, "w_in", None) is not None for m in self.members):
            self.w_in = torch.cat([m.w_in for m in self.members], dim=0).contiguous()
            at = 0
            for m in self.members:                       # the members' matrices are parts of it now
                m.w_in = self.w_in[at:at + m.w_in.shape[0]]
                at += m.w_in.shape[0]
        if self.out_norms:
            self.norm_weights = [get(name, "vector").float().contiguous() for name in self.out_norms]

    def forward_addends(self, x, ctx, cache: LayerCache) -> List[Addend]:
        rows = self._results(x, ctx, cache)
        if self.norm_weights is None:
            return [Addend(r, factor=s) for r, s in zip(rows, self.scales)]
        return [Addend(r, w, self.out_norm_eps, s) for r, w, s in zip(rows, self.norm_weights, self.scales)]

    def _results(self, x, ctx, cache: LayerCache) -> List[torch.Tensor]:
        results = []
        proj = linear(x, self.w_in, out_dtype=torch.float32) if self.w_in is not None else None
        at = 0
        for m, span in zip(self.members, self._state_at):
            state = cache.state[:, span[0]:span[1]] if span is not None and cache.state is not None else None
            view = LayerCache(pages=cache.pages if m.cache_spec() is not None else None, group=cache.group, state=state,
                              writes=cache.writes)
            if proj is not None:
                out, bias = m.forward_from(proj[:, at:at + m.w_in.shape[0]], ctx, view)
                at += m.w_in.shape[0]
            else:
                out, bias = m.forward(x, ctx, view)
            out = out.float() if out.dtype != torch.float32 else out
            if bias is not None:
                out = out + bias.float()
            results.append(out.contiguous())
        return results

    def forward(self, x, ctx, cache: LayerCache):
        results = self._results(x, ctx, cache)
        if self.norm_weights is not None:
            total = torch.zeros_like(results[0])
            for rows, weight, scale in zip(results, self.norm_weights, self.scales):
                kernels.add_norm_mix(total, delta=rows, delta_weight=weight * scale, delta_eps=self.out_norm_eps)
            return total, None
        total = torch.empty_like(results[0])
        kernels.scaled_sum(results[0], self.scales[0], results[1], self.scales[1], total)
        return total, None
