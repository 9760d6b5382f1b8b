"""A feed-forward of many small experts, of which every token uses a few.

With h the feed-forward's input, E experts with matrices, ``identity`` further router outputs without any, and ``top``
choices per token::

    z = Wr h (+ b)                            router logits, float32; one per expert and identity expert (``router_bias``: b)
    s = sigmoid(z)  or  softmax(z)            ``score``: each logit alone, or over all router outputs
    chosen = the top outputs by s (+ correction, a stored vector, if the router has one)
                                              ``score`` "chosen_softmax": the top outputs by z, s = softmax over those alone
    an expert's weight w is its s (without the correction, not renormalised)
    expert_e(v), ``form`` "clamped": g = min(Wg_e v, limit), u = clamp(Wu_e v, -limit, limit), y = g sigmoid(1.702 g) (u + 1),
                                     Wd_e y, and the weight scales the expert's input: out += expert_e(w h)
                 ``form`` "silu":    Wd_e (silu(Wg_e v) (Wu_e v)), and the weight scales its output: out += w expert_e(h)
                 ``form`` "relu_squared":  Wd_e max(Wu_e v, 0)^2 without a gate, the weight on its output as well
    an identity expert adds w h
    ``groups`` = (n, keep): the router outputs form n equal groups of neighbours; only those of the ``keep`` groups whose best
    entries are the largest can be chosen. ``normalize``: w <- w / (sum of the chosen w + 1e-20); ``factor``: w <- factor w
    ``shared_size``: one more expert of the "silu" form that every token uses, added times sigmoid(w_sg . h), or (without
    ``shared_gate``) as it is

The weight never makes a scaled copy: on the input side ``Wg_e (w h) = w (Wg_e h)`` puts it on the float32 sums of the
first two products, on the output side ``w (Wd_e y) = Wd_e (w y)`` puts it on the float32 activation. Routing happens on
the device (``csrc/routed_experts.cu``): nothing of a step depends on the host seeing the choices, so the part can be
captured in a CUDA graph. The experts' matrices are stacked: ``[E, 2 ff, hidden]`` (gate rows, then up rows; ``[E, ff,
hidden]`` for a form without a gate) and ``[E, hidden, ff]``. The shared expert's gate is one more row of the float32 router matrix; its products are the
engine's ``linear`` and fused gate/up kernels."""

from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..ops import kernels
from ..ops.linear import gate_up_swiglu, linear
from ..weights.source import ParamSpec
from .base import Addend, FeedForward, TensorGetter
from .registry import register_feed_forward


@register_feed_forward("routed_experts")
class RoutedExperts(FeedForward):
    graph_safe = True

    def __init__(self, prefix: str, hidden_size: int, intermediate_size: int, num_experts: int, top: int, limit: float = 0.0,
                 score: str = "sigmoid", form: str = "clamped", identity: int = 0, correction: bool = False,
                 shared_size: Optional[int] = None, router_bias: bool = False, groups: Optional[Tuple[int, int]] = None,
                 normalize: bool = False, factor: float = 1.0, shared_gate: bool = True):
        if not 0 < top <= num_experts + identity:
            raise ValueError(f"a token cannot use {top} of {num_experts + identity} experts")
        if score not in kernels.ROUTER_SCORES:
            raise ValueError(f"router scores are one of {sorted(kernels.ROUTER_SCORES)}, not {score!r}")
        if score == "chosen_softmax" and correction:
            raise ValueError("a softmax over the chosen logits takes them as they are: no correction")
        if form not in kernels.EXPERT_FORMS:
            raise ValueError(f"unknown expert form {form!r}; known: {sorted(kernels.EXPERT_FORMS)}")
        if num_experts < 1 or identity < 0:
            raise ValueError(f"{num_experts} experts and {identity} identity experts")
        self.prefix, self.hidden_size, self.intermediate_size = prefix, int(hidden_size), int(intermediate_size)
        self.num_experts, self.top, self.limit = int(num_experts), int(top), float(limit)
        self.score, self.form, self.identity, self.correction = score, form, int(identity), bool(correction)
        self.shared_size = int(shared_size) if shared_size else None
        self.router_bias, self.gated = bool(router_bias), form not in kernels.UNGATED_EXPERT_FORMS
        self.b_router = None
        self.groups, self.normalize, self.factor = tuple(int(n) for n in groups) if groups else (0, 0), bool(normalize), float(factor)
        self.shared_gate = bool(shared_gate and self.shared_size)
        if groups:
            count, keep = self.groups
            outputs = self.num_experts + self.identity
            if count <= 0 or outputs % count or not 0 < keep <= count or keep * (outputs // count) < self.top:
                raise ValueError(f"{self.top} choices cannot come from {keep} of {count} groups of {outputs} router outputs")
        self.w_router = self.w_gate_up = self.w_down = self.router_correction = self.w_shared_gate_up = self.w_shared_down = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        p, H, I = self.prefix, self.hidden_size, self.intermediate_size
        outputs = self.num_experts + self.identity
        specs = {f"{p}.router": ParamSpec((outputs, H))}
        if self.correction:
            specs[f"{p}.correction"] = ParamSpec((outputs,), role="vector", init="small")
        if self.router_bias:
            specs[f"{p}.router.b"] = ParamSpec((outputs,), role="vector", init="small")
        for e in range(self.num_experts):
            if self.gated:
                specs[f"{p}.e{e}.gate"] = ParamSpec((I, H))
            specs[f"{p}.e{e}.up"] = ParamSpec((I, H))
            specs[f"{p}.e{e}.down"] = ParamSpec((H, I))
        if self.shared_size:
            S = self.shared_size
            specs.update({f"{p}.shared.gate": ParamSpec((S, H)), f"{p}.shared.up": ParamSpec((S, H)),
                          f"{p}.shared.down": ParamSpec((H, S))})
        if self.shared_gate:
            specs[f"{p}.shared.sg"] = ParamSpec((1, H))
        return specs

    def load(self, get: TensorGetter) -> None:
        p = self.prefix
        router = get(f"{p}.router", "matrix").float()                            # the logits are a 32-bit product
        if self.shared_gate:
            router = torch.cat([router, get(f"{p}.shared.sg", "matrix").float().view(1, -1)], dim=0)
        if self.shared_size:
            self.w_shared_gate_up = torch.cat([get(f"{p}.shared.gate", "matrix"), get(f"{p}.shared.up", "matrix")], dim=0).contiguous()
            self.w_shared_down = get(f"{p}.shared.down", "matrix").contiguous()
        self.w_router = router.contiguous()
        if self.correction:
            self.router_correction = get(f"{p}.correction", "vector").float().contiguous()
        if self.router_bias:
            self.b_router = get(f"{p}.router.b", "vector").float().contiguous()
        first = ("gate", "up") if self.gated else ("up",)
        self.w_gate_up = torch.stack([torch.cat([get(f"{p}.e{e}.{n}", "matrix") for n in first], dim=0)
                                      for e in range(self.num_experts)]).contiguous()
        self.w_down = torch.stack([get(f"{p}.e{e}.down", "matrix") for e in range(self.num_experts)]).contiguous()

    def forward(self, x, ctx):
        out, *shared = self.forward_addends(x, ctx)
        if shared:
            out.rows.add_(shared[0].rows)
        return out.rows, None

    def forward_addends(self, x, ctx) -> List[Addend]:
        """The routed experts' sum and, beside it, an ungated shared expert's rows."""
        N = x.shape[0]
        ids = torch.empty((N, self.top), dtype=torch.int32, device=x.device)
        weights = torch.empty((N, self.top), dtype=torch.float32, device=x.device)
        gate = torch.empty((N,), dtype=torch.float32, device=x.device) if self.shared_gate else None
        kernels.route_topk(x, self.w_router, self.top, ids, weights, score=self.score, bias=self.b_router,
                           correction=self.router_correction, gate=gate, groups=self.groups[0], keep=self.groups[1],
                           normalize=self.normalize, factor=self.factor)
        out = torch.empty((N, self.hidden_size), dtype=torch.float32, device=x.device)
        kernels.routed_experts(x, self.w_gate_up, self.w_down, ids, weights, self.limit, out, self.form, self.identity)
        if self.shared_size:
            act = gate_up_swiglu(x, self.w_shared_gate_up)      # the few rows of a decode step: product and activation in one kernel
            if act is None:
                gate_up = linear(x, self.w_shared_gate_up)
                act = torch.empty((N, self.shared_size), dtype=x.dtype, device=x.device)
                kernels.swiglu(gate_up, act)
            shared = linear(act, self.w_shared_down, out_dtype=torch.float32)
            if not self.shared_gate:
                return [Addend(out), Addend(shared)]
            kernels.add_scaled_rows(out, shared, gate)
        return [Addend(out)]
