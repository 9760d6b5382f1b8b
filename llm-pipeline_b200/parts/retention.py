"""Retention: linear attention whose state forgets by one constant per head (``retention``).

With h the mixer's input, H heads with queries and keys of ``dim`` entries and values of ``vdim``, and a decay a_h per head::

    q, k, v, z = Wq h, Wk h, Wv h, Wg h
    q, k <- the first ``rotary_dim`` entries of every head turned by the token's position (half-split pairs);  k <- k dim^(-1/2)
    S_t = a_h S_(t-1) + k_t v_t^T   (S is dim x vdim, zero before the first token),   o_t = S_t^T q_t
    o <- o / sqrt(mean(o^2) + eps)  per head;   out = Wo (o * silu(z))

There is no softmax and no denominator. The four products that read h are one product against [Wq; Wk; Wv; Wg] with a float32
result; rotation, decay, state, read-out, norm and gate are float32 (``csrc/retention.cu``, ``csrc/state_space.cu``: the
recurrence is the state-space one with a constant decay, a step size of one and a group per head); in bfloat16, requests of many
tokens run in chunks on the tensor cores with the rotated q, k and the v rounded to bfloat16 (``csrc/chunked_scan.cu``); the gated rows are rounded
once to the compute type for the output product, whose result is float32 again.

State of a request: one float32 vector with two copies of [H, dim, vdim] that take turns by the parity of the last position
written (see ``state_space.py``)."""

from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

from ..cache.spec import StateSpec
from ..ops import kernels
from ..ops.linear import linear
from ..weights.source import ParamSpec
from .base import LayerCache, Mixer, TensorGetter
from .registry import register_mixer
from .state_space import chunk_plan


@register_mixer("retention")
class Retention(Mixer):
    graph_safe = True

    def __init__(self, prefix: str, hidden_size: int, heads: int, dim: int, vdim: int, decay: Sequence[float], eps: float,
                 position: Optional[str] = None, rotary_dim: int = 0, names: Optional[Dict[str, str]] = None):
        """``decay``: one constant per head; ``names``: the tensors' names below ``prefix`` where they differ from ``q``, ``k``,
        ``v``, ``g``, ``o``."""
        self.prefix, self.hidden_size, self.heads, self.dim, self.vdim = prefix, int(hidden_size), int(heads), int(dim), int(vdim)
        self.decay, self.eps = [float(a) for a in decay], float(eps)
        if self.heads <= 0 or self.dim <= 0 or self.vdim <= 0 or len(self.decay) != self.heads:
            raise ValueError(f"retention with {heads} heads of {dim} and {vdim} needs as many decays, got {len(self.decay)}")
        if not all(0.0 <= a <= 1.0 for a in self.decay):
            raise ValueError(f"decays lie between 0 and 1, got {self.decay}")
        self.position, self.rotary_dim = position, int(rotary_dim) if position else 0
        if self.rotary_dim < 0 or self.rotary_dim > self.dim or self.rotary_dim % 2:
            raise ValueError(f"{self.rotary_dim} rotated entries do not fit heads of {self.dim}")
        self.qk_size, self.v_size = self.heads * self.dim, self.heads * self.vdim
        self.names = {n: n for n in ("q", "k", "v", "g", "o")}
        self.names.update(names or {})
        self.w_in = self.w_out = self.decays = self.log_decay = None

    def state_entries(self) -> int:
        return 2 * self.heads * self.dim * self.vdim

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.state_entries(),), torch.float32)

    def graph_key_group(self):
        return "retention"                    # launches of a step of single tokens depend on the number of requests alone

    def _name(self, key: str) -> str:
        return f"{self.prefix}.{self.names[key]}"

    def param_specs(self) -> Dict[str, ParamSpec]:
        D = self.hidden_size
        return {self._name("q"): ParamSpec((self.qk_size, D)), self._name("k"): ParamSpec((self.qk_size, D)),
                self._name("v"): ParamSpec((self.v_size, D)), self._name("g"): ParamSpec((self.v_size, D)),
                self._name("o"): ParamSpec((D, self.v_size))}

    def load(self, get: TensorGetter) -> None:
        self.w_in = torch.cat([get(self._name(n), "matrix") for n in ("q", "k", "v", "g")], dim=0).contiguous()
        self.w_out = get(self._name("o"), "matrix").contiguous()
        exact = torch.tensor(self.decay, dtype=torch.float64)
        high = exact.float()
        self.decays = torch.stack([high, (exact - high.double()).float()]).contiguous().to(self.w_out.device)
        # a decay of zero: finite, and so far down that a token later nothing is left
        self.log_decay = torch.log(exact).clamp(min=-1e30).float().to(self.w_out.device)

    def forward(self, x, ctx, cache: LayerCache):
        return self.forward_from(linear(x, self.w_in, out_dtype=torch.float32), ctx, cache)         # [N, q | k | v | gate]

    def forward_from(self, proj, ctx, cache: LayerCache):
        if cache.state is None:
            raise RuntimeError("the retention mixer needs its state slots")
        N, Q, V = ctx.num_tokens, self.qk_size, self.v_size
        cos, sin = ctx.position_tables[self.position] if self.rotary_dim else (None, None)
        gate = proj[:, 2 * Q + V:]
        gated = torch.empty((N, V), dtype=ctx.dtype, device=proj.device)
        if ctx.max_q_len == 1 and kernels.state_step_supports(cache.state, 0, self.dim, self.vdim):
            # one token a request: rotation, state, norm and gate in one kernel
            kernels.retention_step(proj[:, :Q], proj[:, Q:2 * Q], proj[:, 2 * Q:2 * Q + V], gate, cos, sin, self.rotary_dim, self.dim ** -0.5,
                                   self.decays, self.eps, cache.state, 0, ctx.slots, ctx.positions, gated, self.heads, self.dim, self.vdim)
            return linear(gated, self.w_out, out_dtype=torch.float32), None
        plan = None
        if kernels.chunked_scan_supports(ctx.dtype, self.dim, self.vdim, 0, cache.state.stride(0)) and cache.state.data_ptr() % 16 == 0:
            plan = chunk_plan(ctx)
        rows = torch.empty((N, 2 * Q + V), dtype=ctx.dtype, device=proj.device) if plan is not None else None
        single = plan is None or not plan[2]                                # requests whose tokens are walked one by one
        kernels.rotate_heads(proj[:, :2 * Q + V] if plan is not None else proj[:, :2 * Q], cos, sin, self.rotary_dim, 2 * self.heads, self.heads,
                             self.dim, self.dim ** -0.5, typed=rows, in_place=single)
        o = torch.empty((N, V), dtype=torch.float32, device=proj.device)
        if plan is not None:
            kernels.chunked_scan(rows[:, Q:2 * Q], rows[:, :Q], rows[:, 2 * Q:], cache.state, 0, ctx.q_start, ctx.slots, ctx.positions, plan[0], plan[1],
                                 o, self.heads, self.heads, self.dim, self.vdim, log_decay=self.log_decay)
        if single:
            kernels.retention_scan(proj[:, :Q], proj[:, Q:2 * Q], proj[:, 2 * Q:2 * Q + V], self.decays, cache.state, 0, ctx.q_start, ctx.slots,
                                   ctx.positions, o, self.heads, self.dim, self.vdim,
                                   max_tokens=kernels.CHUNKED_SCAN_MIN_TOKENS - 1 if plan is not None else None)
        kernels.gated_group_norm(o, gate, None, gated, self.vdim, self.eps, gate_first=False)
        return linear(gated, self.w_out, out_dtype=torch.float32), None
