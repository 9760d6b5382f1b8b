"""Time mixing with a matrix state per head whose rows decay channel by channel (``wkv``).

With h the mixer's input, h' the row of the token before (zeros for the first), H heads of d channels::

    m_s = h + (h' - h) mu_s                                    for s in r, k, v, g, w: five mixes, each with its own vector
    r, k, v = Wr m_r, Wk m_k, Wv m_v;   z = Wg m_g
    w = exp(-exp(W2 tanh(W1 m_w) + w0))                        a decay per head, key channel and token
    o_t = (S + diag(u) k_t v_t^T)^T r_t;   S <- diag(w_t) S + k_t v_t^T        S is d x d, zero before the first token
    o <- o / sqrt(mean(o^2) + eps)  per head;   out = Wo (o * norm * silu(z))

The mixes are formed from the float32 residual and rounded once to the compute type; the products leave float32. The
second step of the decays' projection, decays, bonus, state, read-out, norm and gate are float32 (``csrc/wkv.cu``); the
gated rows are rounded once for the output product. The inner size of the two-step projection is whatever the tensors have.

State of a request: one float32 vector ``[row before | S]``, each piece two copies that take turns by the parity of the last
position written, so that a step of one token never overwrites what it read and a captured decode step can be replayed."""

from __future__ import annotations

from typing import Dict, Optional

import torch

from ..cache.spec import StateSpec
from ..ops import kernels
from ..ops.linear import linear
from ..weights.source import ParamSpec
from .base import LayerCache, Mixer, TensorGetter
from .registry import register_mixer

_MIXES = ("r", "k", "v", "g", "w")


@register_mixer("wkv")
class WKV(Mixer):
    graph_safe = True
    reads_float32 = True                  # the mixes with the row before are formed from the float32 residual

    def __init__(self, prefix: str, hidden_size: int, heads: int, dim: int, eps: float, decay_rank: Optional[int] = None,
                 names: Optional[Dict[str, str]] = None):
        """``decay_rank``: the inner size of the decays' two-step projection (None: the tensors give it); ``names``: the
        tensors' names below ``prefix`` where they differ from the keys used here."""
        self.prefix, self.hidden_size, self.heads, self.dim, self.eps = prefix, int(hidden_size), int(heads), int(dim), float(eps)
        if self.heads <= 0 or not 0 < self.dim <= kernels.WKV_MAX_DIM:
            raise ValueError(f"the wkv kernel takes heads of 1 to {kernels.WKV_MAX_DIM} channels, got {heads} of {dim}")
        self.decay_rank = int(decay_rank) if decay_rank else None
        self.size = self.heads * self.dim
        self.scan_entries = kernels.wkv_state_entries(self.heads, self.dim)
        self.names = {n: n for n in tuple(f"mu.{m}" for m in _MIXES) + ("r", "k", "v", "g", "w1", "w2", "w0", "u", "norm", "o")}
        self.names.update(names or {})
        self.mu = self.w_rkvg = self.w1 = self.w2t = self.w0 = self.bonus = self.norm_w = self.w_out = None

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((2 * self.hidden_size + 2 * self.scan_entries,), torch.float32)

    def graph_key_group(self):
        return "wkv"                      # its launches for a step of single tokens depend on the number of requests alone

    def _name(self, key: str) -> str:
        return f"{self.prefix}.{self.names[key]}"

    def param_specs(self) -> Dict[str, ParamSpec]:
        D, C = self.hidden_size, self.size
        specs = {self._name(f"mu.{m}"): ParamSpec((D,), role="vector", init="unit") for m in _MIXES}
        specs.update({self._name(n): ParamSpec((C, D)) for n in ("r", "k", "v", "g")})
        specs.update({self._name("w1"): ParamSpec((self.decay_rank, D)), self._name("w2"): ParamSpec((C, self.decay_rank)),
                      self._name("w0"): ParamSpec((C,), role="vector", init="small"),
                      self._name("u"): ParamSpec((self.heads, self.dim), role="vector", init="unit"),
                      self._name("norm"): ParamSpec((C,), role="vector", init="norm"), self._name("o"): ParamSpec((D, C))})
        return specs

    def load(self, get: TensorGetter) -> None:
        self.mu = torch.stack([get(self._name(f"mu.{m}"), "vector").float() for m in _MIXES]).contiguous()
        self.w_rkvg = torch.stack([get(self._name(n), "matrix") for n in ("r", "k", "v", "g")]).contiguous()
        self.w1 = get(self._name("w1"), "matrix").contiguous()
        self.w2t = get(self._name("w2"), "matrix").float().t().contiguous()
        if self.w1.shape[0] != self.w2t.shape[0]:
            raise ValueError(f"{self.prefix}: the two steps of the decays' projection disagree on their inner size")
        self.decay_rank = int(self.w1.shape[0])
        self.w0, self.bonus, self.norm_w = (get(self._name(n), "vector").float().contiguous() for n in ("w0", "u", "norm"))
        self.w_out = get(self._name("o"), "matrix").contiguous()

    def forward(self, x, ctx, cache: LayerCache):
        """``x``: the float32 residual rows."""
        if cache.state is None:
            raise RuntimeError("the wkv mixer needs its state slots")
        N, C = ctx.num_tokens, self.size
        mixes = torch.empty((len(_MIXES), N, self.hidden_size), dtype=ctx.dtype, device=x.device)
        kernels.wkv_shift(x, self.mu, cache.state, 0, ctx.q_start, ctx.slots, ctx.positions, ctx.token_request, mixes)
        r, k, v, z = (linear(mixes[i], self.w_rkvg[i], out_dtype=torch.float32) for i in range(4))
        low = linear(mixes[4], self.w1, out_dtype=torch.float32)
        decay = kernels.wkv_decay(low, self.w2t, self.w0, torch.empty((N, C), dtype=torch.float32, device=x.device))
        o = torch.empty((N, C), dtype=torch.float32, device=x.device)
        kernels.wkv_scan(r, k, v, decay, self.bonus, cache.state, 2 * self.hidden_size, ctx.q_start, ctx.slots, ctx.positions, o,
                         self.heads, self.dim, kernels.wkv_segments(ctx.max_q_len, ctx.num_requests, self.heads, self.dim))
        gated = torch.empty((N, C), dtype=ctx.dtype, device=x.device)
        kernels.wkv_gate(o, z, self.norm_w, gated, self.heads, self.dim, self.eps)
        return linear(gated, self.w_out, out_dtype=torch.float32), None
