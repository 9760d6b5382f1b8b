"""Hyper-connections: several copies ("streams") of the hidden state instead of one residual.

With streams x_1 .. x_s, all equal to the embedding's output at the start, a sublayer F with its norm and the learned
``in`` [s], ``mix`` [s, s] (from, to), ``out`` [s] and, where it has one, a scale per column::

    u = sum_s in[s] x_s;   y = F(norm(u)) * scale;   x_t <- sum_s mix[s, t] x_s + out[t] y   (all t at once)

and after the last layer the streams are summed. ``HyperStream`` is the residual stream of such a model. The update is not
taken where a sublayer ends: it stays pending, with the addends the sublayer left, and the next norm's kernel
(``csrc/hyper_connections.cu``) takes it, forms the next reader's input and norms that in one pass over the row. The streams
are float32 ``[tokens, s, hidden]``; until the first update they are the embedding's one row per token."""

from __future__ import annotations

from typing import Dict, Optional, Sequence

import torch

from ..ops import kernels
from ..weights.source import ParamSpec
from .base import Addend, Block, LayerCache, Part, ResidualStream, TensorGetter
from .registry import register_block


class HyperStream(ResidualStream):
    plain = False                         # its norms always go through ``fold``

    def __init__(self, residual: torch.Tensor, streams: int):
        """``residual``: [tokens, hidden], every stream's start, or the streams [tokens, streams, hidden]."""
        super().__init__(residual)
        self.streams = int(streams)
        self._addends: Sequence[Addend] = ()
        self._update: Optional["HyperConnection"] = None
        self._reader: Optional["HyperConnection"] = None

    def read_through(self, connection: "HyperConnection") -> None:
        """The next norm of all rows sees the streams combined by this connection's ``in`` weights (else: their sum)."""
        self._reader = connection

    def update(self, addends: Sequence[Addend], connection: "HyperConnection") -> None:
        """The sublayer behind this connection is done and left ``addends``."""
        if self._update is not None:
            raise RuntimeError("the streams already hold a pending update")
        self._addends, self._update = tuple(addends), connection

    def add(self, delta, bias=None, norm=None) -> None:
        raise RuntimeError("streams joined by hyper-connections are updated through a connection, not by a plain addend")

    add_beside = mix = add

    def fold(self, weight: Optional[torch.Tensor] = None, eps: float = 0.0, out: Optional[torch.Tensor] = None,
             rows: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
        update = self._update
        dst = None
        if update is not None and rows is None:
            dst = self.residual if self.residual.dim() == 3 else torch.empty(
                (self.residual.shape[0], self.streams, self.residual.shape[-1]), dtype=torch.float32, device=self.residual.device)
        kernels.stream_step(self.residual, self.streams, dst=dst, addends=[(a.rows, a.weight, a.eps, a.factor) for a in self._addends],
                            scale=update.scale if update is not None else None, mix=update.mix if update is not None else None,
                            out_weights=update.out if update is not None else None,
                            in_weights=self._reader.into if self._reader is not None and rows is None else None,
                            weight=weight, eps=eps, out=out, rows=rows)
        if rows is None:
            if dst is not None:
                self.residual = dst
            self._addends, self._update, self._reader = (), None, None
        return out

    def settled_rows(self, dtype: torch.dtype) -> torch.Tensor:
        out = torch.empty((self.residual.shape[0], self.residual.shape[-1]), dtype=dtype, device=self.residual.device)
        return self.fold(out=out)

    def settle(self) -> torch.Tensor:
        if self._update is not None:
            self.fold()
        if self.residual.dim() == 2:
            self.residual = self.residual.unsqueeze(1).expand(-1, self.streams, -1).contiguous()
        return self.residual

    def take_addends(self):
        raise RuntimeError("a norm that adds plain addends cannot stand between hyper-connections")

    def take_pending_product(self):
        return None


class HyperConnection(Part):
    """The learned numbers around one sublayer: ``<prefix>.in``, ``.out`` [streams], ``.mix`` [streams, streams] and the scale per
    column ``scale_name`` [size] (None: none), all float32 on the device."""

    graph_safe = True

    def __init__(self, prefix: str, streams: int, size: int, scale_name: Optional[str] = None, unused: Optional[Dict[str, tuple]] = None):
        """``unused``: names and shapes of tensors a checkpoint may hold although nothing reads them."""
        self.prefix, self.streams, self.size, self.scale_name = prefix, int(streams), int(size), scale_name
        self.unused = dict(unused or {})
        if not 1 <= self.streams <= kernels.HYPER_MAX_STREAMS:
            raise ValueError(f"hyper-connections join 1 to {kernels.HYPER_MAX_STREAMS} streams, got {streams}")
        self.into = self.out = self.mix = self.scale = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        p, S = self.prefix, self.streams
        specs = {f"{p}.in": ParamSpec((S,), role="vector", init="average"), f"{p}.out": ParamSpec((S,), role="vector", init="unit"),
                 f"{p}.mix": ParamSpec((S, S), role="vector", init="average")}
        if self.scale_name:
            specs[self.scale_name] = ParamSpec((self.size,), role="vector", init="unit")
        specs.update({name: ParamSpec(tuple(shape), role="vector", optional=True, init="small") for name, shape in self.unused.items()})
        return specs

    def load(self, get: TensorGetter) -> None:
        p = self.prefix
        self.into, self.out, self.mix = (get(f"{p}.{n}", "vector").float().contiguous() for n in ("in", "out", "mix"))
        self.scale = get(self.scale_name, "vector").float().contiguous() if self.scale_name else None


@register_block("hyper_connected")
class HyperConnectedBlock(Block):
    """A norm before each sublayer, hyper-connections around it. ``connections``: the arguments of one ``HyperConnection`` per
    sublayer (mixer, then feed-forward if the layer has one)."""

    NORMS = ("mixer", "feed_forward")

    def __init__(self, mixer, feed_forward, mixer_norm=None, feed_forward_norm=None, norms=None, depth_mix=None, connections=()):
        super().__init__(mixer, feed_forward, mixer_norm, feed_forward_norm, norms, depth_mix)
        self.connections = [HyperConnection(**c) for c in connections]
        if len(self.connections) != (1 if feed_forward is None else 2):
            raise ValueError(f"a layer needs one connection per sublayer, got {len(self.connections)}")

    def needed_norms(self):
        return self.NORMS if self.feed_forward is not None else ("mixer",)

    def parts(self):
        return super().parts() + tuple(self.connections)

    def forward(self, stream: HyperStream, ctx, cache: LayerCache) -> None:
        for name, part, connection in zip(self.NORMS, (self.mixer, self.feed_forward), self.connections):
            stream.read_through(connection)
            h = self.norms[name].add_norm(stream, ctx)
            args = (h, ctx, cache) if name == "mixer" else (h, ctx)
            addends = getattr(part, "forward_addends", None)
            if addends is not None:
                stream.update(addends(*args), connection)
            else:
                out, bias = part.forward(*args)
                stream.update([Addend(out if bias is None else out.float() + bias.float())], connection)
