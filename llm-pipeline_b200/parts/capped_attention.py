"""Softmax attention with grouped key/value heads whose scores may be capped and lose a distance bias, over every earlier
token, a sliding window that keeps the first tokens, or chunks, with a sink in the denominator and a gate on the output
(``capped_attention``).

With h the mixer's input, H query heads, G key/value heads (head i uses key/value head i // (H / G)), queries and keys
of ``dim`` entries and values of ``vdim``::

    q, k, v = Wq h + bq, Wk h + bk, Wv h + bv
    v <- v / sqrt(mean(v^2) + eps)  per head, where ``value_norm_eps`` is given (cached so)
    s(i, j) = (q(i) . k(j)) * scale;   s <- cap * tanh(s / cap)  where ``softcap`` is given
    s(i, j) <- s(i, j) - slope_h (i - j),   slope_h = 2^(-8 (h + 1) / H)                  where ``distance_bias`` is set
    seen(i, j) = j <= i and (i - j < window or j < keep_first)                            (no window: every j <= i)
                 with ``chunk`` = n: j <= i and i // n == j // n, the chunks counted from position 0
    p(i, j) = exp(s(i, j)) / (exp(sink_h) + sum_seen exp(s))       sink_h: a constant (``sink`` = 0.0: one is added to the
                                                                   denominator), a tensor per head (``sink`` = "learned"), or none
    o_h(i) = sum_j p(i, j) v(j);   o <- o * sigmoid(Wg h)  where ``gate`` is set (``gate`` = "head": one number per head);   out = Wo o + bo

Without ``position`` there is no rotation: positions enter through the distance bias and the mask alone; kept tokens keep
their true positions. With ``row_norm_eps`` the whole rows of q and of k, before they are cut into heads, are divided by
their root mean square times a weight per entry, and then rotated where ``position`` names an encoding (the first
``rotary_dim`` entries of every head; ``interleaved``: entry 2i with 2i + 1 instead of i with i + rotary_dim / 2). ``values`` =
"keys": there is no Wv, v is k as projected, before norm and rotation. ``own_rows`` False: the layer has queries alone and
attends over the keys and values another layer cached.
The projections that read h are one product against [Wq; Wk; Wv; Wg] with a float32 result; one kernel adds the biases and
norms the values (or norms and rotates the rows of q and k), writes the queries in the compute type and the token's [k | v] rows into its page slot; the attention
kernel reads all keys and values from pages, this step's included, and applies the gate as it stores. Scores, cap, bias,
softmax and weighted sums are float32 (``csrc/capped_attention.cu``: any sizes, both types; ``csrc/capped_attention_mma.cu``:
bfloat16 on the tensor cores for key and value sizes of 16, 32, 64 and 128 and for keys and values of 48 or 96, the probabilities rounded to bfloat16 for the
product with the values; steps of single tokens over many keys cut them into segments with blocks of their own). The pages of
a windowed or chunked layer go back to the pool as soon as no later token sees them, but for those of the kept tokens
(``HeadRowPagesSpec(window, keep_first, chunk)``)."""

from __future__ import annotations

from typing import Dict, Optional, Union

import torch

from ..cache.spec import HeadRowPagesSpec
from ..ops import kernels
from ..ops.linear import linear
from ..weights.source import ParamSpec
from .attention import AttentionPolicy
from .base import LayerCache, Mixer, TensorGetter
from .registry import register_mixer


@register_mixer("capped_attention")
class CappedAttention(Mixer):
    graph_safe = True      # a step only writes this step's keys and values: repeating it changes nothing

    def __init__(self, prefix: str, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: Optional[float] = None, window: Optional[int] = None, keep_first: int = 0, distance_bias: bool = False,
                 sink: Union[None, float, str] = None, value_norm_eps: Optional[float] = None, gate: Union[bool, str] = False,
                 bias: bool = True, names: Optional[Dict[str, str]] = None, chunk: Optional[int] = None,
                 row_norm_eps: Optional[float] = None, position: Optional[str] = None, rotary_dim: int = 0, interleaved: bool = False,
                 values: str = "projected", own_rows: bool = True):
        """``names``: the tensors' names below ``prefix`` where they differ from ``q``, ``k``, ``v``, ``o``, ``g``, ``sink``
        (biases add ``.b``, row norms ``.norm``)."""
        self.prefix, self.hidden_size = prefix, int(hidden_size)
        self.num_heads, self.num_kv_heads, self.dim, self.vdim = int(num_heads), int(num_kv_heads), int(dim), int(vdim)
        if self.num_heads <= 0 or self.num_kv_heads <= 0 or self.num_heads % self.num_kv_heads:
            raise ValueError(f"{self.num_heads} query heads cannot share {self.num_kv_heads} key/value heads")
        if not 0 < self.vdim <= 512:
            raise ValueError(f"the capped attention kernel takes value sizes up to 512, got {self.vdim}")
        self.scale, self.softcap = float(scale), float(softcap) if softcap else 0.0
        self.window = int(window) if window else None
        self.keep_first = int(keep_first or 0) if self.window else 0
        self.chunk = int(chunk) if chunk else None
        if gate not in (False, True, "head"):
            raise ValueError(f"a gate is True, False or 'head', got {gate!r}")
        self.distance_bias, self.gate, self.bias = bool(distance_bias), gate, bool(bias)
        if sink is not None and sink != "learned" and not isinstance(sink, (int, float)):
            raise ValueError(f"a sink is a number, 'learned' or None, got {sink!r}")
        self.sink = sink
        self.value_norm_eps = None if value_norm_eps is None else float(value_norm_eps)
        self.row_norm_eps = None if row_norm_eps is None else float(row_norm_eps)
        self.position, self.rotary_dim, self.interleaved = position, int(rotary_dim) if position else 0, bool(interleaved)
        if self.rotary_dim < 0 or self.rotary_dim > self.dim or self.rotary_dim % 2:
            raise ValueError(f"{self.rotary_dim} rotated entries do not fit heads of {self.dim}")
        if values not in ("projected", "keys"):
            raise ValueError(f"values are 'projected' or the 'keys', got {values!r}")
        self.values_are_keys, self.own_rows = values == "keys", bool(own_rows)
        if self.values_are_keys and self.vdim != self.dim:
            raise ValueError(f"values that are the keys have their size, got {self.vdim} and {self.dim}")
        if self.row_norm_eps is None and (self.rotary_dim or self.values_are_keys or not self.own_rows):
            raise ValueError("rotation, values that are the keys and another layer's rows go with norms over the rows of q and k")
        if self.row_norm_eps is not None and (self.bias or self.value_norm_eps is not None):
            raise ValueError("norms over the rows of q and k come without biases and value norm")
        self.q_size, self.k_size, self.v_size = self.num_heads * self.dim, self.num_kv_heads * self.dim, self.num_kv_heads * self.vdim
        self.o_size = self.num_heads * self.vdim
        self.names = {n: n for n in ("q", "k", "v", "o", "g", "sink")}
        self.names.update(names or {})
        self.w_in = self.b_qkv = self.w_o = self.b_o = self.slopes = self.sinks = self.q_norm = self.k_norm = None

    # Single tokens whose tiles are fewer than this many blocks an SM share their keys among segments, from this many keys on.
    SEGMENTS_BELOW_BLOCKS_PER_SM = 4
    SEGMENTS_MIN_KEYS = 512

    def cache_spec(self) -> Optional[HeadRowPagesSpec]:
        return HeadRowPagesSpec(self.num_kv_heads, self.dim + self.vdim, self.window, self.keep_first, self.chunk) if self.own_rows else None

    def graph_key_group(self):
        return ("capped_attention", self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.window, self.keep_first, self.chunk)

    def _projections(self):
        """The matrices whose products are the columns of the one input product, in their order (the gate follows them)."""
        if not self.own_rows:
            return ("q",)
        return ("q", "k") if self.values_are_keys else ("q", "k", "v")

    def _segments(self, ctx) -> int:
        """Into how many segments a step of single tokens cuts its keys (0: not at all)."""
        if ctx.max_q_len != 1:
            return 0
        longest = ctx.decode_ctx_bound or ctx.max_ctx_len
        tile = kernels.CAPPED_TILE_KEYS
        bounds = [n for n in (self.window, self.chunk) if n]
        reach = min([longest] + [n + tile for n in bounds])            # from the tile a row's keys begin in
        blocks = ctx.num_requests * self.num_kv_heads * -(-(self.num_heads // self.num_kv_heads) // 16)
        if reach < self.SEGMENTS_MIN_KEYS or blocks >= self.SEGMENTS_BELOW_BLOCKS_PER_SM * kernels.sm_count():
            return 0
        return -(-reach // kernels.CAPPED_SEGMENT_KEYS)

    def _name(self, key: str) -> str:
        return f"{self.prefix}.{self.names[key]}"

    def _tiles(self, ctx, per_tile: int):
        key = ("capped_attention_tiles", per_tile)
        tiles = ctx.memo.get(key)
        if tiles is None:
            if ctx.max_q_len == 1:
                # one token a request: tile r is request r (made on the device, so that a captured step holds no copy from the host)
                tiles = (torch.arange(ctx.num_requests, dtype=torch.int32, device=ctx.device),
                         torch.zeros(ctx.num_requests, dtype=torch.int32, device=ctx.device))
            else:
                req, tok0, _seg, _slot, _places = AttentionPolicy.plan_items(ctx.starts, ctx.q_lens, per_tile, 0, 1, 1, kernels.sm_count())
                host = torch.tensor([req, tok0], dtype=torch.int32).pin_memory()
                dev = host.to(ctx.device, non_blocking=True)
                tiles = (dev[0].contiguous(), dev[1].contiguous())
            ctx.memo[key] = tiles
        return tiles

    def param_specs(self) -> Dict[str, ParamSpec]:
        D = self.hidden_size
        sizes = {"q": self.q_size, "k": self.k_size, "v": self.v_size}
        specs = {self._name(n): ParamSpec((sizes[n], D)) for n in self._projections()}
        specs[self._name("o")] = ParamSpec((D, self.o_size))
        if self.bias:
            specs.update({self._name(n) + ".b": ParamSpec((sizes[n],), role="vector", init="small") for n in ("q", "k", "v")})
            specs[self._name("o") + ".b"] = ParamSpec((D,), role="vector", init="small")
        if self.gate:
            specs[self._name("g")] = ParamSpec((self.num_heads if self.gate == "head" else self.o_size, D))
        if self.row_norm_eps is not None:
            specs[self._name("q") + ".norm"] = ParamSpec((self.q_size,), role="vector", init="norm")
            if self.own_rows:
                specs[self._name("k") + ".norm"] = ParamSpec((self.k_size,), role="vector", init="norm")
        if self.sink == "learned":
            specs[self._name("sink")] = ParamSpec((self.num_heads,), role="vector", init="small")
        return specs

    def load(self, get: TensorGetter) -> None:
        parts = [get(self._name(n), "matrix") for n in self._projections()]
        if self.gate:
            parts.append(get(self._name("g"), "matrix"))
        self.w_in = torch.cat(parts, dim=0).contiguous()
        self.w_o = get(self._name("o"), "matrix").contiguous()
        device = self.w_o.device
        if self.row_norm_eps is not None:
            self.q_norm = get(self._name("q") + ".norm", "vector").float().contiguous()
            if self.own_rows:
                self.k_norm = get(self._name("k") + ".norm", "vector").float().contiguous()
        if self.bias:
            self.b_qkv = torch.cat([get(self._name(n) + ".b", "vector").float() for n in ("q", "k", "v")]).contiguous()
            self.b_o = get(self._name("o") + ".b", "vector").float().contiguous()
        H = self.num_heads
        self.slopes = (torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=torch.float64).float().to(device)
                       if self.distance_bias else None)
        if self.sink == "learned":
            self.sinks = get(self._name("sink"), "vector").float().contiguous()
        elif self.sink is not None:
            self.sinks = torch.full((H,), float(self.sink), dtype=torch.float32, device=device)

    def forward(self, x, ctx, cache: LayerCache):
        return self.forward_from(linear(x, self.w_in, out_dtype=torch.float32), ctx, cache)         # [N, q | k | v | gate]

    def forward_from(self, proj, ctx, cache: LayerCache):
        if cache.pages is None or cache.group is None:
            raise RuntimeError("the capped attention mixer needs the pages of its cache")
        N = ctx.num_tokens
        sizes = {"q": self.q_size, "k": self.k_size, "v": self.v_size}
        width = sum(sizes[n] for n in self._projections())
        q = torch.empty((N, self.q_size), dtype=ctx.dtype, device=proj.device)
        writes = cache.writes and self.own_rows
        pages, slots = (cache.pages, ctx.slot_mapping[cache.group]) if writes else (None, None)
        if self.row_norm_eps is None:
            kernels.capped_qkv_post(proj[:, :width], self.b_qkv, self.value_norm_eps, q, slots, pages, self.num_heads, self.num_kv_heads,
                                    self.dim, self.vdim)
        else:
            cos, sin = ctx.position_tables[self.position] if self.rotary_dim else (None, None)
            v_at = self.q_size + (0 if self.values_are_keys else self.k_size)
            kernels.capped_rows_post(proj, self.q_norm, self.k_norm, self.row_norm_eps, cos, sin, self.rotary_dim, self.interleaved, q, slots,
                                     pages, v_at, self.num_heads, self.num_kv_heads, self.dim, self.vdim)
        out = torch.empty((N, self.o_size), dtype=ctx.dtype, device=proj.device)
        gate = proj[:, width:] if self.gate else None
        tables = ctx.block_tables[cache.group]
        sizes = (self.num_heads, self.num_kv_heads, self.dim, self.vdim, self.window or 0, self.keep_first, self.scale, self.softcap)
        if kernels.capped_mma_supports(ctx.dtype, self.dim, self.vdim) and (width % 2 == 0 or self.gate is not True):
            # bfloat16 and sizes the tensor-core kernel has instances of: prompts in tiles of 64 rows (token, head of a group),
            # single tokens with the four warps of a block sharing the keys
            tile_req, tile_tok0 = self._tiles(ctx, kernels.capped_mma_tokens_per_tile(self.num_heads, self.num_kv_heads))
            kernels.capped_attention_mma(q, cache.pages, tables, ctx.q_start, ctx.ctx_len, tile_req, tile_tok0, out, *sizes, slopes=self.slopes,
                                         sink=self.sinks, gate=gate, split=ctx.max_q_len == 1, chunk=self.chunk or 0,
                                         segments=self._segments(ctx))
        else:
            kernels.capped_attention(q, cache.pages, tables, ctx.token_request, ctx.positions, out, *sizes, slopes=self.slopes, sink=self.sinks,
                                     gate=gate, chunk=self.chunk or 0)
        return linear(out, self.w_o, out_dtype=torch.float32), self.b_o
