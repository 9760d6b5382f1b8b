"""A plain, slow implementation of the Zasudra decoder for the tests: whole sequences, no cache, float64, one function
per mechanism, written from the design's equations. It shares no code with the engine.

A model is ``(config, weights)``: ``config`` the dictionary of ``config.json``, ``weights`` a dictionary from tensor
names to tensors. Positions count from 0. Linear weights are ``[out, in]``."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float, w: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if w is None else y * w


def bigram_rows(tokens: List[int], mul_prev: int, mul_cur: int, buckets: int) -> List[int]:
    """The row of the bigram table for every token; the first token of a sequence has the row after the hashed ones."""
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embed(tokens: List[int], W: Dict[str, torch.Tensor], bigram: Optional[dict]) -> torch.Tensor:
    x = W["embed"][torch.tensor(tokens)].to(F)
    if bigram:
        rows = bigram_rows(tokens, int(bigram["mul_prev"]), int(bigram["mul_cur"]), int(bigram["buckets"]))
        x = x + W["bigram"][torch.tensor(rows)].to(F)
    return x


def rotate_interleaved(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, n]: the first ``dims`` entries of every head turn by their token's position, entry 2i with 2i + 1."""
    T = x.shape[0]
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    angle = torch.arange(T, dtype=F)[:, None, None] * f
    cos, sin = torch.cos(angle), torch.sin(angle)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def seen(T: int, chunk: Optional[int]) -> torch.Tensor:
    """[T, T]: whether the token of the row sees the key of the column."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    mask = j <= i
    return mask & (i // chunk == j // chunk) if chunk else mask


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, chunk: Optional[int], sink: torch.Tensor) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim], sink [H]: a softmax whose denominator also holds exp(sink). Returns
    [T, H, vdim]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    group = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, group]) * scale
    s = s.masked_fill(~seen(T, chunk), -math.inf)
    top = torch.maximum(s.max(dim=-1).values, sink[:, None])
    e = torch.exp(s - top[..., None])
    prob = e / (e.sum(dim=-1) + torch.exp(sink[:, None] - top))[..., None]
    return torch.einsum("hij,jhd->ihd", prob, v[:, group])


def chunked_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Values that are the projected keys, whole-row norms of q and k, interleaved rotation, chunks, a learned sink."""
    T, H, G, dim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    raw = h @ W[f"{p}.k"].T
    q = rms(h @ W[f"{p}.q"].T, eps, W[f"{p}.q.norm"]).view(T, H, dim)
    k = rms(raw, eps, W[f"{p}.k.norm"]).view(T, G, dim)
    rot = m.get("rot")
    if rot:
        q, k = (rotate_interleaved(a, int(rot["dims"]), float(rot["base"])) for a in (q, k))
    size = (m.get("mask") or {}).get("size")
    heads = attend(q, k, raw.view(T, G, dim), float(m["scale"]), int(size) if size else None, W[f"{p}.sink"].to(F))
    return heads.reshape(T, -1) @ W[f"{p}.o"].T


def gated_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float, shared=None):
    """Causal attention without rotation, one added to the denominator, a gate per head. ``shared``: (k, v) of the layer
    whose keys and values this one reads, or None. Returns (output, (k, v))."""
    T, H, G, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms(h @ W[f"{p}.q"].T, eps, W[f"{p}.q.norm"]).view(T, H, dim)
    if shared is None:
        k = rms(h @ W[f"{p}.k"].T, eps, W[f"{p}.k.norm"]).view(T, G, dim)
        shared = (k, (h @ W[f"{p}.v"].T).view(T, G, vdim))
    size = (m.get("mask") or {}).get("size")
    heads = attend(q, shared[0], shared[1], float(m["scale"]), int(size) if size else None, torch.zeros(H, dtype=F))
    heads = heads * torch.sigmoid(h @ W[f"{p}.g"].T)[..., None]
    return heads.reshape(T, -1) @ W[f"{p}.o"].T, shared


def token_shift(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def wkv_decay(mix: torch.Tensor, w1: torch.Tensor, w2: torch.Tensor, w0: torch.Tensor) -> torch.Tensor:
    return torch.exp(-torch.exp(torch.tanh(mix @ w1.T) @ w2.T + w0))


def wkv_scan(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, w: torch.Tensor, u: torch.Tensor,
             state: Optional[torch.Tensor] = None):
    """r, k, v, w [T, H, d], u [H, d]; the state [H, d, d] (key channel, value channel). Returns (o [T, H, d], state)."""
    T, H, d = r.shape
    S = torch.zeros(H, d, d, dtype=r.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hcj,hc->hj", S + u[:, :, None] * kv, r[t]))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out), S


def wkv(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, d = h.shape[0], int(m["heads"]), int(m["dim"])
    mix = {n: token_shift(h, W[f"{p}.mu.{n}"]) for n in ("r", "k", "v", "g", "w")}
    r, k, v = ((mix[n] @ W[f"{p}.{n}"].T).view(T, H, d) for n in ("r", "k", "v"))
    z = mix["g"] @ W[f"{p}.g"].T
    w = wkv_decay(mix["w"], W[f"{p}.w1"], W[f"{p}.w2"], W[f"{p}.w0"]).view(T, H, d)
    o, _state = wkv_scan(r, k, v, w, W[f"{p}.u"].to(F))
    o = rms(o, eps).reshape(T, H * d) * W[f"{p}.norm"] * (z * torch.sigmoid(z))
    return o @ W[f"{p}.o"].T


def route(h: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int):
    """(the chosen experts, largest logit first; their weights: a softmax over the chosen logits)"""
    z = h @ router.T + bias
    values, chosen = torch.sort(z, dim=-1, descending=True, stable=True)
    return chosen[:, :top], torch.softmax(values[:, :top], dim=-1)


def experts(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    chosen, weights = route(h, W[f"{p}.router"], W[f"{p}.router.b"], int(mlp["router"]["top"]))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            out[t] += w * (W[f"{p}.e{e}.down"] @ torch.relu(W[f"{p}.e{e}.up"] @ h[t]) ** 2)
    return out


def layer(x: torch.Tensor, W: Dict[str, torch.Tensor], i: int, spec: dict, eps: float, mult: float, shared: Dict[int, tuple]) -> torch.Tensor:
    p, m = f"l{i}.mix", spec["mixer"]
    if spec["type"] == "attention":
        y = chunked_attention(x, W, p, m, eps)
    elif spec["type"] == "wkv":
        y = wkv(x, W, p, m, eps)
    else:
        source = m.get("kv_from")
        y, shared[i] = gated_attention(x, W, p, m, eps, shared[int(source)] if source is not None else None)
    x = x + mult * rms(y, eps, W[f"l{i}.norm1"])
    if spec.get("mlp") is not None:
        x = x + mult * rms(experts(x, W, f"l{i}.mlp", spec["mlp"]), eps, W[f"l{i}.norm2"])
    return x


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], after_layers: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab], float64. ``after_layers``: receives the residual stream after every layer."""
    W = {name: t.to(F) for name, t in weights.items()}
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    x = embed(tokens, W, (config.get("embedding") or {}).get("bigram"))
    shared: Dict[int, tuple] = {}
    for i, spec in enumerate(config["layers"]):
        x = layer(x, W, i, spec, eps, mult, shared)
        if after_layers is not None:
            after_layers.append(x)
    return rms(x, eps, W["final.norm"]) @ W["head"].T * float(config["logit_scale"])


def expected_tensors(config: dict, low_rank: int = 16) -> Dict[str, tuple]:
    """Names and shapes of a model of this configuration; ``low_rank``: the inner size of the decays' two-step projection,
    which the tensors alone give."""
    D, V = int(config["width"]), int(config["vocab"])
    out: Dict[str, tuple] = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    bigram = (config.get("embedding") or {}).get("bigram")
    if bigram:
        out["bigram"] = (int(bigram["buckets"]) + 1, D)
    for i, spec in enumerate(config["layers"]):
        p, m = f"l{i}.mix", spec["mixer"]
        out[f"l{i}.norm1"] = (D,)
        H, d = int(m["heads"]), int(m["dim"])
        if spec["type"] == "wkv":
            out.update({f"{p}.mu.{n}": (D,) for n in ("r", "k", "v", "g", "w")})
            out.update({f"{p}.{n}": (H * d, D) for n in ("r", "k", "v", "g")})
            out.update({f"{p}.w1": (low_rank, D), f"{p}.w2": (H * d, low_rank), f"{p}.w0": (H * d,), f"{p}.u": (H, d),
                        f"{p}.norm": (H * d,), f"{p}.o": (D, H * d)})
        else:
            G, vdim = int(m["kv_heads"]), int(m["vdim"])
            out.update({f"{p}.q": (H * d, D), f"{p}.q.norm": (H * d,), f"{p}.o": (D, H * vdim)})
            if m.get("kv_from") is None:
                out.update({f"{p}.k": (G * d, D), f"{p}.k.norm": (G * d,)})
            if spec["type"] == "attention":
                out[f"{p}.sink"] = (H,)
            else:
                out[f"{p}.g"] = (H, D)
                if m.get("kv_from") is None:
                    out[f"{p}.v"] = (G * vdim, D)
        mlp = spec.get("mlp")
        if mlp is not None:
            E, ff = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            out[f"l{i}.norm2"] = (D,)
            out.update({f"l{i}.mlp.router": (E, D), f"l{i}.mlp.router.b": (E,)})
            for e in range(E):
                out.update({f"l{i}.mlp.e{e}.up": (ff, D), f"l{i}.mlp.e{e}.down": (D, ff)})
    return out
