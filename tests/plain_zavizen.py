"""A plain, slow implementation of the Zavizen decoder for the tests: whole sequences, no cache, float64, one function per
mechanism, written from the design's equations. It shares no code with the engine.

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


def silu(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def rotate(x: torch.Tensor, rot: Optional[dict]) -> torch.Tensor:
    """x [T, heads, n]: entry i of the first ``dims`` of every head turns with entry i + dims / 2 by the token's position
    times ``base ** (-2 i / dims) / factor``."""
    if not rot or not int(rot["dims"]):
        return x
    dims, base = int(rot["dims"]), float(rot["base"])
    half = dims // 2
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(half)], dtype=F)
    angle = torch.arange(x.shape[0], dtype=F)[:, None, None] * f
    cos, sin = torch.cos(angle), torch.sin(angle)
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * cos - v * sin
    out[..., half:dims] = v * cos + u * sin
    return out


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]: an ordinary causal softmax. Returns [T, H, vdim]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    group = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, group]) * scale
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v[:, group])


def attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms(h @ W[f"{p}.q"].T, eps, W[f"{p}.q.norm"]).view(T, H, dim)
    k = rms(h @ W[f"{p}.k"].T, eps, W[f"{p}.k.norm"]).view(T, G, dim)
    v = (h @ W[f"{p}.v"].T).view(T, G, vdim)
    out = attend(rotate(q, m.get("rot")), rotate(k, m.get("rot")), v, float(m["scale"]))
    return out.reshape(T, -1) @ W[f"{p}.o"].T


def retention_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: Optional[torch.Tensor] = None):
    """q, k [T, H, dim], v [T, H, vdim], decay [H]; the state [H, dim, vdim]. Returns (o [T, H, vdim], state)."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hcj,hc->hj", S, q[t]))
    return torch.stack(out), S


def retention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, dim, vdim = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate((h @ W[f"{p}.q"].T).view(T, H, dim), m.get("rot"))
    k = rotate((h @ W[f"{p}.k"].T).view(T, H, dim), m.get("rot")) / math.sqrt(dim)
    v = (h @ W[f"{p}.v"].T).view(T, H, vdim)
    o, _state = retention_scan(q, k, v, torch.tensor([float(d) for d in m["decay"]], dtype=F))
    return (rms(o, eps).reshape(T, -1) * silu(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def parallel(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    left = rms(attention(h, W, f"{p}.left", m["left"], eps), eps, W[f"{p}.left.out"])
    right = rms(retention(h, W, f"{p}.right", m["right"], eps), eps, W[f"{p}.right.out"])
    return 0.5 * (left + right)


def short_conv(x: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    T, K = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return sum(padded[k:k + T] * taps[:, k] for k in range(K)) + bias


def ssd_scan(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor, skip: torch.Tensor) -> torch.Tensor:
    """x [T, H, P], B, C [T, G, N], dt [T, H] after its softplus. Returns [T, H, P]."""
    T, H, P = x.shape
    group = torch.arange(H) // (H // B.shape[1])
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    out = []
    for t in range(T):
        a = torch.exp(-torch.exp(a_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t, group][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t, group]) + skip[:, None] * x[t])
    return torch.stack(out)


def mamba2(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, P, N, G = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * P
    z, xbc, dt = (h @ W[f"{p}.in"].T).split([inner, inner + 2 * G * N, H], dim=1)
    x, B, C = silu(short_conv(xbc, W[f"{p}.conv"], W[f"{p}.conv.b"])).split([inner, G * N, G * N], dim=1)
    raw = dt + W[f"{p}.dt_bias"]
    dt = torch.clamp(raw, min=0.0) + torch.log1p(torch.exp(-raw.abs()))
    y = ssd_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, W[f"{p}.A_log"], W[f"{p}.D"])
    y = y.reshape(T, inner) * silu(z)
    parts = int(m["norm_groups"])
    y = rms(y.view(T, parts, inner // parts), eps).reshape(T, inner) * W[f"{p}.norm"]
    return y @ W[f"{p}.o"].T


def gated(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ W[f"{p}.gate"].T) * (h @ W[f"{p}.up"].T)) @ W[f"{p}.down"].T


def route(h: torch.Tensor, router: torch.Tensor, r: dict):
    """(the chosen experts, largest score first; their weights). Only experts of the groups whose best scores are the largest
    can be chosen."""
    s = torch.softmax(h @ router.T, dim=-1)
    eligible = s
    groups = r.get("groups")
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        best = s.view(s.shape[0], count, -1).max(dim=-1).values
        kept = torch.sort(best, dim=-1, descending=True, stable=True).indices[:, :keep]
        mask = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True)
        eligible = s.masked_fill(~mask.repeat_interleave(s.shape[1] // count, dim=1), -1.0)
    chosen = torch.sort(eligible, dim=-1, descending=True, stable=True).indices[:, :int(r["top"])]
    w = s.gather(1, chosen)
    return chosen, w / (w.sum(dim=-1, keepdim=True) + 1e-20) * float(r.get("scale", 1.0))


def experts(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mlp: dict) -> torch.Tensor:
    chosen, weights = route(h, W[f"{p}.router"], mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t].tolist(), weights[t]):
            out[t] += w * gated(h[t:t + 1], W, f"{p}.e{e}")[0]
    return out + gated(h, W, f"{p}.shared") if mlp.get("shared") else out


MIXERS = {"parallel": parallel, "mamba2": mamba2}


def sublayer(xs: torch.Tensor, W: Dict[str, torch.Tensor], layer: str, q: int, eps: float, fn) -> torch.Tensor:
    """One sublayer between hyper-connections. xs [streams, T, D]."""
    hc = f"{layer}.hc{q}"
    u = torch.einsum("s,std->td", W[f"{hc}.in"], xs)
    y = fn(rms(u, eps, 1.0 + W[f"{layer}.norm{q}"])) * W[f"{layer}.ls{q}"]
    return torch.einsum("st,snd->tnd", W[f"{hc}.mix"], xs) + W[f"{hc}.out"][:, None, None] * y


def layer_order(config: dict) -> List[int]:
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def forward(config: dict, weights: Dict[str, torch.Tensor], tokens: List[int], after_layers: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits [T, vocab], float64. ``after_layers``: receives the sum of the streams after every layer run."""
    W = {name: t.to(F) for name, t in weights.items()}
    eps = float(config["norm"]["eps"])
    x = W["embed"][torch.tensor(tokens)]
    xs = torch.stack([x] * int(config["streams"]))
    for i in layer_order(config):
        spec = config["layers"][i]
        xs = sublayer(xs, W, f"l{i}", 1, eps, lambda h: MIXERS[spec["type"]](h, W, f"l{i}.mix", spec["mixer"], eps))
        mlp = spec.get("mlp")
        if mlp is not None:
            feed = gated if mlp["kind"] == "dense" else lambda h, W, p: experts(h, W, p, mlp)
            xs = sublayer(xs, W, f"l{i}", 2, eps, lambda h: feed(h, W, f"l{i}.mlp"))
        if after_layers is not None:
            after_layers.append(xs.sum(dim=0))
    return rms(xs.sum(dim=0), eps, 1.0 + W["final.norm"]) @ W["head"].T


def expected_tensors(config: dict) -> Dict[str, tuple]:
    """Names and shapes of a model of this configuration."""
    D, V, s = int(config["width"]), int(config["vocab"]), int(config["streams"])
    out: Dict[str, tuple] = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    for i, spec in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.mix", spec["mixer"], spec.get("mlp")
        for q in ((1, 2) if mlp is not None else (1,)):
            out.update({f"l{i}.norm{q}": (D,), f"l{i}.ls{q}": (D,), f"l{i}.hc{q}.in": (s,), f"l{i}.hc{q}.out": (s,), f"l{i}.hc{q}.mix": (s, s)})
        if spec["type"] == "mamba2":
            H, P, N, G = (int(m[k]) for k in ("heads", "vdim", "state", "groups"))
            channels = H * P + 2 * G * N
            out.update({f"{p}.in": (H * P + channels + H, D), f"{p}.conv": (channels, int(m["conv"])), f"{p}.conv.b": (channels,),
                        f"{p}.dt_bias": (H,), f"{p}.A_log": (H,), f"{p}.D": (H,), f"{p}.norm": (H * P,), f"{p}.o": (D, H * P)})
        else:
            a, r = m["left"], m["right"]
            H, G, dim, vdim = (int(a[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
            out.update({f"{p}.left.q": (H * dim, D), f"{p}.left.k": (G * dim, D), f"{p}.left.v": (G * vdim, D), f"{p}.left.o": (D, H * vdim),
                        f"{p}.left.q.norm": (H * dim,), f"{p}.left.k.norm": (G * dim,), f"{p}.left.out": (D,), f"{p}.right.out": (D,)})
            H, dim, vdim = (int(r[k]) for k in ("heads", "dim", "vdim"))
            out.update({f"{p}.right.{n}": (H * dim, D) for n in ("q", "k")})
            out.update({f"{p}.right.{n}": (H * vdim, D) for n in ("v", "g")})
            out[f"{p}.right.o"] = (D, H * vdim)
        if mlp is not None:
            sizes = {"": int(mlp["ff"])} if mlp["kind"] == "dense" else {f".e{e}": int(mlp["expert"]["ff"]) for e in range(int(mlp["router"]["experts"]))}
            if mlp["kind"] == "moe":
                out[f"l{i}.mlp.router"] = (int(mlp["router"]["experts"]), D)
                if mlp.get("shared"):
                    sizes[".shared"] = int(mlp["shared"]["ff"])
            for name, ff in sizes.items():
                out.update({f"l{i}.mlp{name}.gate": (ff, D), f"l{i}.mlp{name}.up": (ff, D), f"l{i}.mlp{name}.down": (D, ff)})
    return out
