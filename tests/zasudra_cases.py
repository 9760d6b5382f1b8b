"""Small Zasudra configurations with weights made for the tests, and the comparison with the plain implementation.

The weights are drawn so that every mechanism carries weight in the logits: projections of unit gain, norm weights, sinks,
mixes with the token before, bonuses, router biases well away from their neutral values, decays between "forgets within a
few tokens" and "keeps hundreds". They are rounded to bfloat16 once, so the engine in either type and the float64 oracle
read the same numbers. ``sharpen`` raises the score scales so that a softmax sits on one or two keys anywhere in what a
token sees, and a key that is lost, shifted by one or read from another page changes the result by its whole value."""

from __future__ import annotations

import copy
import math
from typing import Dict, List, Optional

import torch

import plain_zasudra as plain
from razelorn_cases import assert_matches, row_errors, write_model, TOL  # noqa: F401  (shared test helpers)


def moe(ff: int, experts: int, top: int) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def chunked(heads: int, kv_heads: int, dim: int, size: Optional[int], rot: Optional[int] = None, base: float = 50.0,
            mlp: Optional[dict] = None) -> dict:
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 1.0 / math.sqrt(dim)}
    if size is not None:
        mixer["mask"] = {"size": size}
    if rot is not None:
        mixer["rot"] = {"base": base, "dims": rot}
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def wkv(heads: int, dim: int, mlp: Optional[dict] = None) -> dict:
    return {"type": "wkv", "mlp": mlp, "mixer": {"heads": heads, "dim": dim}}


def causal(heads: int, kv_heads: int, dim: int, vdim: int, kv_from: Optional[int] = None, mlp: Optional[dict] = None) -> dict:
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.0 / math.sqrt(dim)}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention_2", "mlp": mlp, "mixer": mixer}


def config(layers: List[dict], width: int = 64, vocab: int = 131, eps: float = 1e-5, mult: float = 0.6, logit_scale: float = 1.7,
           bigram=(53, 7, 3)) -> dict:
    out = {"architecture": "Zasudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
           "logit_scale": logit_scale, "layers": layers}
    if bigram is not None:
        out["embedding"] = {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}
    return out


# Several shapes. Key/value heads that are one, several or as many as the heads; values wider than, as wide as and narrower
# than keys; chunks shorter and longer than a page and no multiple of it, and none; a rotation of all, a part or none of a
# head; layers that read another layer's rows, also two of them; layers without experts; one expert a token and all of
# them; heads of the recurrence that are and are not powers of two; sizes that are no multiples of 4; with and without a
# bigram table, one of a single bucket; multipliers larger than the buckets.
CONFIGS: Dict[str, dict] = {
    "mixed": config([
        chunked(4, 2, 16, 24, 8, mlp=moe(40, 5, 2)),
        wkv(3, 20, mlp=moe(24, 4, 3)),
        causal(6, 3, 16, 24, mlp=moe(32, 6, 1)),
        causal(6, 3, 16, 24, kv_from=2),
        chunked(2, 2, 32, 10, 32, 1000.0),
        wkv(5, 16, mlp=moe(48, 3, 3)),
    ]),
    "causal_first": config([
        causal(8, 2, 32, 32, mlp=moe(24, 4, 2)),
        causal(8, 2, 32, 32, kv_from=0, mlp=moe(16, 9, 4)),
        chunked(3, 1, 64, 37, 16, mlp=moe(40, 2, 1)),
        wkv(2, 48),
        causal(8, 2, 32, 32, kv_from=0),
        chunked(4, 4, 16, None, None, mlp=moe(24, 3, 2)),
    ], width=48, vocab=97, eps=3e-6, mult=1.0, logit_scale=0.4, bigram=(1, 5, 2)),
    "odd_sizes": config([
        chunked(3, 1, 10, 7, 6, 37.0, mlp=moe(30, 3, 2)),
        wkv(3, 7, mlp=moe(18, 2, 2)),
        causal(3, 3, 10, 14),
        causal(3, 3, 10, 14, kv_from=2, mlp=moe(22, 7, 5)),
        wkv(1, 33, mlp=None),
    ], width=54, vocab=61, mult=0.35, bigram=(17, 1000003, 999983)),
    "wkv_only": config([wkv(4, 16, mlp=moe(32, 4, 2)), wkv(1, 100)], width=40, vocab=80, bigram=None),
    "wide_heads": config([
        causal(12, 3, 48, 48, mlp=moe(40, 12, 1)),
        chunked(16, 2, 128, 50, 64, 5000.0, mlp=moe(64, 3, 2)),
        causal(12, 3, 48, 48, kv_from=0, mlp=moe(32, 4, 4)),
        causal(40, 2, 64, 128),
        chunked(2, 1, 96, 33, 96),
        causal(4, 1, 80, 40, mlp=moe(24, 5, 2)),
    ], width=96, vocab=150, mult=0.5, logit_scale=2.5, bigram=(211, 2, 31)),
}


def sharpen(cfg: dict, sharp: float) -> dict:
    """Scores of spread ``sharp`` (the row norms give queries and keys of unit entries)."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["type"] != "wkv":
            layer["mixer"]["scale"] = sharp / math.sqrt(layer["mixer"]["dim"])
    return cfg


def decided(cfg: dict) -> dict:
    """Every token uses every expert: for bfloat16 where one close call of a router would move all tokens after it."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] is not None:
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


def weights_for(cfg: dict, seed: int, slow: bool = False, low_rank: int = 12) -> Dict[str, torch.Tensor]:
    """``slow``: decays close to one, so that the states keep what the first tokens wrote for hundreds of tokens."""
    gen = torch.Generator().manual_seed(seed)
    W: Dict[str, torch.Tensor] = {}

    def normal(*shape, std=1.0, mean=0.0):
        return torch.randn(*shape, generator=gen, dtype=torch.float32) * std + mean

    for name, shape in plain.expected_tensors(cfg, low_rank).items():
        leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
        if name in ("embed", "bigram"):
            W[name] = normal(*shape)
        elif name == "head":
            W[name] = normal(*shape, std=4.0 / math.sqrt(shape[1]))           # logits of a spread that leaves few near ties
        elif leaf.startswith("norm") or name == "final.norm" or leaf.endswith(".norm"):
            W[name] = normal(*shape, std=0.25, mean=1.0)
        elif ".mu." in leaf:
            W[name] = torch.rand(*shape, generator=gen) * 0.9 + 0.05
        elif leaf.endswith(".w0"):
            W[name] = normal(*shape, std=0.5, mean=-6.0) if slow else normal(*shape, std=1.2, mean=-1.8)
        elif leaf.endswith(".w2"):
            W[name] = normal(*shape, std=(0.3 if slow else 1.0) / math.sqrt(shape[1]))
        elif leaf.endswith(".u"):
            W[name] = normal(*shape, std=0.7, mean=0.5)
        elif leaf.endswith(".sink"):
            W[name] = normal(*shape, std=1.0, mean=0.7)
        elif leaf.endswith("router.b"):
            W[name] = normal(*shape, std=0.7)
        elif len(shape) == 2:
            W[name] = normal(*shape, std=1.0 / math.sqrt(shape[1]))
        else:
            raise AssertionError(f"no rule for {name} {shape}")
    return {name: t.to(torch.bfloat16).float() for name, t in W.items()}


def oracle(cfg: dict, W: Dict[str, torch.Tensor], requests: Dict[str, List[int]]) -> Dict[str, torch.Tensor]:
    return {rid: plain.forward(cfg, W, toks).float() for rid, toks in requests.items()}
