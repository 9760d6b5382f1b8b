"""Small Zavizen configurations with weights made for the tests, and the comparison with the plain implementation.

The weights are drawn so that every mechanism carries weight in the logits: projections of unit gain, norm weights, layer
scales and hyper-connections well away from their neutral values, decays and step sizes between "forgets within a few tokens"
and "keeps hundreds". They are rounded to bfloat16 once, so the engine in either type and the float64 oracle read the same
numbers. ``sharpen`` raises the score scales so that a softmax sits on one or two keys anywhere before a token, and a key that is
lost, shifted by one or read from another page changes the result by its whole value."""

from __future__ import annotations

import copy
import math
from typing import Dict, List, Optional, Sequence

import torch

import plain_zavizen as plain
from razelorn_cases import assert_matches, row_errors, write_model, TOL  # noqa: F401  (shared test helpers)


def dense(ff: int) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(ff: int, experts: int, top: int, groups: Optional[tuple] = None, shared: Optional[int] = None, scale: Optional[float] = 1.7) -> dict:
    router: dict = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        router["scale"] = scale
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def rot(dims: int, base: float = 60.0, factor: Optional[float] = None) -> dict:
    out: dict = {"base": base, "dims": dims}
    if factor is not None:
        out["scaling"] = {"factor": factor}
    return out


def parallel(left: tuple, right: tuple, mlp: Optional[dict] = None, left_rot: Optional[dict] = None, right_rot: Optional[dict] = None,
             decay: Optional[Sequence[float]] = None) -> dict:
    """``left`` = (heads, kv_heads, dim, vdim), ``right`` = (heads, dim, vdim)."""
    a = dict(zip(("heads", "kv_heads", "dim", "vdim"), left))
    a["scale"] = 1.0 / math.sqrt(a["dim"])
    b = dict(zip(("heads", "dim", "vdim"), right))
    b["decay"] = list(decay) if decay is not None else [1.0 - 2.0 ** -(1.5 + 2.3 * h) for h in range(right[0])]
    if left_rot:
        a["rot"] = left_rot
    if right_rot:
        b["rot"] = right_rot
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": a, "right": b}}


def mamba2(heads: int, vdim: int, state: int, groups: int, conv: int, norm_groups: int, mlp: Optional[dict] = None) -> dict:
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                                    "norm_groups": norm_groups}}


def config(layers: List[dict], streams: int = 2, width: int = 64, vocab: int = 131, eps: float = 1e-5, loop: Optional[tuple] = None) -> dict:
    out = {"architecture": "Zavizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# Several shapes. One stream and many; a loop of one layer, of several, of the whole model, and none; key/value heads that are one,
# several or as many as the heads; values wider and narrower than keys; rotations of all, a part and none of a head, with and
# without scaled frequencies; one decay of zero and one of one; routers with and without groups, scale and shared expert, one
# choice and all experts; a state of one group and of as many groups as heads, convolutions of 1 to 5 taps, norms over the whole
# row and over parts that cut through heads; sizes that are no multiples of 4.
CONFIGS: Dict[str, dict] = {
    "mixed": config([
        parallel((4, 2, 16, 24), (3, 16, 20), dense(72), rot(8), rot(16, 900.0)),
        mamba2(4, 16, 24, 2, 4, 2, moe(40, 8, 3, (4, 2), 56)),
        parallel((6, 1, 32, 32), (2, 24, 16), moe(24, 6, 2, (3, 1)), rot(32, 5000.0, 3.0), rot(10)),
        mamba2(3, 8, 16, 1, 3, 1),
    ], streams=3, loop=(1, 3, 2)),
    "all_looped": config([
        parallel((3, 3, 16, 16), (4, 8, 32), moe(32, 5, 5, None, 24, None), None, rot(4, 30.0, 2.0), [0.0, 1.0, 0.75, 0.984375]),
        mamba2(6, 12, 20, 3, 5, 4, dense(40)),
    ], streams=4, width=48, vocab=97, eps=3e-6, loop=(0, 2, 3)),
    "odd_sizes": config([
        mamba2(3, 7, 5, 3, 1, 7, dense(30)),
        parallel((3, 1, 10, 14), (5, 6, 9), moe(22, 9, 2, (3, 3), 18, 0.6), rot(6), rot(6, 200.0, 0.5)),
        parallel((1, 1, 6, 10), (1, 33, 5)),
    ], streams=5, width=54, vocab=61),
    "one_stream": config([
        parallel((8, 2, 48, 48), (4, 32, 32), dense(64), rot(16, 100.0, 8.0), rot(32)),
        mamba2(2, 64, 64, 2, 2, 2, moe(40, 16, 4, (4, 3), 40)),
    ], streams=1, width=96, vocab=150, loop=(1, 2, 2)),
    "wide_heads": config([
        parallel((4, 4, 128, 128), (2, 128, 64), moe(64, 12, 1, (2, 1), None, 3.0), rot(64, 5000.0), rot(128, 5000.0)),
        mamba2(2, 128, 128, 1, 4, 1, moe(40, 4, 2, None, 72)),
        parallel((12, 3, 96, 96), (3, 64, 96), None, rot(24, 300.0, 4.0), None, [0.9, 0.97, 0.995]),
    ], streams=2, width=96, vocab=110, loop=(1, 3, 2)),
}


def sharpen(cfg: dict, sharp: float) -> dict:
    """Scores of spread ``sharp`` (the row norms give queries and keys of unit entries)."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["type"] == "parallel":
            layer["mixer"]["left"]["scale"] = sharp / math.sqrt(layer["mixer"]["left"]["dim"])
    return cfg


def decided(cfg: dict) -> dict:
    """Every token uses every expert: for bfloat16 where one close call of a router would move all tokens after it."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            router = layer["mlp"]["router"]
            router["top"] = router["experts"]
            if router.get("groups"):
                router["groups"]["keep"] = router["groups"]["count"]
    return cfg


def weights_for(cfg: dict, seed: int, slow: bool = False) -> Dict[str, torch.Tensor]:
    """``slow``: state-space decays close to one, so that the states keep what the first tokens wrote for hundreds of tokens."""
    gen = torch.Generator().manual_seed(seed)
    W: Dict[str, torch.Tensor] = {}

    def normal(*shape, std=1.0, mean=0.0):
        return torch.randn(*shape, generator=gen, dtype=torch.float32) * std + mean

    streams = cfg["streams"]
    for name, shape in plain.expected_tensors(cfg).items():
        leaf = name.split(".", 1)[1] if name[1].isdigit() else name
        if name == "embed":
            W[name] = normal(*shape)
        elif name == "head":
            W[name] = normal(*shape, std=4.0 / math.sqrt(shape[1]))           # logits of a spread that leaves few near ties
        elif leaf in ("norm1", "norm2", "final.norm"):
            W[name] = normal(*shape, std=0.25)                                 # stored around zero
        elif leaf.startswith("ls"):
            W[name] = normal(*shape, std=0.15, mean=0.45)
        elif leaf.startswith("hc"):
            kind = leaf.split(".")[1]
            W[name] = {"in": lambda: normal(*shape, std=0.4, mean=1.0 / streams), "out": lambda: normal(*shape, std=0.3, mean=0.7),
                       "mix": lambda: torch.eye(streams) * 0.7 + normal(*shape, std=0.25 / math.sqrt(streams), mean=0.2 / streams)}[kind]()
        elif leaf.endswith(("mix.norm", ".q.norm", ".k.norm", "left.out", "right.out")):
            W[name] = normal(*shape, std=0.25, mean=1.0)
        elif leaf.endswith("mix.conv"):
            W[name] = normal(*shape, std=0.8 / math.sqrt(shape[1]), mean=0.2)
        elif leaf.endswith("conv.b"):
            W[name] = normal(*shape, std=0.3)
        elif leaf.endswith("dt_bias"):
            W[name] = normal(*shape, std=0.3, mean=-4.5 if slow else -1.0)
        elif leaf.endswith("A_log"):
            W[name] = normal(*shape, std=0.3, mean=-1.0) if slow else normal(*shape, std=0.8)
        elif leaf.endswith("mix.D"):
            W[name] = normal(*shape, std=0.5, mean=0.7)
        elif leaf.endswith("mlp.router"):
            W[name] = normal(*shape, std=2.0 / math.sqrt(shape[1]))
        elif len(shape) == 2:
            W[name] = normal(*shape, std=1.0 / math.sqrt(shape[1]))
        else:
            raise AssertionError(f"no rule for {name} {shape}")
    return {name: t.to(torch.bfloat16).float() for name, t in W.items()}


def oracle(cfg: dict, W: Dict[str, torch.Tensor], requests: Dict[str, List[int]]) -> Dict[str, torch.Tensor]:
    return {rid: plain.forward(cfg, W, toks).float() for rid, toks in requests.items()}
