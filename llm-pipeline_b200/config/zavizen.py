"""Typed configuration of the Zavizen decoder, read from its ``config.json``.

A small hybrid decoder whose hidden state is several streams joined by hyper-connections (``parts/hyper_connections.py``): a
sublayer reads a weighted sum of the streams behind a norm, and its output, scaled column by column, enters all of them. A
run of layers may be executed several times in a row with the same weights (``loop``), each pass with a cache and state of
its own. A layer names its mixer by ``type``:

* ``mamba2``: a state-space recurrence with a scalar decay per head and token;
* ``parallel``: causal attention with norms over the whole rows of q and k beside retention, which read the same input; the
  result is half the sum of the two, each normed over the row.

The feed-forward (``mlp``) is ``dense`` (gated SiLU), ``moe`` (gated SiLU experts chosen by a softmax router inside the best
groups of experts, the chosen scores renormalised and scaled, a shared expert that every token uses) or null for none.
Keys::

    {"architecture": "Zavizen", "vocab": V, "width": D, "norm": {"eps": e}, "streams": s,
     "loop": {"start": i, "stop": j, "times": n},
     "layers": [{"type": "mamba2", "mlp": {"kind": "dense", "ff": F},
                 "mixer": {"heads": H, "vdim": P, "state": N, "groups": G, "conv": K, "norm_groups": g}},
                {"type": "parallel", "mlp": {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": S},
                                             "router": {"experts": E, "top": k, "scale": c, "groups": {"count": n, "keep": m}}},
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": v, "scale": c,
                                    "rot": {"base": b, "dims": r, "scaling": {"factor": f}}},
                           "right": {"heads": H, "dim": d, "vdim": v, "decay": [one per head], "rot": {"base": b, "dims": r}}}}]}

Tensor names: ``embed``, ``final.norm``, ``head``; per layer i and sublayer q (1: mixer, 2: feed-forward) ``l<i>.norm<q>``,
``l<i>.ls<q>``, ``l<i>.hc<q>.{in,out,mix}``; ``l<i>.mix.*`` (``.mix.left.*`` and ``.mix.right.*`` in a parallel layer) and
``l<i>.mlp.*``. The weights of ``norm1``, ``norm2`` and ``final.norm`` are stored around zero."""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import LayerSpec, ModelConfig, ModelSpec, PartSpec, ScheduleEntry
from .registry import register_architecture

_MAMBA2 = ("heads", "vdim", "state", "groups", "conv", "norm_groups")
_LEFT = ("heads", "kv_heads", "dim", "vdim", "scale")
_RIGHT = ("heads", "dim", "vdim", "decay")
_MLPS = ("dense", "moe")


def _rot_problems(part: Dict[str, Any], side: str) -> List[str]:
    rot = part.get("rot")
    if not rot:
        return []
    dims = int(rot.get("dims", part["dim"]) or 0)
    out = []
    if dims and rot.get("base") is None:
        out.append(f"{side}: a rotation needs rot.base")
    if dims % 2 or not 0 <= dims <= int(part["dim"]):
        out.append(f"{side}: rot.dims must be even and at most dim, got {dims}")
    scaling = rot.get("scaling")
    if scaling and not float(scaling.get("factor", 0.0)) > 0:
        out.append(f"{side}: rot.scaling needs a positive factor")
    return out


@dataclass(frozen=True)
class ZavizenConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    streams: int = 1
    loop: Optional[Dict[str, int]] = None
    layers: Tuple[Dict[str, Any], ...] = field(default_factory=tuple)
    max_position_embeddings: int = 1 << 20

    architecture = "Zavizen"
    model_type = "zavizen"

    # the names other parts of the engine read from any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_json(cls, data: Dict[str, Any]) -> "ZavizenConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm", "streams") if data.get(k) is None]
        if missing:
            raise ValueError(f"Zavizen config.json lacks required keys: {missing}")
        if "eps" not in data["norm"]:
            raise ValueError("Zavizen config.json lacks norm.eps")
        loop = data.get("loop")
        if loop:
            lacking = [k for k in ("start", "stop", "times") if loop.get(k) is None]
            if lacking:
                raise ValueError(f"Zavizen config.json: loop lacks {lacking}")
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
        config = cls(vocab=int(data["vocab"]), width=int(data["width"]), norm_eps=float(data["norm"]["eps"]), streams=int(data["streams"]),
                     loop=loop or None, layers=tuple(copy.deepcopy(list(data["layers"]))),
                     max_position_embeddings=int(data.get("max_position_embeddings", 1 << 20)))
        config.validate()
        return config

    def validate(self) -> None:
        problems: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            problems.append(f"vocab and width must be positive, got {self.vocab} and {self.width}")
        if not self.norm_eps > 0:
            problems.append(f"norm.eps must be positive, got {self.norm_eps}")
        if self.streams <= 0:
            problems.append(f"streams must be positive, got {self.streams}")
        if not self.layers:
            problems.append("the model has no layers")
        if self.loop is not None:
            a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
            if not 0 <= a <= b <= len(self.layers) or n < 1:
                problems.append(f"loop must run layers of the model at least once, got {self.loop}")
        for i, layer in enumerate(self.layers):
            problems.extend(f"layer {i}: {p}" for p in self._layer_problems(layer))
        if problems:
            raise ValueError("invalid Zavizen configuration: " + "; ".join(problems))

    @staticmethod
    def _layer_problems(layer: Dict[str, Any]) -> List[str]:
        kind, m, mlp = layer.get("type"), layer.get("mixer") or {}, layer.get("mlp")
        out: List[str] = []
        if kind == "mamba2":
            lacking = [k for k in _MAMBA2 if m.get(k) is None]
            if lacking:
                return [f"the mamba2 mixer lacks {lacking}"]
            if int(m["heads"]) % int(m["groups"]):
                out.append(f"{m['heads']} heads cannot share {m['groups']} groups")
            if (int(m["heads"]) * int(m["vdim"])) % int(m["norm_groups"]):
                out.append("norm_groups must divide heads * vdim")
        elif kind == "parallel":
            left, right = m.get("left") or {}, m.get("right") or {}
            lacking = [f"left.{k}" for k in _LEFT if left.get(k) is None] + [f"right.{k}" for k in _RIGHT if right.get(k) is None]
            if lacking:
                return [f"the parallel mixer lacks {lacking}"]
            if int(left["heads"]) % int(left["kv_heads"]):
                out.append(f"{left['heads']} heads cannot share {left['kv_heads']} key/value heads")
            if len(right["decay"]) != int(right["heads"]):
                out.append(f"right.decay needs one constant per head, got {len(right['decay'])} for {right['heads']}")
            out.extend(_rot_problems(left, "left") + _rot_problems(right, "right"))
        else:
            return [f"unknown type {kind!r} (known: ['mamba2', 'parallel'])"]
        if mlp is not None:
            if mlp.get("kind") not in _MLPS:
                out.append(f"unknown mlp kind {mlp.get('kind')!r} (known: {list(_MLPS)})")
            elif mlp["kind"] == "dense":
                if mlp.get("ff") is None:
                    out.append("a dense mlp needs ff")
            else:
                expert, router, shared = mlp.get("expert") or {}, mlp.get("router") or {}, mlp.get("shared")
                if expert.get("ff") is None or router.get("experts") is None or router.get("top") is None:
                    out.append("routed experts need expert.ff, router.experts and router.top")
                elif not 0 < int(router["top"]) <= int(router["experts"]):
                    out.append(f"a token cannot use {router['top']} of {router['experts']} experts")
                else:
                    groups = router.get("groups")
                    if groups:
                        count, keep = int(groups.get("count", 0)), int(groups.get("keep", 0))
                        if count <= 0 or int(router["experts"]) % count or not 0 < keep <= count:
                            out.append(f"router.groups must cut the experts into equal groups and keep some of them, got {groups}")
                        elif keep * (int(router["experts"]) // count) < int(router["top"]):
                            out.append(f"{keep} groups of {int(router['experts']) // count} experts do not hold {router['top']}")
                if shared is not None and shared.get("ff") is None:
                    out.append("a shared expert needs shared.ff")
        return out

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "streams": self.streams, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = dict(self.loop)
        return out

    def eos_token_ids(self) -> List[int]:
        return []

    def parameter_counts(self) -> Dict[str, int]:
        from ..models import expected_params

        total = 0
        for spec in expected_params(self.model_spec()).values():
            if spec.optional:
                continue
            count = 1
            for n in spec.shape:
                count *= n if n is not None else 0
            total += count
        return {"total_parameters": total}

    def layer_order(self) -> List[int]:
        """The layers in the order they run, looped ones once per pass."""
        order = list(range(len(self.layers)))
        if self.loop is None:
            return order
        a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
        return order[:a] + order[a:b] * n + order[b:]

    @staticmethod
    def _position(part: Dict[str, Any], positions: Dict[str, PartSpec]) -> Dict[str, Any]:
        """The mixer arguments of its rotation; the encoding itself goes into ``positions``, once per distinct one."""
        rot = part.get("rot")
        dims = int(rot.get("dims", part["dim"]) or 0) if rot else 0
        if not dims:
            return {"position": None, "rotary_dim": 0}
        base, factor = float(rot["base"]), float((rot.get("scaling") or {}).get("factor", 1.0))
        name = f"rotary_{dims}_{base!r}_{factor!r}"
        positions.setdefault(name, PartSpec("rotary", {"rotary_dim": dims, "theta": base,
                                                       "frequency_scaling": {"kind": "linear", "factor": factor}}))
        return {"position": name, "rotary_dim": dims}

    def _mixer(self, layer: Dict[str, Any], p: str, positions: Dict[str, PartSpec]) -> PartSpec:
        D, m = self.width, layer["mixer"]
        if layer["type"] == "mamba2":
            return PartSpec("ssd", {"hidden_size": D, **{k: int(m[k]) for k in _MAMBA2}, "eps": self.norm_eps}, p)
        left, right = m["left"], m["right"]
        return PartSpec("side_by_side", {
            "left": {"kind": "capped_attention", "prefix": "left", "args": {
                "hidden_size": D, "num_heads": int(left["heads"]), "num_kv_heads": int(left["kv_heads"]), "dim": int(left["dim"]),
                "vdim": int(left["vdim"]), "scale": float(left["scale"]), "bias": False, "row_norm_eps": self.norm_eps,
                **self._position(left, positions)}},
            "right": {"kind": "retention", "prefix": "right", "args": {
                "hidden_size": D, "heads": int(right["heads"]), "dim": int(right["dim"]), "vdim": int(right["vdim"]),
                "decay": [float(a) for a in right["decay"]], "eps": self.norm_eps, **self._position(right, positions)}},
            "left_scale": 0.5, "right_scale": 0.5, "out_norm_eps": self.norm_eps, "out_norms": [f"{p}.left.out", f"{p}.right.out"],
            "hidden_size": D}, p)

    def _feed_forward(self, mlp: Optional[Dict[str, Any]], p: str) -> Optional[PartSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return PartSpec("swiglu", {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "float32_out": True,
                                       "names": {n: n for n in ("gate", "up", "down")}}, p)
        router, groups, shared = mlp["router"], mlp["router"].get("groups"), mlp.get("shared")
        scale = router.get("scale")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": int(mlp["expert"]["ff"]), "num_experts": int(router["experts"]),
            "top": int(router["top"]), "score": "softmax", "form": "silu", "normalize": True, "factor": 1.0 if scale is None else float(scale),
            "groups": (int(groups["count"]), int(groups["keep"])) if groups else None,
            "shared_size": int(shared["ff"]) if shared else None, "shared_gate": False}, p)

    def model_spec(self) -> ModelSpec:
        D, S = self.width, self.streams
        positions: Dict[str, PartSpec] = {}
        layers: List[LayerSpec] = []
        for i, layer in enumerate(self.layers):
            p, feed_forward = f"l{i}", self._feed_forward(layer.get("mlp"), f"l{i}.mlp")
            count = 1 if feed_forward is None else 2
            # a checkpoint may hold the second sublayer's small tensors for a layer without a feed-forward
            spare = {f"{p}.norm2": (D,), f"{p}.ls2": (D,), f"{p}.hc2.in": (S,), f"{p}.hc2.out": (S,), f"{p}.hc2.mix": (S, S)} if count == 1 else {}
            norms = {name: PartSpec("rms_norm", {"size": D, "eps": self.norm_eps, "name": f"{p}.norm{q}", "offset": 1.0})
                     for q, name in ((1, "mixer"), (2, "feed_forward"))[:count]}
            connections = [{"prefix": f"{p}.hc{q}", "streams": S, "size": D, "scale_name": f"{p}.ls{q}", "unused": spare}
                           for q in range(1, count + 1)]
            layers.append(LayerSpec(block="hyper_connected", mixer=self._mixer(layer, f"{p}.mix", positions), feed_forward=feed_forward,
                                    norms=norms, block_args={"connections": connections}))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": D, "name": "embed"}, "embed"),
            positions=positions, layers=tuple(layers),
            schedule=tuple(ScheduleEntry(layer, i) for i, layer in enumerate(self.layer_order())),
            final_norm=PartSpec("rms_norm", {"size": D, "eps": self.norm_eps, "name": "final.norm", "offset": 1.0}),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D, "name": "head"}, "head"),
            max_position=self.max_position_embeddings, streams=S,
        )
        spec.validate()
        return spec


register_architecture("Zavizen", ZavizenConfig)
