"""Typed configuration of the Zasudra decoder, read from its ``config.json``.

A small hybrid decoder. A sublayer reads the residual itself and its output is normed before it is added:
``x += m norm1(mixer(x))``, then ``x += m norm2(experts(x))``, with one factor m for the model (``residual_mult``). The token
embedding gains a row of a second table, chosen by a hash of the previous and the current token. A layer names its mixer
by ``type``:

* ``attention``: grouped key/value heads whose values are the projected keys, norms over the whole rows of q and k, the
  interleaved rotation of a part of every head, chunks of ``mask.size`` tokens, a learned sink per head;
* ``wkv``: a matrix state per head with a decay per key channel and token, fed from mixes of each token's input with
  the previous token's, a bonus for the current token and a gate;
* ``attention_2``: causal attention without rotation, norms over the whole rows of q and k, one added to the softmax's
  denominator and a sigmoid gate per head; with ``kv_from: j`` the layer reads the keys and values layer j cached.

The feed-forward is routed experts (squared ReLU, a router with bias, a softmax over the chosen logits), or absent
(``mlp`` null). Keys::

    {"architecture": "Zasudra", "vocab": V, "width": D, "norm": {"eps": e}, "residual_mult": m, "logit_scale": c,
     "embedding": {"bigram": {"buckets": B, "mul_prev": a, "mul_cur": b}},
     "layers": [{"type": "attention", "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k}},
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": s, "mask": {"size": n},
                           "rot": {"base": b, "dims": r}}},
                {"type": "wkv", "mlp": ..., "mixer": {"heads": H, "dim": d}},
                {"type": "attention_2", "mlp": ...,
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": v, "scale": s, "kv_from": j}}]}

Tensor names: ``embed``, ``bigram``, ``final.norm``, ``head``; per layer i ``l<i>.norm1``, ``.norm2`` (only with a
feed-forward), ``.mix.*`` and ``.mlp.*``."""

from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import LayerSpec, ModelConfig, ModelSpec, PartSpec, ScheduleEntry
from .registry import register_architecture

_NEEDS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale"), "wkv": ("heads", "dim"),
          "attention_2": ("heads", "kv_heads", "dim", "vdim", "scale")}


@dataclass(frozen=True)
class ZasudraConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    bigram: Optional[Dict[str, int]] = None
    layers: Tuple[Dict[str, Any], ...] = field(default_factory=tuple)
    max_position_embeddings: int = 1 << 20

    architecture = "Zasudra"
    model_type = "zasudra"

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
    def from_json(cls, data: Dict[str, Any]) -> "ZasudraConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if data.get(k) is None]
        if missing:
            raise ValueError(f"Zasudra config.json lacks required keys: {missing}")
        if "eps" not in data["norm"]:
            raise ValueError("Zasudra config.json lacks norm.eps")
        bigram = (data.get("embedding") or {}).get("bigram")
        if bigram is not None:
            lacking = [k for k in ("buckets", "mul_prev", "mul_cur") if bigram.get(k) is None]
            if lacking:
                raise ValueError(f"Zasudra config.json: embedding.bigram lacks {lacking}")
            bigram = {k: int(bigram[k]) for k in ("buckets", "mul_prev", "mul_cur")}
        mult, scale = data.get("residual_mult"), data.get("logit_scale")
        config = cls(vocab=int(data["vocab"]), width=int(data["width"]), norm_eps=float(data["norm"]["eps"]),
                     residual_mult=1.0 if mult is None else float(mult), logit_scale=1.0 if scale is None else float(scale),
                     bigram=bigram, layers=tuple(copy.deepcopy(list(data["layers"]))),
                     max_position_embeddings=int(data.get("max_position_embeddings", 1 << 20)))
        config.validate()
        return config

    def validate(self) -> None:
        problems: List[str] = []
        if self.vocab <= 0 or self.width <= 0:
            problems.append(f"vocab and width must be positive, got {self.vocab} and {self.width}")
        if not self.norm_eps > 0:
            problems.append(f"norm.eps must be positive, got {self.norm_eps}")
        if self.bigram is not None and self.bigram["buckets"] <= 0:
            problems.append(f"embedding.bigram.buckets must be positive, got {self.bigram['buckets']}")
        if not self.layers:
            problems.append("the model has no layers")
        for i, layer in enumerate(self.layers):
            problems.extend(f"layer {i}: {p}" for p in self._layer_problems(i, layer))
        if problems:
            raise ValueError("invalid Zasudra configuration: " + "; ".join(problems))

    def _layer_problems(self, i: int, layer: Dict[str, Any]) -> List[str]:
        kind, m, mlp = layer.get("type"), layer.get("mixer") or {}, layer.get("mlp")
        if kind not in _NEEDS:
            return [f"unknown type {kind!r} (known: {sorted(_NEEDS)})"]
        lacking = [k for k in _NEEDS[kind] if m.get(k) is None]
        if lacking:
            return [f"the {kind} mixer lacks {lacking}"]
        out: List[str] = []
        if kind != "wkv":
            if int(m["heads"]) % int(m["kv_heads"]):
                out.append(f"{m['heads']} heads cannot share {m['kv_heads']} key/value heads")
            size = (m.get("mask") or {}).get("size")
            if size is not None and int(size) <= 0:
                out.append(f"mask.size must be positive, got {size}")
        if kind == "attention":
            if int(m["vdim"]) != int(m["dim"]):
                out.append(f"the values are the keys, so vdim must equal dim, got {m['vdim']} and {m['dim']}")
            rot = m.get("rot")
            if rot is not None:
                if rot.get("base") is None:
                    out.append("a rotation needs rot.base")
                dims = int(rot.get("dims", m["dim"]))
                if dims % 2 or not 0 <= dims <= int(m["dim"]):
                    out.append(f"rot.dims must be even and at most dim, got {dims}")
        source = m.get("kv_from")
        if source is not None:
            j = int(source)
            other = self.layers[j] if 0 <= j < i else None
            om = (other or {}).get("mixer") or {}
            if kind != "attention_2" or other is None or other.get("type") != kind or om.get("kv_from") is not None:
                out.append(f"kv_from must name an earlier attention_2 layer with projections of its own, got {source}")
            elif any(om.get(k) != m.get(k) for k in ("kv_heads", "dim", "vdim")):
                out.append(f"kv_heads, dim and vdim must equal those of layer {j}")
            elif (om.get("mask") or {}).get("size") not in (None, (m.get("mask") or {}).get("size")):
                out.append(f"layer {j} keeps the keys of its own chunk alone, which is not what this layer sees")
        if mlp is not None:
            expert, router = mlp.get("expert") or {}, mlp.get("router") or {}
            if mlp.get("kind") != "moe":
                out.append(f"unknown mlp kind {mlp.get('kind')!r} (known: moe)")
            elif expert.get("ff") is None or router.get("experts") is None or router.get("top") is None:
                out.append("routed experts need expert.ff, router.experts and router.top")
            elif not 0 < int(router["top"]) <= int(router["experts"]):
                out.append(f"a token cannot use {router['top']} of {router['experts']} experts")
        return out

    def to_json(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                               "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}
        if self.bigram is not None:
            out["embedding"] = {"bigram": dict(self.bigram)}
        return out

    def eos_token_ids(self) -> List[int]:
        return []

    def parameter_counts(self) -> Dict[str, int]:
        from ..models import expected_params

        total = 0
        for spec in expected_params(self.model_spec()).values():
            count = 1
            for n in spec.shape:
                count *= n if n is not None else 0
            total += count
        return {"total_parameters": total}

    def _attention(self, m: Dict[str, Any], prefix: str, positions: Dict[str, PartSpec], first_kind: bool) -> PartSpec:
        size = (m.get("mask") or {}).get("size")
        args: Dict[str, Any] = {
            "hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]), "dim": int(m["dim"]),
            "vdim": int(m["vdim"]), "scale": float(m["scale"]), "chunk": int(size) if size else None, "bias": False,
            "row_norm_eps": self.norm_eps}
        if first_kind:
            args.update({"values": "keys", "sink": "learned"})
            rot = m.get("rot")
            dims = int(rot.get("dims", m["dim"])) if rot else 0
            if dims > 0:
                name = f"rotary_{dims}_{float(rot['base'])!r}"
                positions.setdefault(name, PartSpec("rotary", {"rotary_dim": dims, "theta": float(rot["base"])}))
                args.update({"position": name, "rotary_dim": dims, "interleaved": True})
        else:
            args.update({"sink": 0.0, "gate": "head", "own_rows": m.get("kv_from") is None})
        return PartSpec("capped_attention", args, prefix)

    def model_spec(self) -> ModelSpec:
        D = self.width
        positions: Dict[str, PartSpec] = {}
        layers: List[LayerSpec] = []
        schedule: List[ScheduleEntry] = []
        for i, layer in enumerate(self.layers):
            p, m, mlp = f"l{i}", layer["mixer"], layer.get("mlp")
            source = m.get("kv_from")
            if layer["type"] == "wkv":
                mixer = PartSpec("wkv", {"hidden_size": D, "heads": int(m["heads"]), "dim": int(m["dim"]), "eps": self.norm_eps}, f"{p}.mix")
            else:
                mixer = self._attention(m, f"{p}.mix", positions, layer["type"] == "attention")
            spare = [] if mlp is not None else [f"{p}.norm2"]           # a checkpoint may hold it for a layer without a feed-forward
            norms = {"mixer_out": PartSpec("rms_norm", {"size": D, "eps": self.norm_eps, "name": f"{p}.norm1", "gain": self.residual_mult,
                                                        "unused": spare})}
            feed_forward = None
            if mlp is not None:
                feed_forward = PartSpec("routed_experts", {
                    "hidden_size": D, "intermediate_size": int(mlp["expert"]["ff"]), "num_experts": int(mlp["router"]["experts"]),
                    "top": int(mlp["router"]["top"]), "score": "chosen_softmax", "form": "relu_squared", "router_bias": True}, f"{p}.mlp")
                norms["feed_forward_out"] = PartSpec("rms_norm", {"size": D, "eps": self.norm_eps, "name": f"{p}.norm2",
                                                                  "gain": self.residual_mult})
            layers.append(LayerSpec(block="output_norm_residual", mixer=mixer, feed_forward=feed_forward, norms=norms))
            schedule.append(ScheduleEntry(i, i, int(source) if source is not None else None))
        embedding: Dict[str, Any] = {"vocab_size": self.vocab, "hidden_size": D, "name": "embed"}
        if self.bigram is not None:
            embedding.update({"table_name": "bigram", **self.bigram})
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D,
            embedding=PartSpec("bigram_token_embedding" if self.bigram is not None else "token_embedding", embedding, "embed"),
            positions=positions, layers=tuple(layers), schedule=tuple(schedule),
            # the head is linear: the factor on the logits is the gain of the norm before it
            final_norm=PartSpec("rms_norm", {"size": D, "eps": self.norm_eps, "name": "final.norm", "gain": self.logit_scale}),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": D, "name": "head"}, "head"),
            max_position=self.max_position_embeddings,
        )
        spec.validate()
        return spec


register_architecture("Zasudra", ZasudraConfig)
