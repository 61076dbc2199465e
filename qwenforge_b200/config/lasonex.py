"""Typed configuration of the Lasonex decoder: layers listed one by one, each with two sublayers side by side on the same stream, a norm for
each, `x += mixer(rms_1(x)) + ff(rms_2(x))`, a mixer that is one of two kinds (a windowed differential attention; a retention with a fixed
decay per head) and a feed-forward with clamped halves that is dense, a mixture of small experts chosen among groups, or absent.

config.json (every size and every constant that differs between models of the design is read from it):
  architecture      "Lasonex"
  vocab, width
  embedding.scale   factor on the embedding's rows
  norm.eps          eps of every RMS norm and unit norm
  layers[i].type    "attention": mixer {heads, kv_heads, dim (of one map), vdim, scale, diff, mask.size,
                                        rot.{dims, base, scaling{factor, original, fast, slow} (optional)}}
                    "retention": mixer {heads, dim, vdim, decay (one number per head), rot.{dims, base}}
  layers[i].mlp     null | {kind: "dense", ff, limit}
                         | {kind: "moe", router{experts, top, groups{count, keep} (optional)}, expert{ff, limit}}
What the design fixes stands here as constants: the slope 1.702 of the gates, softmax scores over all experts that are renormalised over
the chosen, a group's score being its largest.
A sequence has no longest length: nothing in the design depends on one.

Tensor names: embed, final.norm, head; per layer l<i>.norm1, l<i>.norm2, l<i>.mix.{q, k, v, o}; attention l<i>.mix.{lq1, lk1, lq2, lk2};
retention l<i>.mix.g; dense l<i>.mlp.{gate, up, down}; moe l<i>.mlp.router, l<i>.mlp.e<j>.{gate, up, down}.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .registry import ModelConfig, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

GATE_SLOPE = 1.702              # g * sigmoid(1.702 g) * (u + 1)
GROUP_BEST = 1                  # a group's score is its largest one
NO_LENGTH_LIMIT = 1 << 30       # what the runtime is told where it asks for a longest sequence


def _need(data: Mapping[str, Any], key: str, where: str = "config.json"):
    if not isinstance(data, Mapping) or key not in data or data[key] is None:
        raise ValueError(f"{where}: required key {key!r} is missing")
    return data[key]


def _positive(data, keys, where):
    for key in keys:
        if not float(_need(data, key, where)) > 0:
            raise ValueError(f"{where}: {key} must be positive")


@dataclass(frozen=True)
class LasonexConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple          # the config's own layer entries (plain dicts), validated
    torch_dtype: str = "bfloat16"

    architecture = "Lasonex"
    model_type = "lasonex"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "LasonexConfig":
        layers = _need(data, "layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab=int(_need(data, "vocab")), width=int(_need(data, "width")),
                     eps=float(_need(_need(data, "norm"), "eps", "config.json norm")),
                     embedding_scale=float(_need(_need(data, "embedding"), "scale", "config.json embedding")),
                     layers=tuple(copy.deepcopy(dict(layer)) for layer in layers),
                     torch_dtype=str(data.get("torch_dtype", data.get("dtype", "bfloat16"))))
        config.validate()
        return config

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.eps <= 0:
            raise ValueError("config.json: vocab, width and norm.eps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"config.json layers[{i}]"
            kind, mixer = _need(layer, "type", where), _need(layer, "mixer", where)
            where += ".mixer"
            if kind not in ("attention", "retention"):
                raise ValueError(f"config.json layers[{i}]: mixer type {kind!r} is not supported ('attention', 'retention')")
            _positive(mixer, ("heads", "dim", "vdim"), where)
            rot = _need(mixer, "rot", where)
            if int(_need(rot, "dims", where + ".rot")) % 2 or not 0 <= int(rot["dims"]) <= int(mixer["dim"]):
                raise ValueError(f"{where}.rot: dims must be even and at most dim")
            if int(rot["dims"]):
                _positive(rot, ("base",), where + ".rot")
            if rot.get("scaling"):
                _positive(rot["scaling"], ("factor", "original", "fast", "slow"), where + ".rot.scaling")
            if kind == "attention":
                _positive(mixer, ("kv_heads", "scale"), where)
                float(_need(mixer, "diff", where))
                _positive(_need(mixer, "mask", where), ("size",), where + ".mask")
                if int(mixer["heads"]) % int(mixer["kv_heads"]):
                    raise ValueError(f"{where}: kv_heads must divide heads")
            elif len(_need(mixer, "decay", where)) != int(mixer["heads"]):
                raise ValueError(f"{where}: decay must list one number per head")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            where = f"config.json layers[{i}].mlp"
            if _need(mlp, "kind", where) == "dense":
                _positive(mlp, ("ff", "limit"), where)
            elif mlp["kind"] == "moe":
                router = _need(mlp, "router", where)
                experts, top = int(_need(router, "experts", where + ".router")), int(_need(router, "top", where + ".router"))
                _positive(_need(mlp, "expert", where), ("ff", "limit"), where + ".expert")
                if not 1 <= top <= experts:
                    raise ValueError(f"{where}: 1 <= router.top <= router.experts is required")
                groups = router.get("groups")
                if groups:
                    count, keep = int(_need(groups, "count", where + ".router.groups")), int(_need(groups, "keep", where + ".router.groups"))
                    if not 1 <= keep <= count or experts % count or keep * (experts // count) < top:
                        raise ValueError(f"{where}.router.groups: count must divide the experts, and the kept groups must hold `top` experts")
            else:
                raise ValueError(f"{where}: kind {mlp['kind']!r} is not supported ('dense', 'moe' or null)")

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
                "norm": {"eps": self.eps}, "layers": [copy.deepcopy(layer) for layer in self.layers], "torch_dtype": self.torch_dtype}

    def _rotary(self, m) -> PartSpec | None:
        rot = m["rot"]
        if not int(rot["dims"]):
            return None
        return PartSpec("rotary_half", {"head_dim": int(m["dim"]), "rotary_dim": int(rot["dims"]), "theta": float(rot["base"]), "precise": True,
                                        "scaling": dict(rot["scaling"]) if rot.get("scaling") else None})

    def _mixer_spec(self, kind: str, m: Mapping[str, Any], p: str) -> PartSpec:
        params = {"hidden_size": self.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "eps": self.eps,
                  "position": self._rotary(m)}
        tensors = {s + "_weight": p + s for s in "qkvo"}
        if kind == "retention":
            params["decay"] = tuple(float(d) for d in m["decay"])
            tensors["g_weight"] = p + "g"
            return PartSpec("retention", params, tensors)
        params.update({"num_kv_heads": int(m["kv_heads"]), "scale": float(m["scale"]), "window": int(m["mask"]["size"]), "offset": float(m["diff"])})
        tensors.update({name: p + name for name in ("lq1", "lk1", "lq2", "lk2")})
        return PartSpec("differential_attention", params, tensors)

    def _feed_forward_spec(self, mlp: Mapping[str, Any], p: str) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("clamped_glu", {"hidden_size": self.width, "intermediate_size": int(mlp["ff"]), "limit": float(mlp["limit"]),
                                            "alpha": GATE_SLOPE},
                            {"gate_weight": p + "gate", "up_weight": p + "up", "down_weight": p + "down"})
        router = mlp["router"]
        experts, groups = int(router["experts"]), router.get("groups")
        tensors = {"router": p + "router"}
        for e in range(experts):
            for which in ("gate", "up", "down"):
                tensors[f"{which}.{e}"] = f"{p}e{e}.{which}"
        return PartSpec("routed_experts",
                        {"hidden_size": self.width, "expert_size": int(mlp["expert"]["ff"]), "experts": experts, "top": int(router["top"]),
                         "score": "softmax", "renormalize": True, "weight_on": "output", "gate": "clamped",
                         "limit": float(mlp["expert"]["limit"]), "alpha": GATE_SLOPE, "group_best": GROUP_BEST,
                         "groups": (int(groups["count"]), int(groups["keep"])) if groups else None},
                        tensors)

    def model_spec(self) -> ModelSpec:
        def norm(name: str) -> PartSpec:
            return PartSpec("rms_norm", {"width": self.width, "eps": self.eps}, {"weight": name})

        layers, ignored = [], []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            parts = {"norm": norm(p + "norm1"), "mixer": self._mixer_spec(layer["type"], layer["mixer"], p + "mix.")}
            if layer.get("mlp") is None:
                ignored.append(p + "norm2")   # a file may still carry it
            else:
                parts["feed_forward_norm"] = norm(p + "norm2")
                parts["feed_forward"] = self._feed_forward_spec(layer["mlp"], p + "mlp.")
            layers.append(LayerSpec("parallel", parts))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=NO_LENGTH_LIMIT,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "width": self.width, "scale": self.embedding_scale},
                               {"weight": "embed"}),
            layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "width": self.width, "tied": False}, {"weight": "head"}),
            ignored_tensors=tuple(ignored))
        spec.validate()
        return spec


register_architecture(LasonexConfig.architecture, LasonexConfig, LasonexConfig.model_type)
