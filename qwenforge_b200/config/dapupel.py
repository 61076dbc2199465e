"""Typed configuration of the Dapupel decoder: several residual streams (hyper-connections) around layers that are listed one by
one, a Dynamic Tanh in every norm's place, a short causal convolution in front of every sublayer, a mixer that is one of three
kinds (a latent attention with a rotated key part, a gated delta rule with a decay per key channel, a windowed attention whose values
are its keys and whose positions enter as a distance bias) and a mixture of small experts (or no feed-forward). The logits come
from the embedding table.

config.json (every size and every constant that differs between models of the design is read from it):
  architecture      "Dapupel"
  vocab, width
  streams           residual streams
  norm.eps          eps of the latents' RMS norms and of the norm behind the delta rule (the Dynamic Tanh has none)
  canon.taps        taps of the convolution in front of every sublayer
  layers[i].type    "latent_attention": mixer {heads, dim, rot_dim, vdim, kv_rank, q_rank, scale,
                                               rot.{dims, base, scaling{factor, original, fast, slow} (optional)}}
                    "channel_delta":    mixer {heads, kv_heads, dim, vdim, conv}
                    "attention":        mixer {heads, kv_heads, dim, vdim, conv, scale, softcap, mask.size}
  layers[i].mlp     null | {kind: "moe", router{experts, top}, expert{ff, limit}}
The ranks of the delta rule's low-rank pairs (`a1`/`a2`, `g1`/`g2`) are read from the tensors; a mixer may name them (`rank`,
`gate_rank`), which the random-weights mode needs.
What the design fixes stands here as constants: the slope 1.702 of the experts' gate, sigmoid scores that are not renormalised and
multiply the expert's input, the tied output table.
A sequence has no longest length: nothing in the design depends on one.

Tensor names: embed, final.norm(.b, .alpha); per layer l<i>.norm1(.b, .alpha), l<i>.hc1.{in, out, mix}, l<i>.canon1, and with a
feed-forward the same with 2; latent_attention l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, o};
channel_delta l<i>.mix.{q, k, v}(.conv), l<i>.mix.{b, A_log, a1, a2, dt_bias, g1, g2, norm, o};
attention l<i>.mix.{q, k}(.conv), l<i>.mix.{r1, r2, g, o}; moe l<i>.mlp.router, l<i>.mlp.e<j>.{gate, up, down}.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Mapping

from .registry import ModelConfig, register_architecture
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

EXPERT_GATE_SLOPE = 1.702       # g * sigmoid(1.702 g) * (u + 1)
NO_LENGTH_LIMIT = 1 << 30       # what the runtime is told where it asks for a longest sequence


def _need(data: Mapping[str, Any], key: str, where: str = "config.json"):
    if not isinstance(data, Mapping) or key not in data or data[key] is None:
        raise ValueError(f"{where}: required key {key!r} is missing")
    return data[key]


def _positive(data, keys, where):
    for key in keys:
        if not float(_need(data, key, where)) > 0:
            raise ValueError(f"{where}: {key} must be positive")


def _check_mixer(kind, m, where):
    if kind == "latent_attention":
        _positive(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale"), where)
        rot = _need(m, "rot", where)
        _positive(rot, ("dims", "base"), where + ".rot")
        if int(m["rot_dim"]) % 2 or int(rot["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"{where}.rot: the rotated part is turned whole, dims = rot_dim (even)")
        if rot.get("scaling"):
            _positive(rot["scaling"], ("factor", "original", "fast", "slow"), where + ".rot.scaling")
        return
    if kind not in ("channel_delta", "attention"):
        raise ValueError(f"{where}: mixer type {kind!r} is not supported ('latent_attention', 'channel_delta', 'attention')")
    _positive(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
    if int(m["heads"]) % int(m["kv_heads"]):
        raise ValueError(f"{where}: kv_heads must divide heads")
    if kind == "attention":
        _positive(m, ("scale",), where)
        _positive(_need(m, "mask", where), ("size",), where + ".mask")
        if m.get("softcap"):
            _positive(m, ("softcap",), where)
        if int(m["vdim"]) != int(m["dim"]):
            raise ValueError(f"{where}: the values are the keys, so vdim is dim")


@dataclass(frozen=True)
class DapupelConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    eps: float
    taps: int
    layers: tuple          # the config's own layer entries (plain dicts), validated
    torch_dtype: str = "bfloat16"

    architecture = "Dapupel"
    model_type = "dapupel"

    @classmethod
    def from_dict(cls, data: Mapping[str, Any]) -> "DapupelConfig":
        layers = _need(data, "layers")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        config = cls(vocab=int(_need(data, "vocab")), width=int(_need(data, "width")), streams=int(_need(data, "streams")),
                     eps=float(_need(_need(data, "norm"), "eps", "config.json norm")),
                     taps=int(_need(_need(data, "canon"), "taps", "config.json canon")),
                     layers=tuple(copy.deepcopy(dict(layer)) for layer in layers),
                     torch_dtype=str(data.get("torch_dtype", data.get("dtype", "bfloat16"))))
        config.validate()
        return config

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.eps <= 0 or self.streams <= 0 or self.taps <= 0:
            raise ValueError("config.json: vocab, width, streams, norm.eps and canon.taps must be positive")
        for i, layer in enumerate(self.layers):
            where = f"config.json layers[{i}]"
            _check_mixer(_need(layer, "type", where), _need(layer, "mixer", where), where + ".mixer")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            where += ".mlp"
            if _need(mlp, "kind", where) != "moe":
                raise ValueError(f"{where}: kind {mlp['kind']!r} is not supported ('moe' or null)")
            router = _need(mlp, "router", where)
            experts, top = int(_need(router, "experts", where + ".router")), int(_need(router, "top", where + ".router"))
            _positive(_need(mlp, "expert", where), ("ff", "limit"), where + ".expert")
            if not 1 <= top <= experts:
                raise ValueError(f"{where}: 1 <= router.top <= router.experts is required")

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "norm": {"eps": self.eps}, "canon": {"taps": self.taps}, "layers": [copy.deepcopy(layer) for layer in self.layers],
                "torch_dtype": self.torch_dtype}

    def _dyt(self, name: str) -> PartSpec:
        return PartSpec("dynamic_tanh", {"width": self.width}, {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})

    def _mixer_spec(self, kind: str, m: Mapping[str, Any], p: str) -> PartSpec:
        sizes = {"hidden_size": self.width, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]), "value_dim": int(m["vdim"])}
        if kind == "latent_attention":
            dims = int(m["rot_dim"])
            position = PartSpec("rotary_interleaved", {"head_dim": dims, "rotary_dim": dims, "theta": float(m["rot"]["base"]), "precise": True,
                                                       "scaling": dict(m["rot"]["scaling"]) if m["rot"].get("scaling") else None})
            return PartSpec("latent_attention",
                            {**sizes, "kv_rank": int(m["kv_rank"]), "q_rank": int(m["q_rank"]), "scale": float(m["scale"]), "eps": self.eps,
                             "sinks": False, "rot_dim": dims, "position": position},
                            {"q_down": p + "dq", "q_norm": p + "dq.norm", "q_up": p + "uq", "kv_down": p + "dkv", "kv_norm": p + "dkv.norm",
                             "k_up": p + "uk", "v_up": p + "uv", "o_weight": p + "o"})
        if kind == "channel_delta":
            tensors = {n + "_weight": p + n for n in ("q", "k", "v", "b", "o")}
            tensors.update({n + "_conv": p + n + ".conv" for n in ("q", "k", "v")})
            tensors.update({"rate_log": p + "A_log", "a1": p + "a1", "a2": p + "a2", "dt_bias": p + "dt_bias", "g1": p + "g1", "g2": p + "g2",
                            "norm": p + "norm"})
            return PartSpec("channel_delta", {**sizes, "num_kv_heads": int(m["kv_heads"]), "conv_taps": int(m["conv"]), "eps": self.eps,
                                              "rank": m.get("rank"), "gate_rank": m.get("gate_rank")}, tensors)
        return PartSpec("gqa_attention",
                        {**sizes, "num_kv_heads": int(m["kv_heads"]), "qkv_bias": False, "out_bias": False, "scale": float(m["scale"]),
                         "window": int(m["mask"]["size"]), "position": None, "softcap": float(m.get("softcap") or 0.0),
                         "conv_taps": int(m["conv"]), "shared_values": True, "distance_bias": True, "out_gate": True},
                        {"q_weight": p + "q", "k_weight": p + "k", "o_weight": p + "o", "q_conv": p + "q.conv", "k_conv": p + "k.conv",
                         "bias_scale": p + "r1", "bias_rate": p + "r2", "g_weight": p + "g"})

    def _feed_forward_spec(self, mlp: Mapping[str, Any], p: str) -> PartSpec:
        experts = int(mlp["router"]["experts"])
        tensors = {"router": p + "router"}
        for e in range(experts):
            for which in ("gate", "up", "down"):
                tensors[f"{which}.{e}"] = f"{p}e{e}.{which}"
        return PartSpec("routed_experts",
                        {"hidden_size": self.width, "expert_size": int(mlp["expert"]["ff"]), "experts": experts,
                         "top": int(mlp["router"]["top"]), "score": "sigmoid", "renormalize": False, "weight_on": "input",
                         "gate": "clamped", "limit": float(mlp["expert"]["limit"]), "alpha": EXPERT_GATE_SLOPE},
                        tensors)

    def model_spec(self) -> ModelSpec:
        layers, ignored = [], []
        for i, layer in enumerate(self.layers):
            p = f"l{i}."
            parts = {"mixer": self._mixer_spec(layer["type"], layer["mixer"], p + "mix.")}
            if layer.get("mlp") is not None:
                parts["feed_forward"] = self._feed_forward_spec(layer["mlp"], p + "mlp.")
            for which, name in ((1, "mixer"), (2, "feed_forward")):
                around = {name + "_norm": self._dyt(f"{p}norm{which}"),
                          name + "_streams": PartSpec("stream_mix", {"streams": self.streams},
                                                      {k: f"{p}hc{which}.{k}" for k in ("in", "out", "mix")}),
                          name + "_input": PartSpec("input_convolution", {"width": self.width, "taps": self.taps}, {"weight": f"{p}canon{which}"})}
                if name in parts:
                    parts.update(around)
                else:   # a file may still carry them
                    ignored += [t for part in around.values() for t in part.tensors.values()]
            layers.append(LayerSpec("streams", parts))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=self.width, max_positions=NO_LENGTH_LIMIT,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "width": self.width}, {"weight": "embed"}),
            layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))), final_norm=self._dyt("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "width": self.width, "tied": True}, {"weight": "embed"}),
            ignored_tensors=tuple(ignored))
        spec.validate()
        return spec


register_architecture(DapupelConfig.architecture, DapupelConfig, DapupelConfig.model_type)
