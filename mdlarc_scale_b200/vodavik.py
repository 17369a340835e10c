"""The Vodavik design: how its ``config.json`` and tensor names map to a layered model.

A decoder-only model whose residual stream is normed AFTER every sum (centred norm, gain only, the
residual weighted by ``postln_alpha``), mixing softmax-attention layers and mLSTM layers in any order,
each with or without a feed-forward.  Its attention has no positional rotation: per-head RMS norms of
queries and keys, a query gain that grows with the logarithm of the position, a learned sink per head in
the softmax denominator, an output gate, grouped key/value heads, and layers that read another layer's
keys and values.
"""
from __future__ import annotations

from .layered import LayeredEngine, LayerSpec, ModelSpec
from .registry import collect_tensors, register

_ATTENTION = {"Q": "q", "Q_B": "q.b", "G": "g", "O": "o", "Q_NORM": "q.norm", "SINK": "sink"}
_ATTENTION_KV = {"K": "k", "K_B": "k.b", "V": "v", "V_B": "v.b", "K_NORM": "k.norm"}
_MLSTM = {"Q": "q", "K": "k", "V": "v", "G": "g", "O": "o", "HEAD_NORM": "norm",
          "I": "i", "I_B": "i.b", "F": "f", "F_B": "f.b"}


def _whole(value, name: str) -> int:
    if int(value) != value:
        raise ValueError(f"{name} must be a whole number, not {value!r}")
    return int(value)


def layer_spec(entry: dict) -> LayerSpec:
    mixer, kind = entry["mixer"], entry["type"]
    mlp = entry.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"unknown feed-forward {mlp['kind']!r}")
    common = dict(heads=int(mixer["heads"]), dim=int(mixer["dim"]), vdim=int(mixer["vdim"]),
                  mlp=None if mlp is None else "relu2", d_ff=0 if mlp is None else int(mlp["ff"]))
    if kind == "attention":
        temp = mixer.get("q_temp") or {"coef": 0.0, "every": 0}
        kv_from = mixer.get("kv_from")
        return LayerSpec(mixer="attention", kv_heads=int(mixer["kv_heads"]), kv_from=-1 if kv_from is None else int(kv_from),
                         qkv_bias=True, qk_norm=True, sink=True, out_gate=True, scale=float(mixer["scale"]),
                         q_temp_coef=float(temp["coef"]), q_temp_every=_whole(temp["every"], "q_temp.every"), **common)
    if kind == "mlstm":
        return LayerSpec(mixer="mlstm", kv_heads=int(mixer["heads"]), out_gate=True, gate_cap=float(mixer["gate_cap"]), **common)
    raise ValueError(f"unknown mixer {kind!r}")


def model_spec(config: dict) -> ModelSpec:
    return ModelSpec(width=int(config["width"]), vocab=int(config["vocab"]), norm="layer",
                     norm_eps=float(config["norm"]["eps"]), residual_alpha=float(config["postln_alpha"]),
                     logit_scale=float(config["logit_scale"]), layers=[layer_spec(e) for e in config["layers"]])


def tensor_names(spec: ModelSpec) -> dict[tuple[str, int], str]:
    """(tensor kind, layer) -> name in the checkpoint."""
    names = {("EMBED", 0): "embed", ("FINAL_NORM", 0): "final.norm", ("HEAD", 0): "head"}
    for n, layer in enumerate(spec.layers):
        if layer.mixer == "attention":
            mix = dict(_ATTENTION, **(_ATTENTION_KV if layer.kv_from < 0 else {}))
        else:
            mix = _MLSTM
        names.update({(kind, n): f"l{n}.mix.{suffix}" for kind, suffix in mix.items()})
        names[("NORM1", n)] = f"l{n}.norm1"
        if layer.mlp is not None:
            names.update({("NORM2", n): f"l{n}.norm2", ("UP", n): f"l{n}.mlp.up", ("DOWN", n): f"l{n}.mlp.down"})
    return names


@register("Vodavik")
def build(config: dict, tensors: dict, device="cuda:0", act_format: str = "f16", **options) -> LayeredEngine:
    spec = model_spec(config)
    return LayeredEngine(spec, collect_tensors(tensor_names(spec), tensors), device, act_format, **options)
