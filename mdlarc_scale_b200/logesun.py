"""The Logesun design: how its ``config.json`` and tensor names map to a layered model.

A decoder-only model with a norm before and after every sublayer.  Its attention caches a small latent and one
rotated key part per token (shared by all heads); per-head keys and values are linear maps of the latent, queries go
through a latent of their own.  Every layer sees a window and has a sink per head in the softmax denominator.
Feed-forwards are gated linear units, or mixtures of clamped ones whose routing score multiplies the expert's input,
beside a shared expert.  A range of layers runs several times with the same weights, the embedding added ahead of
every pass but the first.
"""
from __future__ import annotations

from .layered import LayeredEngine, LayerSpec, ModelSpec
from .registry import collect_tensors, register

_LATENT = {"DQ": "dq", "DQ_NORM": "dq.norm", "UQ": "uq", "DKV": "dkv", "DKV_NORM": "dkv.norm", "UK": "uk", "UV": "uv",
           "SINK": "sink", "O": "o"}


def layer_spec(entry: dict) -> LayerSpec:
    mixer, kind = entry["mixer"], entry["type"]
    if kind != "latent_attention":
        raise ValueError(f"unknown mixer {kind!r}")
    rot, mask = mixer["rot"], mixer.get("mask")
    return LayerSpec(mixer="latent", heads=int(mixer["heads"]), kv_heads=int(mixer["heads"]), dim=int(mixer["dim"]),
                     vdim=int(mixer["vdim"]), sink=True, scale=float(mixer["scale"]), window=0 if mask is None else int(mask["size"]),
                     q_rank=int(mixer["q_rank"]), kv_rank=int(mixer["kv_rank"]), rot_dim=int(mixer["rot_dim"]),
                     rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), **feed_forward(entry.get("mlp")))


def feed_forward(mlp: dict | None) -> dict:
    if mlp is None:
        return {}
    if mlp["kind"] == "dense":
        return dict(mlp="glu", glu="silu", d_ff=int(mlp["ff"]))
    if mlp["kind"] == "moe":
        shared = mlp.get("shared") or {"ff": 0, "limit": 0.0}
        return dict(mlp="moe", glu="clamped", d_ff=int(mlp["expert"]["ff"]), glu_limit=float(mlp["expert"]["limit"]),
                    experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), shared_ff=int(shared["ff"]),
                    shared_limit=float(shared["limit"]))
    raise ValueError(f"unknown feed-forward {mlp['kind']!r}")


def model_spec(config: dict) -> ModelSpec:
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 1}
    return ModelSpec(width=int(config["width"]), vocab=int(config["vocab"]), norm="rms", norm_eps=float(config["norm"]["eps"]),
                     norm_place="sandwich", loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])),
                     layers=[layer_spec(e) for e in config["layers"]])


def tensor_names(spec: ModelSpec) -> dict[tuple[str, int], str | list[str]]:
    """(tensor kind, layer) -> name in the checkpoint; a list of names is stacked."""
    names = {("EMBED", 0): "embed", ("FINAL_NORM", 0): "final.norm", ("HEAD", 0): "head"}
    for n, layer in enumerate(spec.layers):
        p = f"l{n}"
        names.update({(kind, n): f"{p}.mix.{suffix}" for kind, suffix in _LATENT.items()})
        names.update({("NORM1", n): f"{p}.norm1", ("NORM1B", n): f"{p}.norm1b"})
        if layer.mlp is not None:
            names.update({("NORM2", n): f"{p}.norm2", ("NORM2B", n): f"{p}.norm2b"})
        if layer.mlp == "glu":
            names.update({(part.upper(), n): f"{p}.mlp.{part}" for part in ("gate", "up", "down")})
        if layer.mlp == "moe":
            names[("ROUTER", n)] = f"{p}.mlp.router"
            for part in ("gate", "up", "down"):
                names[("EXPERT_" + part.upper(), n)] = [f"{p}.mlp.e{e}.{part}" for e in range(layer.experts)]
                if layer.shared_ff:
                    names[("SHARED_" + part.upper(), n)] = f"{p}.mlp.shared.{part}"
    return names


@register("Logesun")
def build(config: dict, tensors: dict, device="cuda:0", act_format: str = "f16", **options) -> LayeredEngine:
    spec = model_spec(config)
    return LayeredEngine(spec, collect_tensors(tensor_names(spec), tensors), device, act_format, **options)
