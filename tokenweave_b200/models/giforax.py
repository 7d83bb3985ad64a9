"""Giforax: a decoder whose sublayers stand between two layer norms, and whose layers pass on a weighted sum of all results so
far, the embedding output among them. Its mixers are a grouped-query attention with sigmoid weights inside chunks of positions
- some layers read the keys and values of an earlier one - and a minGRU; its feed-forwards are a mixture of clamped gated
experts, the routing weight on the expert's input, beside a shared one. Layers, sizes and constants come from ``config.json``:

``{"architecture": "Giforax", "vocab", "width", "norm": {"eps"}, "embedding": {"scale"}, "layers": [{"type", "mixer": {"heads",
"kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"}, "mask": {"size"}, "kv_from"} | {"width"}, "mlp": {"kind": "moe",
"router": {"experts", "top"}, "expert": {"ff", "limit"}, "shared": {"ff", "limit"}} | null}, ...]}``
"""
from __future__ import annotations

from typing import Optional

from ..config import ModelConfig, register_config_reader
from .hybrid import HybridDecoder

GATE_SLOPE = 1.702           # of the experts' sigmoid


class GiforaxForCausalLM(HybridDecoder):
    architecture = "giforax"


def _expert(spec: dict) -> dict:
    return {"ff": spec["ff"], "act": ("clamped", spec["limit"], GATE_SLOPE)}


def layer_spec(layer: dict) -> dict:
    """A layer as the configuration lists it -> mixers and feed-forwards with the options this design fixes."""
    kind, m = layer["type"], layer["mixer"]
    if kind == "attention":
        options = dict(rot=m["rot"], qk_norm="unit", weights="sigmoid", chunk=m["mask"]["size"], head_gate=True,
                       kv_from=m.get("kv_from"))
        out = {"type": "sum", "mixer": {"parts": {"": {"kind": "grouped_attention", "sizes": m, "options": options}}}}
    elif kind == "mingru":
        out = {"type": kind, "mixer": m}
    else:
        raise ValueError(f"unknown mixer {kind!r} (known: attention, mingru)")
    mlp = layer.get("mlp")
    if mlp is not None:
        if mlp["kind"] != "moe":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r} (known: moe)")
        shared = mlp.get("shared")
        mlp = {"kind": "routed", **mlp["router"], **_expert(mlp["expert"]), "scores": "sigmoid", "normalize": False,
               "correction": False, "weigh": "input", "shared": {**_expert(shared), "gated": False} if shared else None}
    return {**out, "mlp": mlp}


def read(cfg: dict) -> dict:
    """Fields of :class:`ModelConfig` from a ``config.json`` of this design."""
    layers = cfg["layers"]
    specs = [layer_spec(l) for l in layers]
    attn = next((l["mixer"] for l in layers if l["type"] == "attention"), None)
    ff = [s["mlp"]["ff"] for s in specs if s["mlp"]]
    # the configuration names no longest context: the engine's default
    return dict(
        architecture="giforax", block="sandwich", norm="layer", depth_average=True,
        embed_scale=float(cfg["embedding"]["scale"]), hidden_size=cfg["width"], num_layers=len(layers),
        num_q_heads=attn["heads"] if attn else 1, num_kv_heads=attn["kv_heads"] if attn else 1,
        head_dim=attn["dim"] if attn else 1, intermediate_size=max(ff, default=0), vocab_size=cfg["vocab"],
        rms_norm_eps=float(cfg["norm"]["eps"]), layers=specs)


@register_config_reader("Giforax")
def read_config(cfg: dict, name: str = "", path: Optional[str] = None) -> ModelConfig:
    return ModelConfig(name=name or "giforax", path=path, **read(cfg))
