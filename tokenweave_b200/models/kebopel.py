"""Kebopel: a decoder of parallel blocks (mixer and feed-forward read one norm and are added together), some of whose layers
run several times in a row. Its mixers are a grouped-query attention with a short convolution of queries, keys and values
and a query temperature, and a pair of an attention with distance biases and a sink beside a lightning attention. A table
of token-pair embeddings is added to the token embeddings. Layers, sizes and constants come from ``config.json``:

``{"architecture": "Kebopel", "vocab", "width", "norm": {"eps"}, "embedding": {"bigram": {"buckets", "mul_prev",
"mul_cur"}}, "loop": {"start", "stop", "times"}, "layers": [{"type", "mixer": {...}, "mlp": {"kind": "dense", "ff"} |
null}, ...]}``
"""
from __future__ import annotations

from typing import Optional

from ..config import ModelConfig, register_config_reader
from .hybrid import HybridDecoder


class KebopelForCausalLM(HybridDecoder):
    architecture = "kebopel"


def layer_spec(layer: dict) -> dict:
    """A layer as the configuration lists it -> the parts, with the options this design fixes."""
    kind, m = layer["type"], layer["mixer"]
    if kind == "attention":
        parts = {"": {"kind": "grouped_attention", "sizes": m,
                      "options": dict(bias=True, conv=m["conv"], qk_norm="head", q_temp=m["q_temp"])}}
    elif kind == "parallel":
        parts = {"left": {"kind": "grouped_attention", "sizes": m["left"],
                          "options": dict(qk_norm="whole", distance_bias=True, sink=True, out_scale=m["left_scale"])},
                 "right": {"kind": "lightning_attention", "sizes": m["right"],
                           "options": dict(out_scale=m["right_scale"])}}
    else:
        raise ValueError(f"unknown mixer {kind!r} (known: attention, parallel)")
    mlp = layer.get("mlp")
    if mlp is not None:
        if mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward {mlp['kind']!r} (known: dense)")
        mlp = {"kind": "gated", "ff": mlp["ff"], "act": "gelu_tanh"}
    return {"type": "sum", "mixer": {"parts": parts}, "mlp": mlp}


def read(cfg: dict) -> dict:
    """Fields of :class:`ModelConfig` from a ``config.json`` of this design."""
    first = cfg["layers"][0]["mixer"]
    first = first.get("left", first)
    return dict(
        architecture="kebopel", block="parallel", hidden_size=cfg["width"], num_layers=len(cfg["layers"]),
        num_q_heads=first["heads"], num_kv_heads=first["kv_heads"], head_dim=first["dim"],
        intermediate_size=next((l["mlp"]["ff"] for l in cfg["layers"] if l.get("mlp")), 0), vocab_size=cfg["vocab"],
        rms_norm_eps=float(cfg["norm"]["eps"]), layers=[layer_spec(l) for l in cfg["layers"]], loop=cfg.get("loop"),
        bigram=(cfg.get("embedding") or {}).get("bigram"))


@register_config_reader("Kebopel")
def read_config(cfg: dict, name: str = "", path: Optional[str] = None) -> ModelConfig:
    # positions are not bounded by the design (no rotation, no table): the engine's default context
    return ModelConfig(name=name or "kebopel", path=path, **read(cfg))
