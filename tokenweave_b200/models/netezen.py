"""Netezen: a decoder with hyper-connections (several residual streams), whose layers mix grouped-query attention over a
sliding window that keeps the first tokens with latent attention over a window with a learned sink, and whose
feed-forwards are dense (square of relu) or a mixture of clamped gated experts beside a shared one. The head is the
embedding table. Layers, sizes and constants come from ``config.json``:

``{"architecture": "Netezen", "vocab", "width", "norm": {"eps"}, "streams", "residual_mult", "layers": [{"type",
"mixer": {..., "rot": {"base", "dims", "scaling"}, "mask": {"size", "keep_first"}}, "mlp": {"kind": "dense", "ff"} |
{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}, "shared": {"ff", "limit"}} | null}, ...]}``
"""
from __future__ import annotations

from typing import Optional

from ..config import ModelConfig, register_config_reader
from .hybrid import HybridDecoder

GATE_SLOPE = 1.702           # of the experts' sigmoid
WEIGHT_SUM_EPS = 1e-20       # joins the sum of the chosen experts' scores


class NetezenForCausalLM(HybridDecoder):
    architecture = "netezen"


def _expert(spec: dict) -> dict:
    return {"ff": spec["ff"], "act": ("clamped", spec["limit"], GATE_SLOPE)}


def layer_spec(layer: dict) -> dict:
    """A layer as the configuration lists it -> mixers and feed-forwards with the options this design fixes."""
    kind, m = layer["type"], layer["mixer"]
    if kind == "attention":
        options = dict(rot=m["rot"], neighbour_pairs=True, window=m["mask"]["size"],
                       keep_first=m["mask"].get("keep_first", 0))
        out = {"type": "sum", "mixer": {"parts": {"": {"kind": "grouped_attention", "sizes": m, "options": options}}}}
    elif kind == "latent_attention":
        out = {"type": kind, "mixer": m, "options": dict(gated=False, sink=True, neighbour_pairs=True,
                                                         window=m["mask"]["size"])}
    else:
        raise ValueError(f"unknown mixer {kind!r} (known: attention, latent_attention)")
    mlp = layer.get("mlp")
    if mlp is not None:
        if mlp["kind"] == "dense":
            mlp = {"kind": "activated", "ff": mlp["ff"], "act": "relu2"}
        elif mlp["kind"] == "moe":
            shared = mlp.get("shared")
            mlp = {"kind": "routed", **mlp["router"], **_expert(mlp["expert"]), "sum_eps": WEIGHT_SUM_EPS,
                   "shared": _expert(shared) if shared else None}
        else:
            raise ValueError(f"unknown feed-forward {mlp['kind']!r} (known: dense, moe)")
    return {**out, "mlp": mlp}


def read(cfg: dict) -> dict:
    """Fields of :class:`ModelConfig` from a ``config.json`` of this design."""
    layers = cfg["layers"]
    m = layers[0]["mixer"]
    specs = [layer_spec(l) for l in layers]
    ff = [s["mlp"]["ff"] for s in specs if s["mlp"]]
    # the configuration names no longest context: what the rotary scaling was made for, else the engine's default
    scalings = [s for s in (l["mixer"]["rot"].get("scaling") for l in layers) if s]
    return dict(
        architecture="netezen", block="streams", streams=int(cfg["streams"]), residual_mult=float(cfg["residual_mult"]),
        norm_offset=1.0, tie_word_embeddings=True, hidden_size=cfg["width"], num_layers=len(layers),
        num_q_heads=m["heads"], num_kv_heads=m.get("kv_heads", 1), head_dim=m["dim"], intermediate_size=max(ff, default=0),
        vocab_size=cfg["vocab"], rms_norm_eps=float(cfg["norm"]["eps"]), layers=specs,
        max_model_len=max([8192] + [int(s["original"] * s["factor"]) for s in scalings]))


@register_config_reader("Netezen")
def read_config(cfg: dict, name: str = "", path: Optional[str] = None) -> ModelConfig:
    return ModelConfig(name=name or "netezen", path=path, **read(cfg))
