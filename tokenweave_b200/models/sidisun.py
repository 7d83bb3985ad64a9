"""Sidisun: a hybrid decoder of latent-attention and Mamba-2 layers with polynomial-norm feed-forwards and RMS norms on
the sublayers' outputs. The layers, their sizes and constants come from the checkpoint's ``config.json``:

``{"architecture": "Sidisun", "vocab", "width", "logit_scale", "norm": {"eps"}, "layers": [{"type", "mixer": {...},
"mlp": {"kind": "dense", "ff"} | null}, ...]}``
"""
from __future__ import annotations

from typing import Optional

from ..config import ModelConfig, register_config_reader
from .hybrid import HybridDecoder


class SidisunForCausalLM(HybridDecoder):
    architecture = "sidisun"


@register_config_reader("Sidisun")
def read_config(cfg: dict, name: str = "", path: Optional[str] = None) -> ModelConfig:
    layers = [dict(l) for l in cfg["layers"]]
    attn = next((l["mixer"] for l in layers if l["type"] == "latent_attention"), None)
    ff = next((l["mlp"]["ff"] for l in layers if l.get("mlp")), 0)
    # the configuration names no longest context: what the rotary scaling was made for, else the engine's default
    max_len = 8192
    for l in layers:
        s = (l["mixer"].get("rot") or {}).get("scaling")
        if s:
            max_len = max(max_len, int(s["original"] * s["factor"]))
    return ModelConfig(
        name=name or "sidisun", architecture="sidisun", hidden_size=cfg["width"], num_layers=len(layers),
        num_q_heads=attn["heads"] if attn else 1, num_kv_heads=1,
        head_dim=attn["dim"] + attn["rot_dim"] if attn else 1, intermediate_size=ff, vocab_size=cfg["vocab"],
        rms_norm_eps=float(cfg["norm"]["eps"]), logit_scale=float(cfg["logit_scale"]), layers=layers,
        max_model_len=max_len, path=path)
