"""Decoders described layer by layer.

Most configurations give one set of sizes for all layers.  A *plan* gives every layer its own: which mixer
it has, the mixer's sizes and constants, and whether a feed-forward follows.  It is kept on
``ModelConfig.layer_plan`` as a list of ``{"mixer": kind, "mlp": bool, "over": {...}}`` where ``over`` holds
``ModelConfig`` fields of that layer (``ModelConfig.layer_config(i)`` applies them), so that the mixers read
a plain ``ModelConfig`` whether or not the model has a plan.

This module turns the configuration format of the Vofelix decoder into such a plan."""
from __future__ import annotations

from typing import Any, Callable, Optional


def _yarn(scaling: Optional[dict]) -> Optional[dict]:
    if not scaling:
        return None
    return {"rope_type": "yarn_interp", "factor": float(scaling["factor"]),
            "original_max_position_embeddings": float(scaling["original"]),
            "beta_fast": float(scaling["fast"]), "beta_slow": float(scaling["slow"])}


def _latent(m: dict) -> dict:
    rot = m["rot"]
    if int(rot["dims"]) != int(m["rot_dim"]):
        raise ValueError("latent attention rotates the whole rotary part: rot.dims must equal rot_dim")
    return dict(num_attention_heads=int(m["heads"]), num_key_value_heads=int(m["heads"]),
                qk_nope_head_dim=int(m["dim"]), qk_rope_head_dim=int(m["rot_dim"]), v_head_dim=int(m["vdim"]),
                head_dim=int(m["dim"]) + int(m["rot_dim"]), kv_lora_rank=int(m["kv_rank"]), q_lora_rank=None,
                rope_theta=float(rot["base"]), rope_scaling=_yarn(rot.get("scaling")),
                attention_multiplier=float(m["scale"]), attention_sink=True,
                sliding_window=int(m["mask"]["size"]) if m.get("mask") else None)


def _delta(m: dict) -> dict:
    return dict(linear_num_key_heads=int(m["kv_heads"]), linear_num_value_heads=int(m["heads"]),
                linear_key_head_dim=int(m["dim"]), linear_value_head_dim=int(m["vdim"]),
                linear_conv_kernel_dim=int(m["conv"]))


_VOFELIX_MIXERS: dict[str, tuple[str, Callable[[dict], dict]]] = {
    "latent_attention": ("latent", _latent), "delta": ("delta", _delta)}


def vofelix_fields(d: dict) -> dict[str, Any]:
    """``ModelConfig`` fields of a Vofelix configuration."""
    plan, kinds = [], []
    for i, layer in enumerate(d["layers"]):
        if layer["type"] not in _VOFELIX_MIXERS:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        mixer, read = _VOFELIX_MIXERS[layer["type"]]
        over = read(layer["mixer"])
        mlp = layer.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            over["intermediate_size"] = int(mlp["ff"])
        plan.append({"mixer": mixer, "mlp": mlp is not None, "over": over})
        kinds.append("linear_attention" if mixer == "delta" else "full_attention")
    loop = d.get("loop")
    if loop:
        loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
        if not (0 <= loop[0] < loop[1] <= len(plan)) or loop[2] < 1:
            raise ValueError(f"loop {loop} does not fit {len(plan)} layers")
    width = int(d["width"])

    def largest(name: str, default: int) -> int:
        return max([default] + [p["over"].get(name) or 0 for p in plan])
    heads = largest("num_attention_heads", 0) or largest("linear_num_value_heads", 1)
    fields: dict[str, Any] = dict(
        vocab_size=int(d["vocab"]), hidden_size=width, num_hidden_layers=len(plan), layer_plan=plan,
        layer_loop=tuple(loop) if loop else None, layer_types=kinds,
        full_attention_interval=2 if "linear_attention" in kinds else 0,
        num_attention_heads=heads, num_key_value_heads=heads, intermediate_size=largest("intermediate_size", width),
        use_mla=True, hidden_act="gelu_pytorch_tanh", norm_type="layer", sandwich_norm=True, attention_sink=True,
        rms_norm_eps=float(d["norm"]["eps"]), embed_scale=float(d["embedding"]["scale"]),
        token_side_dim=int((d.get("token_side") or {}).get("dim", 0)), tie_word_embeddings=False)
    for name in ("kv_lora_rank", "qk_nope_head_dim", "qk_rope_head_dim", "v_head_dim", "head_dim",
                 "linear_num_key_heads", "linear_num_value_heads", "linear_key_head_dim", "linear_value_head_dim"):
        fields[name] = largest(name, 0)
    return fields


#: architecture name -> reader of its configuration format
PLAN_FORMATS: dict[str, Callable[[dict], dict]] = {"Vofelix": vofelix_fields}


def run_order(num_layers: int, loop: Optional[tuple]) -> tuple[list[int], set[int]]:
    """Layer index of every layer run, and the runs in front of which the embedding output joins the stream
    again (the first run of every pass through the loop but the first pass)."""
    if not loop:
        return list(range(num_layers)), set()
    start, stop, times = loop
    body = list(range(start, stop))
    order = list(range(start)) + body * times + list(range(stop, num_layers))
    return order, {start + k * len(body) for k in range(1, times)}
