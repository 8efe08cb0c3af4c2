"""Decoders described layer by layer.

Most configurations give one set of sizes for all layers.  A *plan* gives every layer its own: which mixer
it has, the mixer's sizes and constants, and whether a feed-forward follows.  It is kept on
``ModelConfig.layer_plan`` as a list of ``{"mixer": kind, "mlp": bool, "over": {...}}`` where ``over`` holds
``ModelConfig`` fields of that layer (``ModelConfig.layer_config(i)`` applies them), so that the mixers read
a plain ``ModelConfig`` whether or not the model has a plan.  ``"weights_of": j`` marks a layer that runs with
layer j's parameters and a cache or state of its own.

This module turns the configuration formats of the Vofelix, Pegopel, Dubizen and Nevotar decoders into such plans."""
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


def _attention(m: dict) -> dict:
    """Options every paged grouped-query mixer of a plan has."""
    heads, kv = int(m["heads"]), int(m["kv_heads"])
    if kv < 1 or heads % kv:
        raise ValueError(f"{heads} query heads do not share {kv} key / value heads")
    mask = m.get("mask") or {}
    return dict(num_attention_heads=heads, num_key_value_heads=kv, head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]),
                attention_multiplier=float(m["scale"]), sliding_window=int(mask["size"]) if mask.get("size") else None,
                attn_keep_first=int(mask.get("keep_first") or 0), qk_norm_full=True, rotary_dims=0)


def _biased(m: dict) -> dict:
    return dict(_attention(m), attn_conv_kernel=int(m.get("conv") or 0), attn_distance_max=int(m["bias_max"]),
                attention_sink=True)


def _shared_kv(m: dict) -> dict:
    rot = m["rot"]
    if int(m["vdim"]) != int(m["dim"]):
        raise ValueError("values that are the keys have the keys' size: vdim must equal dim")
    if int(rot["dims"]) % 2 or int(rot["dims"]) > int(m["dim"]):
        raise ValueError(f"cannot rotate {rot['dims']} of {m['dim']} dimensions")
    return dict(_attention(m), attn_values_from_keys=True, rotary_dims=int(rot["dims"]),
                rope_theta=float(rot["base"]), rope_scaling=_yarn(rot.get("scaling")), attn_sink_value=0.0,
                attn_softcap=float(m["softcap"]) if m.get("softcap") else None, attn_head_gate=True)


_PEGOPEL_MIXERS: dict[str, tuple[str, Callable[[dict], dict]]] = {
    "attention": ("attention", _biased), "attention_2": ("attention", _shared_kv)}


def _normed(m: dict) -> dict:
    return dict(_attention(m), qk_norm_full=False, qk_norm=True, attention_bias=True, attention_out_bias=True,
                attn_distance_max=int(m["bias_max"]))


def _latent_query(m: dict) -> dict:
    return dict(_latent(m), attention_sink=False, q_lora_rank=int(m["q_rank"]), rope_half_split=True,
                latent_kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))


_DUBIZEN_MIXERS: dict[str, tuple[str, Callable[[dict], dict]]] = {
    "attention": ("attention", _normed), "latent_attention": ("latent", _latent_query)}


def _rotated(rot: dict, dim: int) -> dict:
    if int(rot["dims"]) % 2 or not 0 <= int(rot["dims"]) <= dim:
        raise ValueError(f"cannot rotate {rot['dims']} of {dim} dimensions")
    return dict(rotary_dims=int(rot["dims"]), rope_theta=float(rot["base"]), rope_half_split=True)


def _map_difference(m: dict) -> dict:
    temp = m.get("q_temp")
    if temp and int(temp["every"]) != temp["every"]:
        raise ValueError("the query temperature changes every whole number of positions")
    return dict(_attention(m), qk_norm_full=False, attention_bias=True, attn_map_diff=float(m["diff"]),
                attn_query_temp=(float(temp["coef"]), int(temp["every"])) if temp else None)


def _attention_and_state(m: dict) -> dict:
    left, right = m["left"], m["right"]
    heads, groups, parts = int(right["heads"]), int(right["groups"]), int(right["norm_groups"])
    if groups < 1 or heads % groups or parts < 1 or heads * int(right["vdim"]) % parts:
        raise ValueError(f"{heads} state-space heads do not divide into {groups} groups and {parts} norms")
    return dict(_attention(left), **_rotated(left["rot"], int(left["dim"])), qk_norm_full=False, qk_norm=True,
                attention_bias=True, attn_talk=True, parallel_scales=(float(m["left_scale"]), float(m["right_scale"])),
                mamba_config={"n_heads": heads, "d_head": int(right["vdim"]), "n_groups": groups, "d_state": int(right["state"]),
                              "d_conv": int(right["conv"]), "norm_groups": parts})


def _forget(m: dict) -> dict:
    return dict(linear_num_key_heads=int(m["heads"]), linear_num_value_heads=int(m["heads"]),
                linear_key_head_dim=int(m["dim"]), linear_value_head_dim=int(m["vdim"]))


_NEVOTAR_MIXERS: dict[str, tuple[str, Callable[[dict], dict]]] = {
    "attention": ("attention", _map_difference), "parallel": ("parallel", _attention_and_state),
    "hgrn2": ("hgrn2", _forget)}


# ---------------------------------------------------------------- feed-forwards
def _gated_mlp(m: dict) -> dict:
    return dict(intermediate_size=int(m["ff"]))


def _plain_mlp(m: dict) -> dict:
    return dict(intermediate_size=int(m["ff"]), mlp_gated=False, hidden_act="gelu", num_experts=0)


def _experts(m: dict) -> dict:
    router, shared = m["router"], m.get("shared")
    groups = router.get("groups") or {"count": 1, "keep": 1}
    experts, count, keep, top = int(router["experts"]), int(groups["count"]), int(groups["keep"]), int(router["top"])
    if count < 1 or experts % count or not 1 <= keep <= count or not 1 <= top <= experts // count * keep:
        raise ValueError(f"cannot choose {top} of {experts} experts from {keep} of {count} groups")
    return dict(num_experts=experts, num_experts_per_tok=top, moe_intermediate_size=int(m["expert"]["ff"]),
                n_group=count, topk_group=keep, moe_group_score="max", scoring_func="softmax", norm_topk_prob=True,
                routed_scaling_factor=float(router.get("scale", 1.0)), e_score_correction_bias=True, router_fp32=True,
                shared_expert_intermediate_size=int(shared["ff"]) if shared else 0, shared_expert_gate=bool(shared))


def _clamped_experts(m: dict) -> dict:
    router, shared = m["router"], m.get("shared")
    experts, top = int(router["experts"]), int(router["top"])
    if not 1 <= top <= experts:
        raise ValueError(f"cannot choose {top} of {experts} experts")
    return dict(num_experts=experts, num_experts_per_tok=top, moe_intermediate_size=int(m["expert"]["ff"]),
                expert_limit=float(m["expert"]["limit"]), scoring_func="sigmoid", norm_topk_prob=False, router_fp32=True,
                moe_weight_input=True, shared_expert_intermediate_size=int(shared["ff"]) if shared else 0,
                shared_expert_limit=float(shared["limit"]) if shared else None)


_DENSE = {"dense": _gated_mlp}


def _read_layers(d: dict, mixers: dict, mlps: dict = _DENSE) -> list[dict]:
    plan = []
    for i, layer in enumerate(d["layers"]):
        if layer["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        mixer, read = mixers[layer["type"]]
        over = read(layer["mixer"])
        mlp = layer.get("mlp")
        if mlp is not None:
            kind = mlp.get("kind", "dense")
            if kind not in mlps:
                raise ValueError(f"layer {i}: unknown feed-forward {kind!r}")
            over.update(mlps[kind](mlp))
        plan.append({"mixer": mixer, "mlp": mlp is not None, "over": over})
    return plan


def _share_weights(d: dict, plan: list) -> None:
    """Mark the layers that run with another layer's parameters; a chain ends at the layer that has them."""
    source = {i: int(layer["weights_of"]) for i, layer in enumerate(d["layers"]) if layer.get("weights_of") is not None}
    for i in source:
        j, seen = i, {i}
        while j in source:
            j = source[j]
            if not 0 <= j < len(plan) or j in seen:
                raise ValueError(f"layer {i}: no layer has the weights it names")
            seen.add(j)
        if plan[i] != plan[j]:
            raise ValueError(f"layer {i} is not of the form of layer {j}, whose weights it uses")
    for i in source:
        j = i
        while j in source:
            j = source[j]
        plan[i]["weights_of"] = j


def _read_loop(d: dict, num_layers: int) -> Optional[tuple]:
    loop = d.get("loop")
    if not loop:
        return None
    loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
    if not (0 <= loop[0] < loop[1] <= num_layers) or loop[2] < 1:
        raise ValueError(f"loop {loop} does not fit {num_layers} layers")
    return loop


def _largest(plan: list, name: str, default: int) -> int:
    return max([default] + [p["over"].get(name) or 0 for p in plan])


def vofelix_fields(d: dict) -> dict[str, Any]:
    """``ModelConfig`` fields of a Vofelix configuration."""
    plan = _read_layers(d, _VOFELIX_MIXERS)
    kinds = ["linear_attention" if p["mixer"] == "delta" else "full_attention" for p in plan]
    width = int(d["width"])
    heads = _largest(plan, "num_attention_heads", 0) or _largest(plan, "linear_num_value_heads", 1)
    fields: dict[str, Any] = dict(
        vocab_size=int(d["vocab"]), hidden_size=width, num_hidden_layers=len(plan), layer_plan=plan,
        layer_loop=_read_loop(d, len(plan)), layer_loop_refeed=True, layer_types=kinds,
        full_attention_interval=2 if "linear_attention" in kinds else 0,
        num_attention_heads=heads, num_key_value_heads=heads,
        intermediate_size=_largest(plan, "intermediate_size", width),
        use_mla=True, hidden_act="gelu_pytorch_tanh", norm_type="layer", sandwich_norm=True, attention_sink=True,
        rms_norm_eps=float(d["norm"]["eps"]), embed_scale=float(d["embedding"]["scale"]),
        token_side_dim=int((d.get("token_side") or {}).get("dim", 0)), tie_word_embeddings=False)
    for name in ("kv_lora_rank", "qk_nope_head_dim", "qk_rope_head_dim", "v_head_dim", "head_dim",
                 "linear_num_key_heads", "linear_num_value_heads", "linear_key_head_dim", "linear_value_head_dim"):
        fields[name] = _largest(plan, name, 0)
    return fields


def pegopel_fields(d: dict) -> dict[str, Any]:
    """``ModelConfig`` fields of a Pegopel configuration."""
    plan = _read_layers(d, _PEGOPEL_MIXERS)
    width = int(d["width"])
    return dict(
        vocab_size=int(d["vocab"]), hidden_size=width, num_hidden_layers=len(plan), layer_plan=plan,
        layer_loop=_read_loop(d, len(plan)), layer_types=["full_attention"] * len(plan),
        num_attention_heads=_largest(plan, "num_attention_heads", 1),
        num_key_value_heads=_largest(plan, "num_key_value_heads", 1), head_dim=_largest(plan, "head_dim", 1),
        v_head_dim=_largest(plan, "v_head_dim", 1), intermediate_size=_largest(plan, "intermediate_size", width),
        hidden_act="gelu_pytorch_tanh", norm_type="rms", rms_norm_eps=float(d["norm"]["eps"]),
        residual_streams=int(d.get("streams") or 1), learned_positions=int(d["max_positions"]),
        max_position_embeddings=int(d["max_positions"]), tie_word_embeddings=True)


def dubizen_fields(d: dict) -> dict[str, Any]:
    """``ModelConfig`` fields of a Dubizen configuration."""
    plan = _read_layers(d, _DUBIZEN_MIXERS, {"dense": _plain_mlp, "moe": _experts})
    for i, p in enumerate(plan):
        src = p["over"].get("latent_kv_from")
        if src is None:
            continue
        other = plan[src]["over"] if 0 <= src < i else {}
        same = ("kv_lora_rank", "qk_rope_head_dim", "rope_theta", "rope_scaling")
        if other.get("latent_kv_from", -1) is not None or any(other[n] != p["over"][n] for n in same):
            raise ValueError(f"layer {i}: layer {src} has no latents of this layer's form")
    width = int(d["width"])
    fields: dict[str, Any] = dict(
        vocab_size=int(d["vocab"]), hidden_size=width, num_hidden_layers=len(plan), layer_plan=plan,
        layer_types=["full_attention"] * len(plan), use_mla=any(p["mixer"] == "latent" for p in plan),
        num_attention_heads=_largest(plan, "num_attention_heads", 1),
        num_key_value_heads=_largest(plan, "num_key_value_heads", 1),
        intermediate_size=_largest(plan, "intermediate_size", width), norm_type="layer", norm_bias=False, pre_norm=False,
        sandwich_norm=True, residual_multiplier=float(d["residual_mult"]), rms_norm_eps=float(d["norm"]["eps"]),
        tie_word_embeddings=True)
    for name in ("head_dim", "v_head_dim", "kv_lora_rank", "qk_nope_head_dim", "qk_rope_head_dim", "num_experts",
                 "num_experts_per_tok", "moe_intermediate_size"):
        fields[name] = _largest(plan, name, 0)
    return fields


def nevotar_fields(d: dict) -> dict[str, Any]:
    """``ModelConfig`` fields of a Nevotar configuration."""
    plan = _read_layers(d, _NEVOTAR_MIXERS, {"moe": _clamped_experts})
    _share_weights(d, plan)
    kinds = ["linear_attention" if p["mixer"] == "hgrn2" else "full_attention" for p in plan]
    width, groups = int(d["width"]), int(d["norm"].get("groups", 1))
    if groups < 1 or width % groups:
        raise ValueError(f"a width of {width} does not divide into {groups} norm groups")
    heads = _largest(plan, "num_attention_heads", 0) or _largest(plan, "linear_num_value_heads", 1)
    fields: dict[str, Any] = dict(
        vocab_size=int(d["vocab"]), hidden_size=width, num_hidden_layers=len(plan), layer_plan=plan, layer_types=kinds,
        full_attention_interval=2 if "linear_attention" in kinds else 0, num_attention_heads=heads,
        num_key_value_heads=_largest(plan, "num_key_value_heads", 0) or heads, intermediate_size=width, norm_type="rms",
        norm_groups=groups, rms_norm_eps=float(d["norm"]["eps"]), tie_word_embeddings=True)
    for name in ("head_dim", "v_head_dim", "linear_num_key_heads", "linear_num_value_heads", "linear_key_head_dim",
                 "linear_value_head_dim", "num_experts", "num_experts_per_tok", "moe_intermediate_size"):
        fields[name] = _largest(plan, name, 0)
    return fields


#: architecture name -> reader of its configuration format
PLAN_FORMATS: dict[str, Callable[[dict], dict]] = {"Vofelix": vofelix_fields, "Pegopel": pegopel_fields,
                                                   "Dubizen": dubizen_fields, "Nevotar": nevotar_fields}


def run_order(num_layers: int, loop: Optional[tuple]) -> tuple[list[int], set[int]]:
    """Layer index of every layer run, and the first run of every pass through the loop but the first pass
    (where ``layer_loop_refeed`` adds the embedding output to the stream again)."""
    if not loop:
        return list(range(num_layers)), set()
    start, stop, times = loop
    body = list(range(start, stop))
    order = list(range(start)) + body * times + list(range(stop, num_layers))
    return order, {start + k * len(body) for k in range(1, times)}
