"""Paged grouped-query attention layer whose options come from its layer's configuration: biases of the
projections, short convolutions on q, k and v, q / k norm over all heads at once or head by head, rotary positions
on part of a head or none, values that are the keys, value heads of another size, sliding window with kept first
tokens, capped scores, learned bias by distance, attention sink, output gate per head.

projection [q | k | v | gate] -> one pass of convolution, norms, rotary and cache write -> paged attention with the
options -> output projection.  Heads are sharded over TP; key / value heads are replicated when there are fewer
than ranks, and the sums of squares of norms over all heads travel in one all-reduce.
"""
from __future__ import annotations

import torch

from ..attention.variant import (AttnOptions, PrepSpec, distance_table, qkv_prep, reserve_decode_scratch,
                                 variant_attention)
from ..config import ModelConfig
from ..parallel import state as pstate
from .layers import Linear, ParamFactory, RowParallelLinear, TPComm, copy_exact, get_cos_sin_cache


class VariantAttention:
    def __init__(self, pf: ParamFactory, cfg: ModelConfig, layer_idx: int, comm: TPComm, max_pos: int):
        tp, r = comm.size, comm.rank
        self.cfg, self.comm, self.max_pos = cfg, comm, max_pos
        self.total_q, self.total_kv = cfg.num_attention_heads, cfg.num_key_value_heads
        if self.total_kv % tp and tp % self.total_kv:
            raise ValueError(f"layer {layer_idx}: {self.total_kv} key / value heads over {tp} tensor-parallel ranks")
        if pstate.get_dcp_group().world_size > 1:
            raise NotImplementedError("decode context parallelism does not serve attention with options")
        self.Hq, self.Hkv = self.total_q // tp, max(1, self.total_kv // tp)
        self.kv_replicas = max(1, tp // self.total_kv)
        self.kv_world, self.kv_rank = tp // self.kv_replicas, r // self.kv_replicas
        self.D, self.Dv = cfg.head_dim, cfg.v_head_dim or cfg.head_dim
        self.from_keys = bool(cfg.attn_values_from_keys)
        self.taps = int(cfg.attn_conv_kernel)
        p, hid = f"model.layers.{layer_idx}.self_attn", cfg.hidden_size
        # rows of the fused projection: name -> (rows of the whole model, heads sharded as q or as kv)
        rows = {"q": self.total_q * self.D, "k": self.total_kv * self.D}
        if not self.from_keys:
            rows["v"] = self.total_kv * self.Dv
        if cfg.attn_head_gate:
            rows["g"] = self.total_q
        self._at, at = {}, 0
        for name, n in rows.items():
            n //= self._shards(name)
            self._at[name] = (at, n)
            at += n
        parts = [self._init(pf, f"{p}.in_proj.{n}", (rows[n], hid), n) for n in rows]
        if at % 8:                           # rows of 16 bytes for the kernels
            parts.append(pf.zeros((8 - at % 8, hid)))
        weight = torch.cat(parts)
        self.in_proj = Linear(weight, pf.zeros((weight.shape[0],)) if cfg.attention_bias else None, name=f"{p}.in_proj")
        self.o_proj = RowParallelLinear(pf, f"{p}.o_proj", self.total_q * self.Dv, hid, comm, bias=cfg.attention_out_bias)
        self.head_norm = bool(cfg.qk_norm and not cfg.qk_norm_full)
        if self.head_norm and self.taps:
            raise NotImplementedError("short convolutions come with a q / k norm over all heads")
        self.q_norm, self.k_norm = (pf.ones((self.D if self.head_norm else h * self.D,)) for h in (self.Hq, self.Hkv))
        self.conv_weight = None
        if self.taps:
            self.conv_weight = torch.cat([self._init(pf, f"{p}.conv.{n}", (rows[n], self.taps), n, std=0.5)
                                          for n in rows if n != "g"])
        self.rel = self.sink = None
        if cfg.attn_distance_max:
            self.rel = pf.normal(f"{p}.rel", (cfg.attn_distance_buckets, self.total_q), 1, r, tp, std=0.5,
                                 dtype=torch.float32)
        if cfg.attention_sink:
            self.sink = pf.normal(f"{p}.sink", (self.total_q,), 0, r, tp, std=1.0, dtype=torch.float32)
        self.rot_dim = self.D if cfg.rotary_dims is None else int(cfg.rotary_dims)
        cos_sin = get_cos_sin_cache(self.rot_dim, max_pos, cfg.rope_theta, cfg.rope_scaling,
                                    pf.device) if self.rot_dim else None
        self.prep = PrepSpec(self.Hq, self.Hkv, self.D, self.Dv, cfg.rms_norm_eps, self.q_norm, self.k_norm,
                             (self.total_q * self.D, self.total_kv * self.D), self.from_keys, self.conv_weight,
                             self.rot_dim, cos_sin, self.head_norm)
        scale = self.D ** -0.5 if cfg.attention_multiplier is None else float(cfg.attention_multiplier)
        self.window = int(cfg.sliding_window or 0)
        fixed = None
        if cfg.attn_sink_value is not None:
            fixed = torch.full((self.Hq,), float(cfg.attn_sink_value), dtype=torch.float32, device=pf.device)
        self.options = AttnOptions(scale, self.window, int(cfg.attn_keep_first), float(cfg.attn_softcap or 0.0),
                                   sink=self.sink if self.sink is not None else fixed)
        self.process_weights_after_loading()

    # ------------------------------------------------------------------ sharding
    def _shards(self, name: str) -> int:
        return self.kv_world if name in ("k", "v") else self.comm.size

    def _init(self, pf: ParamFactory, name: str, shape, part: str, std=None) -> torch.Tensor:
        rank = self.kv_rank if part in ("k", "v") else self.comm.rank
        return pf.normal(name, shape, 0, rank, self._shards(part), std=std)

    def _rows(self, name: str, w: torch.Tensor) -> torch.Tensor:
        """This rank's share of a tensor whose rows belong to the heads of ``name``."""
        n = w.shape[0] // self._shards(name)
        rank = self.kv_rank if name in ("k", "v") else self.comm.rank
        return w[rank * n:(rank + 1) * n]

    def _reduce_sums(self, sums: torch.Tensor) -> torch.Tensor:
        if self.kv_replicas > 1:             # replicated key heads count once
            sums = sums / torch.tensor([1.0, float(self.kv_replicas)], device=sums.device)
        return self.comm.group.all_reduce(sums)

    # ------------------------------------------------------------------ caches
    def kv_cache_heads(self) -> list[tuple[int, int]]:
        """(heads, width) of the paged tensors: keys, values."""
        return [(self.Hkv, self.D), (self.Hkv, self.Dv)]

    def sequence_state_shapes(self, num_slots: int) -> list[tuple]:
        """Per-sequence state beside the pages: the last convolution inputs."""
        return [(num_slots, self.taps - 1, self.prep.columns)] if self.taps > 1 else []

    def reserve_decode_scratch(self, device, batch_sizes: list, max_keys: int) -> None:
        reserve_decode_scratch(device, batch_sizes[-1], self.Hq, self.Hkv, self.Dv, self.options, max_keys)

    # ------------------------------------------------------------------ forward
    def __call__(self, x: torch.Tensor, meta, kv_cache) -> torch.Tensor:
        k_cache, v_cache = kv_cache[0], kv_cache[1]
        state = kv_cache[2] if len(kv_cache) > 2 else None
        qkv = self.in_proj(x)
        q = qkv_prep(self.prep, qkv, meta, k_cache, v_cache, state,
                     self._reduce_sums if self.comm.size > 1 and not self.head_norm else None)
        gate = None
        if "g" in self._at:
            at, n = self._at["g"]
            gate = qkv[:, at:at + n]
        o = variant_attention(q, k_cache, v_cache, meta, self.options, gate)
        return self.o_proj(o.view(x.shape[0], self.Hq * self.Dv))

    # ------------------------------------------------------------------ weights
    def process_weights_after_loading(self) -> None:
        if self.rel is not None:
            reach = min(self.window or self.max_pos, self.max_pos)
            self.options.bias = distance_table(self.rel, int(self.cfg.attn_distance_max), reach)

    def parts(self) -> list[str]:
        out = ["q", "k", "q.norm", "k.norm", "o"]
        if not self.from_keys:
            out.append("v")
        if self.taps:
            out += ["q.conv", "k.conv"] + ([] if self.from_keys else ["v.conv"])
        if self.in_proj.bias is not None:
            out += [f"{n}.b" for n in self._at if n != "g"]
        if self.o_proj.bias is not None:
            out.append("o.b")
        return out + [n for n, on in (("g", "g" in self._at), ("rel", self.rel is not None),
                                      ("sink", self.sink is not None)) if on]

    def load_part(self, part: str, w: torch.Tensor) -> None:
        """One un-fused tensor: projections q, k, v, g (output gate), o and their biases q.b, ...; q.norm, k.norm;
        convolutions q.conv, k.conv, v.conv; rel (bias by distance bucket, [buckets, heads]); sink."""
        tp, r = self.comm.size, self.comm.rank
        name, _, kind = part.partition(".")
        if part == "o":
            n = w.shape[1] // tp
            return copy_exact(self.o_proj.weight, w[:, r * n:(r + 1) * n], part)
        if part == "o.b":
            return copy_exact(self.o_proj.bias, w, part)
        if part == "rel":
            if w.dim() != 2 or w.shape[1] != self.total_q or w.shape[0] < 2:
                raise ValueError(f"tensor rel: unexpected shape {tuple(w.shape)}")
            self.rel = w[:, r * self.Hq:(r + 1) * self.Hq].to(self.rel.device, torch.float32).contiguous()
            return None
        if part == "sink":
            return copy_exact(self.sink, self._rows("g", w), part)
        if kind == "norm":
            return copy_exact(self.q_norm if name == "q" else self.k_norm, w if self.head_norm else self._rows(name, w), part)
        if part not in self.parts():
            raise KeyError(part)
        at, n = self._at[name]
        whole = {"conv": self.conv_weight, "b": self.in_proj.bias, "": self.in_proj.weight}[kind]
        return copy_exact(whole[at:at + n], self._rows(name, w), part)

    def named_tensors(self):
        for attr in ("in_proj", "o_proj"):
            for n, t in getattr(self, attr).named_tensors():
                yield f"{attr}.{n}", t
        for n, t in (("q_norm.weight", self.q_norm), ("k_norm.weight", self.k_norm), ("conv.weight", self.conv_weight),
                     ("rel", self.rel), ("sink", self.sink)):
            if t is not None:
                yield n, t
