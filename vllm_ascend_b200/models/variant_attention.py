"""Paged grouped-query attention layer whose options come from its layer's configuration: biases of the
projections, short convolutions on q, k and v, q / k norm over all heads at once or head by head, rotary positions
on part of a head or none, queries scaled by position, values that are the keys, value heads of another size,
sliding window with kept first tokens, capped scores, learned bias by distance, attention sink, output gate per head,
scores mixed over the heads, the difference of two softmax maps per head.

projection [q | k | v | gate] -> one pass of convolution, norms, rotary and cache write -> paged attention with the
options -> output projection.  Heads are sharded over TP; key / value heads are replicated when there are fewer
than ranks, and the sums of squares of norms over all heads travel in one all-reduce.

Two options use *wide keys*, several projected keys side by side in one cache row.  Scores mixed over the heads,
s_h = sum_g T[h, g] q_g . k_{kv(g)}, are the products of wide queries (part c of head h: sum of T[h, g] q_g over the
heads g that share key head c) with the row of all key heads.  Two maps per head are two queries with one key part
each, the other part zero, over the same values.
"""
from __future__ import annotations

import torch

from ..attention.variant import (AttnOptions, PrepSpec, distance_table, qkv_prep, reserve_decode_scratch,
                                 variant_attention)
from ..config import ModelConfig
from ..ops.linear_recurrence import map_difference
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
        self.talk, self.maps = bool(cfg.attn_talk), 1 if cfg.attn_map_diff is None else 2
        if (self.talk or self.maps == 2) and (self.from_keys or self.taps or cfg.qk_norm_full or cfg.attn_head_gate
                                              or (self.talk and self.maps == 2)):
            raise NotImplementedError("wide keys come without convolutions, values from keys, norms over all heads, gates")
        p, hid = f"model.layers.{layer_idx}.self_attn", cfg.hidden_size
        # rows of the fused projection: name -> (rows of the whole model, heads sharded as q or as kv)
        rows = {"q": self.total_q * self.maps * self.D, "k": self.total_kv * self.maps * self.D}
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
        if (self.head_norm or not cfg.qk_norm_full) and self.taps:
            raise NotImplementedError("short convolutions come with a q / k norm over all heads")
        self.q_norm = self.k_norm = None
        if self.head_norm or cfg.qk_norm_full:
            self.q_norm, self.k_norm = (pf.ones((self.D if self.head_norm else h * self.D,)) for h in (self.Hq, self.Hkv))
        self.mix = self.lam = None
        if self.talk:
            mix = torch.eye(self.total_q, dtype=torch.float32, device=pf.device)
            mix = mix + pf.normal(f"{p}.talk", (self.total_q, self.total_q), std=0.1, dtype=torch.float32)
            self.mix = mix[r * self.Hq:(r + 1) * self.Hq].contiguous()
        if self.maps == 2:                   # lq1, lk1, lq2, lk2
            self.lam = torch.stack([pf.normal(f"{p}.lam.{i}", (self.D,), std=0.1, dtype=torch.float32) for i in range(4)])
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
        if cfg.rope_half_split and (self.rot_dim % 2 or self.rot_dim > self.D):
            raise ValueError(f"layer {layer_idx}: cannot rotate {self.rot_dim} of {self.D} dimensions")
        scale_of = None
        if cfg.attn_query_temp is not None:
            coef, every = cfg.attn_query_temp
            steps = torch.arange(1, max_pos + 1) // int(every)
            scale_of = (1 + float(coef) * torch.log(steps.double() + 1)).float().to(pf.device)
        # heads of the projection: with mixed scores every rank projects all queries and keys
        heads, kv_heads = (self.total_q, self.total_kv) if self.talk else (self.Hq * self.maps, self.Hkv * self.maps)
        self.prep = PrepSpec(heads, kv_heads, self.D, self.Dv, cfg.rms_norm_eps, self.q_norm, self.k_norm,
                             (self.total_q * self.D, self.total_kv * self.D), self.from_keys, self.conv_weight,
                             self.rot_dim, cos_sin, self.head_norm, v_heads=self.Hkv,
                             key_parts=self.total_kv if self.talk else self.maps,
                             part_run=self.total_q // self.total_kv if self.talk else 1, mix=self.mix, q_scale=scale_of)
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
        if self.talk and name in ("q", "k"):
            return 1
        return self.kv_world if name in ("k", "v") else self.comm.size

    def _shard_rank(self, name: str) -> int:
        if self._shards(name) == 1:
            return 0
        return self.kv_rank if name in ("k", "v") else self.comm.rank

    def _init(self, pf: ParamFactory, name: str, shape, part: str, std=None) -> torch.Tensor:
        rank = self._shard_rank(part)
        return pf.normal(name, shape, 0, rank, self._shards(part), std=std)

    def _rows(self, name: str, w: torch.Tensor) -> torch.Tensor:
        """This rank's share of a tensor whose rows belong to the heads of ``name``."""
        n, rank = w.shape[0] // self._shards(name), self._shard_rank(name)
        return w[rank * n:(rank + 1) * n]

    def _reduce_sums(self, sums: torch.Tensor) -> torch.Tensor:
        if self.kv_replicas > 1:             # replicated key heads count once
            sums = sums / torch.tensor([1.0, float(self.kv_replicas)], device=sums.device)
        return self.comm.group.all_reduce(sums)

    # ------------------------------------------------------------------ caches
    def kv_cache_heads(self) -> list[tuple[int, int]]:
        """(heads, width) of the paged tensors: keys, values."""
        return [(self.prep.key_heads, self.prep.key_parts * self.D), (self.Hkv, self.Dv)]

    def sequence_state_shapes(self, num_slots: int) -> list[tuple]:
        """Per-sequence state beside the pages: the last convolution inputs."""
        return [(num_slots, self.taps - 1, self.prep.columns)] if self.taps > 1 else []

    def reserve_decode_scratch(self, device, batch_sizes: list, max_keys: int) -> None:
        for kv_heads in {self.Hkv, self.prep.key_heads}:
            reserve_decode_scratch(device, batch_sizes[-1], self.Hq * self.maps, kv_heads, self.Dv, self.options, max_keys)

    # ------------------------------------------------------------------ forward
    def __call__(self, x: torch.Tensor, meta, kv_cache) -> torch.Tensor:
        o = self.attend(self.in_proj(x), meta, kv_cache[0], kv_cache[1], kv_cache[2] if len(kv_cache) > 2 else None)
        return self.o_proj(o)

    def attend(self, qkv: torch.Tensor, meta, k_cache, v_cache, state=None, out=None) -> torch.Tensor:
        """What lies between the two projections: rows [q | k | v | gate] -> [T, heads * value size] (into ``out``,
        whose rows may be strided)."""
        T = qkv.shape[0]
        q = qkv_prep(self.prep, qkv, meta, k_cache, v_cache, state,
                     self._reduce_sums if self.comm.size > 1 and not self.head_norm else None)
        gate = None
        if "g" in self._at:
            at, n = self._at["g"]
            gate = qkv[:, at:at + n]
        if self.maps == 2:
            o = variant_attention(q, k_cache, v_cache, meta, self.options, None)
            return map_difference(o, self.map_lambda, self.cfg.rms_norm_eps, 1.0 - self.cfg.attn_map_diff, qkv.dtype, out)
        if out is None:
            out = torch.empty((T, self.Hq * self.Dv), dtype=qkv.dtype, device=qkv.device)
        variant_attention(q, k_cache, v_cache, meta, self.options, gate, out.unflatten(1, (self.Hq, self.Dv)))
        return out

    # ------------------------------------------------------------------ weights
    def process_weights_after_loading(self) -> None:
        if self.rel is not None:
            reach = min(self.window or self.max_pos, self.max_pos)
            self.options.bias = distance_table(self.rel, int(self.cfg.attn_distance_max), reach)
        if self.maps == 2:
            lq1, lk1, lq2, lk2 = self.lam.double().cpu()
            self.map_lambda = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum())) + self.cfg.attn_map_diff
            self.options.out_f32 = True      # the maps are subtracted before anything is rounded

    def parts(self) -> list[str]:
        out = ["q", "k", "o"] + ([] if self.q_norm is None else ["q.norm", "k.norm"])
        if not self.from_keys:
            out.append("v")
        if self.taps:
            out += ["q.conv", "k.conv"] + ([] if self.from_keys else ["v.conv"])
        if self.in_proj.bias is not None:
            out += [f"{n}.b" for n in self._at if n != "g"]
        if self.o_proj.bias is not None:
            out.append("o.b")
        if self.maps == 2:
            out += list(self._LAMBDA)
        return out + [n for n, on in (("g", "g" in self._at), ("rel", self.rel is not None), ("talk", self.talk),
                                      ("sink", self.sink is not None)) if on]

    _LAMBDA = ("lq1", "lk1", "lq2", "lk2")

    def _pairs_side_by_side(self, w: torch.Tensor, part: str) -> torch.Tensor:
        """Rows of q or k heads whose rotary pairs are (i, i + rotated / 2), in the order (2i, 2i + 1)."""
        if w.shape[0] % self.D:
            raise ValueError(f"tensor {part}: unexpected shape {tuple(w.shape)}")
        order = torch.arange(self.D)
        order[:self.rot_dim] = order[:self.rot_dim].view(2, -1).T.flatten()
        return w.unflatten(0, (-1, self.D))[:, order.to(w.device)].flatten(0, 1)

    def load_part(self, part: str, w: torch.Tensor) -> None:
        """One un-fused tensor: projections q, k, v, g (output gate), o and their biases q.b, ...; q.norm, k.norm;
        convolutions q.conv, k.conv, v.conv; rel (bias by distance bucket, [buckets, heads]); sink; talk (what head h
        takes of the score of head g, [h, g]); lq1, lk1, lq2, lk2 (factor of the second map)."""
        tp, r = self.comm.size, self.comm.rank
        name, _, kind = part.partition(".")
        if part not in self.parts():
            raise KeyError(part)
        if part in self._LAMBDA:
            return copy_exact(self.lam[self._LAMBDA.index(part)], w, part)
        if part == "talk":
            if tuple(w.shape) != (self.total_q, self.total_q):
                raise ValueError(f"tensor talk: unexpected shape {tuple(w.shape)}")
            return copy_exact(self.mix, w[r * self.Hq:(r + 1) * self.Hq], part)
        if self.cfg.rope_half_split and self.rot_dim and name in ("q", "k"):
            w = self._pairs_side_by_side(w, part)
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
        at, n = self._at[name]
        whole = {"conv": self.conv_weight, "b": self.in_proj.bias, "": self.in_proj.weight}[kind]
        return copy_exact(whole[at:at + n], self._rows(name, w), part)

    def named_tensors(self):
        for attr in ("in_proj", "o_proj"):
            for n, t in getattr(self, attr).named_tensors():
                yield f"{attr}.{n}", t
        for n, t in (("q_norm.weight", self.q_norm), ("k_norm.weight", self.k_norm), ("conv.weight", self.conv_weight),
                     ("rel", self.rel), ("sink", self.sink), ("talk", self.mix), ("lam", self.lam)):
            if t is not None:
                yield n, t
