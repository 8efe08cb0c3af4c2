"""Two mixers side by side on one input: paged attention (``VariantAttention``) and a Mamba-2 state space
(``Mamba2Mixer``), left_scale * attention + right_scale * state space.

Both read the same rows, so their input projections are one matrix product, and both end in a projection to the
model's width, so their scaled read-outs lie side by side and meet one output projection that sums them.  The two
mixers' own weights are views of the fused ones.  The layer owns pages (keys, values) and a state per sequence
(convolution inputs, fp32 recurrent state).  The reference schedules such hybrid caches for attention and Mamba layers
that alternate (vllm_ascend/patch/platform/patch_mamba_config.py)."""
from __future__ import annotations

import torch

from .. import ops
from ..config import ModelConfig
from .layers import Linear, ParamFactory, TPComm
from .mamba2 import Mamba2Mixer
from .variant_attention import VariantAttention


class ParallelMixer:
    def __init__(self, pf: ParamFactory, cfg: ModelConfig, layer_idx: int, comm: TPComm, max_pos: int):
        self.comm = comm
        self.left = VariantAttention(pf, cfg, layer_idx, comm, max_pos)
        self.right = Mamba2Mixer(pf, cfg, layer_idx, comm)
        left_scale, self.right_scale = cfg.parallel_scales
        self.left.options.out_scale = float(left_scale)
        a, b = self.left.in_proj, self.right.in_proj
        self.split = a.weight.shape[0]
        parts = [a.weight, b.weight]
        rows = sum(w.shape[0] for w in parts)
        if rows % 8:
            parts.append(pf.zeros((8 - rows % 8, cfg.hidden_size)))
        weight, bias = torch.cat(parts), None
        rows = b.weight.shape[0]
        a.weight, b.weight = weight[:self.split], weight[self.split:self.split + rows]
        if a.bias is not None:
            bias = torch.cat([a.bias, pf.zeros((weight.shape[0] - self.split,))])
            a.bias = bias[:self.split]
        self.in_proj = Linear(weight, bias, name=f"model.layers.{layer_idx}.in_proj")
        self.inner = self.left.Hq * self.left.Dv
        self.out_weight = torch.cat([self.left.o_proj.weight, self.right.out_proj.weight], 1)
        self.left.o_proj.weight, self.right.out_proj.weight = self.out_weight[:, :self.inner], self.out_weight[:, self.inner:]

    # ------------------------------------------------------------------ caches
    def kv_cache_heads(self) -> list[tuple[int, int]]:
        return self.left.kv_cache_heads()

    def sequence_state_shapes(self, num_slots: int) -> list[tuple]:
        """Convolution inputs (activation type) and the recurrent state (fp32)."""
        conv, ssm = self.right.state_shapes(num_slots)
        return [conv, (ssm, torch.float32)]

    def reserve_decode_scratch(self, device, batch_sizes: list, max_keys: int) -> None:
        self.left.reserve_decode_scratch(device, batch_sizes, max_keys)

    # ------------------------------------------------------------------ forward
    def __call__(self, x: torch.Tensor, meta, cache) -> torch.Tensor:
        k_cache, v_cache, conv_state, ssm_state = cache
        T, n = x.shape[0], self.inner
        proj = self.in_proj(x)
        both = torch.empty((T, self.out_weight.shape[1]), dtype=x.dtype, device=x.device)
        self.left.attend(proj[:, :self.split], meta, k_cache, v_cache, out=both[:, :n])
        self.right.mix(proj[:, self.split:], meta, conv_state, ssm_state, self.right_scale, out=both[:, n:])
        y = ops.linear(both, self.out_weight)
        return self.comm.all_reduce(y) if self.comm.size > 1 else y

    # ------------------------------------------------------------------ weights
    def process_weights_after_loading(self) -> None:
        self.left.process_weights_after_loading()

    def parts(self) -> list[str]:
        return [f"left.{p}" for p in self.left.parts()] + [f"right.{p}" for p in self.right.parts()]

    def load_part(self, part: str, w: torch.Tensor) -> None:
        side, _, name = part.partition(".")
        return {"left": self.left, "right": self.right}[side].load_part(name, w)

    def named_tensors(self):
        for side in ("left", "right"):
            for n, t in getattr(self, side).named_tensors():
                yield f"{side}.{n}", t
