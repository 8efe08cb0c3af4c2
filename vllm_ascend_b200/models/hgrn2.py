"""HGRN2 mixer: linear attention whose forget gate also decides what is written.

Per head, with a gate f per key channel that never falls below a learned bound l:

    f_t = l + (1 - l) sigmoid(W_f h + b)      S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T      o_t = S_t^T silu(W_q h)

then an RMSNorm per head and the output projection.  One projection gives q, f and v; gate, recurrence and (in
decoding) the norm are one kernel (``ops.linear_recurrence.forget_recurrence``).  Instead of a KV cache the layer keeps
the [key x value] state per head in fp32.  Heads are sharded over TP.  The closest layer of the reference is its
lightning attention (vllm_ascend/ops/triton/mamba/lightning_attn.py)."""
from __future__ import annotations

import torch

from ..config import ModelConfig
from ..ops.linear_recurrence import forget_recurrence
from .layers import ColumnParallelLinear, ParamFactory, RowParallelLinear, TPComm, copy_exact


class HGRN2Mixer:
    is_linear_attention = True
    kind = "hgrn2"

    def __init__(self, pf: ParamFactory, cfg: ModelConfig, layer_idx: int, comm: TPComm):
        tp, r = comm.size, comm.rank
        self.cfg, self.comm = cfg, comm
        heads, self.D, self.P = cfg.linear_num_value_heads, cfg.linear_key_head_dim, cfg.linear_value_head_dim
        self.H = heads // tp
        p, qd, vd = f"model.layers.{layer_idx}.hgrn2", heads * self.D, heads * self.P
        self.in_proj = ColumnParallelLinear(pf, f"{p}.in_proj", cfg.hidden_size, [qd, qd, vd], comm)      # q | f | v
        self.out_proj = RowParallelLinear(pf, f"{p}.out_proj", vd, cfg.hidden_size, comm)
        self.f_bias = pf.normal(f"{p}.f_bias", (qd,), 0, r, tp, std=0.5)
        self.lower = pf.normal(f"{p}.lower", (qd,), 0, r, tp, std=0.2).abs().clamp(max=0.9)
        self.norm_weight = pf.ones((self.P,))

    def state_shapes(self, num_slots: int):
        """(unused convolution slot, recurrent state) shapes: the runner allocates a pair per layer."""
        return (num_slots, 1, 1), (num_slots, self.H, self.D, self.P)

    def __call__(self, x: torch.Tensor, meta, cache) -> torch.Tensor:
        state, n = cache[1], self.H * self.D
        qfv = self.in_proj(x)
        o = forget_recurrence(qfv[:, :n], qfv[:, n:2 * n], qfv[:, 2 * n:], self.f_bias, self.lower, state,
                              meta.query_start_loc, meta.state_slots, meta.has_initial_state, self.norm_weight,
                              self.cfg.rms_norm_eps, uniform=meta.max_query_len <= 1)
        return self.out_proj(o)

    @staticmethod
    def parts() -> list[str]:
        return ["q", "f", "f.b", "lower", "v", "norm", "o"]

    def load_part(self, part: str, w: torch.Tensor) -> None:
        """One un-fused tensor: the projections q, f, v, o, the gate's bias f.b and bound lower, norm."""
        tp, r = self.comm.size, self.comm.rank
        if part not in self.parts():
            raise KeyError(part)
        if part == "norm":
            return copy_exact(self.norm_weight, w, part)
        if part == "o":
            n = w.shape[1] // tp
            return copy_exact(self.out_proj.weight, w[:, r * n:(r + 1) * n], part)
        n = w.shape[0] // tp
        rows, at, size = w[r * n:(r + 1) * n], self.H * self.D, self.H * self.D
        dst = {"q": lambda: self.in_proj.weight[:at], "f": lambda: self.in_proj.weight[at:at + size],
               "v": lambda: self.in_proj.weight[at + size:], "f.b": lambda: self.f_bias, "lower": lambda: self.lower}
        return copy_exact(dst[part](), rows, part)

    def named_tensors(self):
        for attr in ("in_proj", "out_proj"):
            for n, t in getattr(self, attr).named_tensors():
                yield f"{attr}.{n}", t
        yield "f_bias", self.f_bias
        yield "lower", self.lower
        yield "norm.weight", self.norm_weight
