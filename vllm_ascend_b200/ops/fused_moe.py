"""MoE routing and expert computation.

``gating_topk`` implements the router of the reference's fused gating op
(softmax / sigmoid scores, correction bias, group-limited top-k, renormalise,
scaling; csrc/moe/moe_gating_top_k, golden model in
tests/e2e/nightly/single_node/ops/singlecard_ops/test_npu_moe_gating_top_k.py:34-90).
``fused_experts`` is dispatch -> grouped GEMM1 -> SwiGLU -> grouped GEMM2 ->
weighted combine for the experts resident on this rank
(vllm_ascend/ops/fused_moe/moe_mlp.py:573-687).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import _native
from . import reference as ref


def gating_topk_ref(logits: torch.Tensor, k: int, scoring: str = "softmax", renorm: bool = True,
                    n_group: int = 1, topk_group: int = 1,
                    bias: Optional[torch.Tensor] = None, scale: float = 1.0, group_score: Optional[str] = None):
    """``group_score``: a group counts by its best expert ("max") or by the sum of its best two ("top2"); by
    default "top2" where a bias is given."""
    x = logits.float()
    scores = torch.softmax(x, dim=-1) if scoring == "softmax" else torch.sigmoid(x)
    choice = scores + bias.float() if bias is not None else scores
    T, E = scores.shape
    if n_group > 1:
        g = choice.view(T, n_group, E // n_group)
        if _top2(group_score, bias) and g.shape[-1] > 1:
            gscore = g.topk(2, dim=-1).values.sum(-1)       # noaux_tc: sum of the top-2 per group
        else:
            gscore = g.max(dim=-1).values
        gidx = gscore.topk(topk_group, dim=-1).indices
        gmask = torch.zeros(T, n_group, dtype=torch.bool, device=x.device)
        gmask.scatter_(1, gidx, True)
        choice = choice.masked_fill(~gmask.unsqueeze(-1).expand(T, n_group, E // n_group)
                                    .reshape(T, E), float("-inf"))
    ids = choice.topk(k, dim=-1).indices
    w = scores.gather(1, ids)
    if renorm:
        w = w / w.sum(dim=-1, keepdim=True).clamp_min(1e-20)
    return (w * scale).float(), ids.to(torch.int32)


def _top2(group_score: Optional[str], bias: Optional[torch.Tensor]) -> bool:
    if group_score not in (None, "max", "top2"):
        raise ValueError(f"unknown group score {group_score!r}")
    return bias is not None if group_score is None else group_score == "top2"


def gating_topk(logits: torch.Tensor, k: int, scoring: str = "softmax", renorm: bool = True,
                n_group: int = 1, topk_group: int = 1, bias: Optional[torch.Tensor] = None,
                scale: float = 1.0, group_score: Optional[str] = None):
    if logits.is_cuda and _native.available() and hasattr(_native.lib(), "b200_moe_gating_topk") \
            and logits.shape[1] <= 512 and k <= 32 and n_group <= 32:
        from . import moe_native
        return moe_native.gating_topk(logits, k, scoring, renorm, n_group, topk_group, bias, scale, group_score)
    return gating_topk_ref(logits, k, scoring, renorm, n_group, topk_group, bias, scale, group_score)


def fused_experts_ref(x: torch.Tensor, w13: torch.Tensor, w2: torch.Tensor,
                      topk_w: torch.Tensor, topk_ids: torch.Tensor,
                      expert_map: Optional[torch.Tensor] = None, limit: Optional[float] = None,
                      weight_input: bool = False) -> torch.Tensor:
    """x [T,H]; w13 [E_local, 2I, H]; w2 [E_local, H, I]; ids are global expert ids,
    ``expert_map`` maps global -> local (-1: not on this rank).  ``limit``: clamped gate instead of SiLU;
    ``weight_input``: an expert works on weight * input, its output is not weighted."""
    T, H = x.shape
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    ids = topk_ids.long()
    if expert_map is not None:
        ids = expert_map.long()[ids]
    E = w13.shape[0]
    for e in range(E):
        tok, slot = (ids == e).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        h = x[tok] @ w13[e].to(x.dtype).t()
        w = topk_w[tok, slot].unsqueeze(-1).float()
        if weight_input:
            h, w = h.float() * w, 1.0
        a = ref.silu_and_mul(h) if limit is None else ref.activation(h, "swiglu_oai", gated=True, limit=limit)
        y = a.to(x.dtype) @ w2[e].to(x.dtype).t()
        out.index_add_(0, tok, y.float() * w)
    return out.to(x.dtype)


def fused_experts(x, w13, w2, topk_w, topk_ids, expert_map=None, quant=None, shared=None, shared_gate=None,
                  limit=None, weight_input=False):
    """Weighted sum of the chosen experts' outputs (``weight_input``: sum of the outputs for weighted inputs);
    ``shared`` [T, H] (a shared expert's output) is added, scaled by sigmoid(x . shared_gate) where that vector is
    given.  ``limit``: the experts' gate is the clamped one, min(g, limit) sigmoid(1.702 .) (clamp(u) + 1)."""
    if x.is_cuda and x.dtype in (torch.bfloat16, torch.float32) and w13.dtype == x.dtype and _native.available() \
            and hasattr(_native.lib(), "b200_moe_permute") and quant is None:
        from . import moe_native
        return moe_native.fused_experts(x, w13, w2, topk_w, topk_ids, expert_map, shared, shared_gate, limit, weight_input)
    if quant is not None:
        if limit is not None or weight_input:
            raise NotImplementedError("quantised experts have SiLU gates and weighted outputs")
        y = quant.apply_experts(x, w13, w2, topk_w, topk_ids, expert_map)
    else:
        y = fused_experts_ref(x, w13, w2, topk_w, topk_ids, expert_map, limit, weight_input)
    if shared is None:
        return y
    g = 1.0 if shared_gate is None else torch.sigmoid(x.float() @ shared_gate.float().view(-1, 1))
    return (y.float() + g * shared.float()).to(y.dtype)


def hash_topk(token_ids: torch.Tensor, table: torch.Tensor):
    """Hash routing: the experts of a token are a fixed function of its token id
    (``table`` [vocab, k] of expert ids), all with equal weight — the router of the first
    layers of some models (vllm_ascend/ops/fused_moe/router/fused_topk_router.py:103-141)."""
    ids = table[token_ids.long()].to(torch.int32)
    k = ids.shape[1]
    w = torch.full(ids.shape, 1.0 / k, dtype=torch.float32, device=ids.device)
    return w, ids
