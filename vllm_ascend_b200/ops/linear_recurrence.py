"""Linear recurrences S_t = d_t S_{t-1} + k_t u_t^T, o_t = S_t^T q_t with an fp32 state per sequence and head, and the
norm of what they read out:

* ``state_space``        Mamba-2: one decay per head, d = exp(-exp(A_log) dt), u = dt x, and D x added to the read-out;
* ``forget_recurrence``  HGRN2: a forget gate f per channel that decides what is written as well, k = 1 - f, d = f;
* ``decayed_attention``  gated linear attention with a given log-decay per token and head;
* ``group_norm``         RMS norm of equal parts of a row, optionally of y * silu(z) or of the difference of two maps.

CUDA kernels (bf16 or fp32 activations; prefill keeps the state in registers and reads tokens in chunks, decode streams
it once) on GPU tensors, PyTorch definitions on the CPU.  The reference runs such layers through Triton kernels and
vLLM's Mamba-2 kernels (vllm_ascend/ops/triton/mamba/lightning_attn.py, vllm_ascend/ops/triton/fla/*)."""
from __future__ import annotations

import ctypes
from ctypes import c_void_p
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .. import _native
from . import linear_attn as la

_DTYPES = {torch.bfloat16: 0, torch.float32: 1}


class _RecurrenceArgs(ctypes.Structure):
    """RecurrenceArgs of csrc/linear_recurrence.cu."""
    _fields_ = _native.struct_fields(
        pointers="q k v f log_decay dt dt_bias A_log D f_bias lower state cu slots has_init norm_w out",
        longs="q_stride k_stride v_stride f_stride dt_stride out_stride num_slots",
        ints="mode num_seqs key_heads heads dk dv dtype uniform", floats="dt_lo dt_hi eps out_scale")


class _GroupNormArgs(ctypes.Structure):
    """GroupNormArgs of csrc/group_norm.cu."""
    _fields_ = _native.struct_fields(
        pointers="y y2 z w out", longs="rows y_stride y_group z_stride out_stride w_len",
        ints="groups size in_f32 dtype", floats="lam eps scale")


_native.register_signature("b200_linear_recurrence", [c_void_p, c_void_p, c_void_p])
_native.register_signature("b200_group_norm", [c_void_p, c_void_p])

LOG_DECAY, STATE_SPACE, FORGET = 0, 1, 2


def _launch(a: _RecurrenceArgs, device) -> int:
    rc = _native.lib().b200_linear_recurrence(ctypes.addressof(a), _native.status_word(device).data_ptr(),
                                              _native.stream_ptr())
    if rc != -1:
        _native.check(rc, "linear_recurrence")
        _native.count_launch()
    return rc


def _common(v, state, cu, slots, has_init, out, uniform, **kw) -> _RecurrenceArgs:
    if state.dtype != torch.float32 or not state.is_contiguous():
        raise TypeError("the recurrent state is a dense fp32 tensor")
    B = cu.numel() - 1
    return _RecurrenceArgs(
        v=v.data_ptr(), v_stride=v.stride(0), state=state.data_ptr(), cu=cu.data_ptr(), slots=slots.data_ptr(),
        has_init=has_init.data_ptr(), out=out.data_ptr(), out_stride=out.stride(0), num_slots=state.shape[0], num_seqs=B,
        heads=state.shape[1], dk=state.shape[2], dv=state.shape[3], dtype=_DTYPES[v.dtype],
        uniform=int(uniform and v.shape[0] == B), out_scale=1.0, **kw)


# ---------------------------------------------------------------- Mamba-2
@dataclass
class StateSpace:
    """Constants of a layer: fp32 per head, and the limits of the step size."""
    A_log: torch.Tensor
    dt_bias: torch.Tensor
    D: torch.Tensor
    groups: int
    dt_limit: tuple = (0.0, float("inf"))
    chunk: int = 64                    # of the chunk-parallel form on host tensors


def state_space(s: StateSpace, xbc: torch.Tensor, dt: torch.Tensor, state: torch.Tensor, cu, slots, has_init, cu_cpu=None,
                uniform: bool = False) -> torch.Tensor:
    """xbc [T, x | B | C] after convolution and SiLU, dt [T, H] raw (rows may be strided), state [slots, H, N, P]
    (updated) -> y [T, H * P], the D x term included."""
    T = xbc.shape[0]
    _, H, N, P = state.shape
    inner, gn = H * P, s.groups * N
    if not xbc.is_cuda:
        x, B, C = (t.reshape(T, -1, n) for t, n in ((xbc[:, :inner], P), (xbc[:, inner:inner + gn], N), (xbc[:, inner + gn:], N)))
        step = torch.clamp(F.softplus(dt.float() + s.dt_bias, threshold=30.0), *s.dt_limit)
        y = la.gated_linear_attention(C, B, x.float() * step.unsqueeze(-1), -torch.exp(s.A_log) * step, state, cu, slots,
                                      has_init, cu_cpu=cu.tolist() if cu_cpu is None else cu_cpu, chunk=s.chunk)
        return (y + s.D.view(1, H, 1) * x.float()).reshape(T, inner).to(xbc.dtype)
    if xbc.dtype not in _DTYPES or dt.dtype != xbc.dtype or xbc.stride(1) != 1 or dt.stride(1) != 1 \
            or any(t.dtype != torch.float32 for t in (s.A_log, s.dt_bias, s.D)):
        raise TypeError("state_space takes bf16 or fp32 rows of one type and fp32 constants")
    out = torch.empty((T, inner), dtype=xbc.dtype, device=xbc.device)
    if T == 0:
        return out
    x, B, C = xbc, xbc[:, inner:], xbc[:, inner + gn:]
    _launch(_common(x, state, cu, slots, has_init, out, uniform, mode=STATE_SPACE, q=C.data_ptr(), k=B.data_ptr(),
                    q_stride=xbc.stride(0), k_stride=xbc.stride(0), dt=dt.data_ptr(), dt_stride=dt.stride(0),
                    dt_bias=s.dt_bias.data_ptr(), A_log=s.A_log.data_ptr(), D=s.D.data_ptr(), key_heads=s.groups,
                    dt_lo=float(s.dt_limit[0]), dt_hi=float(s.dt_limit[1])), xbc.device)
    return out


# ---------------------------------------------------------------- HGRN2
def forget_recurrence_ref(q, f, v, f_bias, lower, state, cu, slots, has_init):
    T = q.shape[0]
    _, H, D, P = state.shape
    qs = F.silu(q.float()).view(T, H, D)
    low = lower.float()
    logit = f.float() + f_bias.float()
    gate = (low + (1 - low) * torch.sigmoid(logit)).view(T, H, D, 1)
    write = ((1 - low) * torch.sigmoid(-logit)).view(T, H, D, 1)         # 1 - gate
    vs = v.float().view(T, H, 1, P)
    out = torch.empty((T, H, P), dtype=torch.float32)
    cu_l = cu.tolist()
    for b in range(len(cu_l) - 1):
        if cu_l[b + 1] == cu_l[b]:
            continue
        i = int(slots[b])
        S = state[i].clone() if bool(has_init[b]) else torch.zeros_like(state[i])
        for t in range(cu_l[b], cu_l[b + 1]):
            S = gate[t] * S + write[t] * vs[t]
            out[t] = torch.einsum("hdv,hd->hv", S, qs[t])
        state[i] = S
    return out


def forget_recurrence(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor, f_bias: torch.Tensor, lower: torch.Tensor,
                      state: torch.Tensor, cu, slots, has_init, norm_w: torch.Tensor, eps: float,
                      uniform: bool = False) -> torch.Tensor:
    """Raw projections q, f [T, H * D] and v [T, H * P] (rows may be strided) -> the read-out, RMS-normed per head with
    ``norm_w`` [P], [T, H * P].  state [slots, H, D, P] is updated."""
    T = q.shape[0]
    _, H, D, P = state.shape
    if not q.is_cuda:
        o = forget_recurrence_ref(q, f, v, f_bias, lower, state, cu, slots, has_init)
        return group_norm(o.view(T, H * P), norm_w, H, eps, dtype=q.dtype)
    if q.dtype not in _DTYPES or any(t.dtype != q.dtype for t in (f, v, f_bias, lower, norm_w)) \
            or any(t.stride(1) != 1 for t in (q, f, v)):
        raise TypeError("forget_recurrence takes bf16 or fp32 rows and weights of one type")
    out = torch.empty((T, H * P), dtype=q.dtype, device=q.device)
    if T == 0:
        return out
    a = _common(v, state, cu, slots, has_init, out, uniform, mode=FORGET, q=q.data_ptr(), f=f.data_ptr(),
                q_stride=q.stride(0), f_stride=f.stride(0), f_bias=f_bias.data_ptr(), lower=lower.data_ptr(),
                norm_w=norm_w.data_ptr(), eps=eps, key_heads=H)
    if _launch(a, q.device) == -1:                # the norm is fused into the decode kernel only
        a.norm_w = None
        _launch(a, q.device)
        return group_norm(out, norm_w, H, eps)
    return out


# ---------------------------------------------------------------- gated linear attention
def decayed_attention(q, k, v, g, state, cu, slots, has_init, uniform: bool = False) -> torch.Tensor:
    """``linear_attn.gated_linear_attention_ref`` on the GPU: q, k [T, Hk, N], v [T, H, P] of one type, g [T, H]."""
    q, k, v = (t if t.stride(2) == 1 and t.stride(1) == t.shape[2] else t.contiguous() for t in (q, k, v))
    if v.dtype not in _DTYPES or q.dtype != v.dtype or k.dtype != v.dtype:
        q, k, v = q.float(), k.float(), v.float()
    g = g.float().contiguous()
    T, H, P = v.shape
    out = torch.empty((T, H, P), dtype=v.dtype, device=v.device)
    if T:
        _launch(_common(v, state, cu, slots, has_init, out, uniform, mode=LOG_DECAY, q=q.data_ptr(), k=k.data_ptr(),
                        q_stride=q.stride(0), k_stride=k.stride(0), log_decay=g.data_ptr(), key_heads=q.shape[1]), v.device)
    return out


# ---------------------------------------------------------------- norms of the read-out
def group_norm(y: torch.Tensor, w: Optional[torch.Tensor], groups: int, eps: float, z: Optional[torch.Tensor] = None,
               scale: float = 1.0, out: Optional[torch.Tensor] = None, dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """scale * w * rms_norm of ``groups`` equal parts of y [T, C], or of y * silu(z).  ``w``: [C], or [C / groups] shared
    by the parts."""
    T, C = y.shape
    size = C // groups
    dtype = dtype or y.dtype
    if not y.is_cuda:
        v = y.float()
        if z is not None:
            v = v * F.silu(z.float())
        v = v.reshape(T, groups, size)
        v = v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps)
        if w is not None:
            v = v * w.float().view(-1, size)
        v = (v * scale).reshape(T, C).to(dtype)
        return v if out is None else out.copy_(v)
    return _group_norm(y, None, 0.0, y.stride(0), size, w, groups, size, eps, z, scale, out, dtype)


def map_difference(o: torch.Tensor, lam: float, eps: float, scale: float, dtype: torch.dtype,
                   out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """o [T, 2 H, D], the outputs of two attention maps per head -> [T, H * D]: map 1 minus ``lam`` times map 2, RMS-normed
    per head without a weight, times ``scale``."""
    T, H2, D = o.shape
    if not o.is_cuda:
        v = o.float().view(T, H2 // 2, 2, D)
        v = v[:, :, 0] - lam * v[:, :, 1]
        v = (v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * scale).reshape(T, -1).to(dtype)
        return v if out is None else out.copy_(v)
    y = o.view(T, H2 * D)
    return _group_norm(y, y[:, D:], lam, y.stride(0), 2 * D, None, H2 // 2, D, eps, None, scale, out, dtype)


def _group_norm(y, y2, lam, y_stride, y_group, w, groups, size, eps, z, scale, out, dtype):
    T = y.shape[0]
    if dtype not in _DTYPES or y.dtype not in (dtype, torch.float32) or any(t is not None and t.dtype != dtype for t in (w, z)) \
            or y.stride(1) != 1 or (z is not None and z.stride(1) != 1):
        raise TypeError("group_norm: rows of the result's type or fp32, gate and weight of the result's type")
    if w is not None and w.numel() not in (size, size * groups):
        raise ValueError("group_norm: a weight per channel or per channel of a part")
    if out is None:
        out = torch.empty((T, groups * size), dtype=dtype, device=y.device)
    if out.dtype != dtype or out.stride(1) != 1 or tuple(out.shape) != (T, groups * size):
        raise TypeError("group_norm: result rows are dense")
    a = _GroupNormArgs(
        y=y.data_ptr(), y2=_native.ptr(y2), z=_native.ptr(z), w=_native.ptr(w), out=out.data_ptr(), rows=T, y_stride=y_stride,
        y_group=y_group, z_stride=0 if z is None else z.stride(0), out_stride=out.stride(0), w_len=0 if w is None else w.numel(),
        groups=groups, size=size, in_f32=int(y.dtype == torch.float32), dtype=_DTYPES[dtype], lam=lam, eps=eps, scale=scale)
    rc = _native.lib().b200_group_norm(ctypes.addressof(a), _native.stream_ptr())
    _native.check(rc, "group_norm")
    _native.count_launch()
    return out
