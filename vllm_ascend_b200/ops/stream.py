"""Ops of decoders with an fp32 residual stream: the pass between two sub-layers (norm of the sub-layer's
output, sum, norm of the next input), the per-layer token input and the gated read-out norm of delta-rule
heads.  CUDA kernels (bf16 or fp32 activations) on GPU tensors, PyTorch definitions on the CPU."""
from __future__ import annotations

from ctypes import c_float, c_int, c_long, c_void_p
from typing import Optional

import torch
import torch.nn.functional as F

from .. import _native

P, I, L, Fl = c_void_p, c_int, c_long, c_float
_native.register_signature("b200_stream_norm", [P, P, L, I, P, P, Fl, I, P, P, L, Fl, I, P, P, P, L, I, I, I, Fl, I, P, P])
_native.register_signature("b200_stream_mix", [P, P, L, I, P, P, P, P, I, P, P, L, Fl, P, P, L, P, I, P, P, P, L, I, I, I,
                                               Fl, I, P, P])
_native.register_signature("b200_side_gate", [P, L, P, P, L, L, L, P, L, I, I, P, P])
_native.register_signature("b200_gated_head_norm", [P, P, L, P, P, L, I, I, Fl, I, P])

_KIND = {None: 0, "layer": 1, "rms": 2, "plain": 3}


class NormSpec:
    """A norm as the stream kernel takes it: kind "layer" (weight, bias), "rms" (weight; over ``groups`` equal parts
    of the row, each by itself) or "plain" (the row as it is)."""
    __slots__ = ("kind", "weight", "bias", "groups")

    def __init__(self, kind: str, weight: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None, groups: int = 1):
        if kind not in ("layer", "rms", "plain"):
            raise ValueError(f"unknown norm kind {kind!r}")
        if groups < 1 or (groups > 1 and (kind != "rms" or bias is not None or weight.shape[0] % groups)):
            raise ValueError(f"a {kind} norm of this width does not come in {groups} groups")
        self.kind, self.weight, self.bias, self.groups = kind, weight, bias, groups


#: the row itself, rounded to the activation type
PLAIN = NormSpec("plain")


def _dtype_code(dtype: torch.dtype) -> int:
    if dtype == torch.bfloat16:
        return 0
    if dtype == torch.float32:
        return 1
    raise TypeError(f"the kernel takes bf16 or fp32 activations, not {dtype}")


def _norm_ref(v: torch.Tensor, n: NormSpec, eps: float) -> torch.Tensor:
    if n.kind == "plain":
        return v
    if n.kind == "layer":
        v = v - v.mean(-1, keepdim=True)
    if n.groups > 1:
        parts = v.unflatten(-1, (n.groups, -1))
        return (parts * torch.rsqrt((parts * parts).mean(-1, keepdim=True) + eps)).flatten(-2) * n.weight.float()
    v = v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * n.weight.float()
    return v if n.bias is None else v + n.bias.float()


def stream_norm(r: torch.Tensor, y: Optional[torch.Tensor], post: Optional[NormSpec], nxt: Optional[NormSpec], eps: float,
                dtype: torch.dtype, embed: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None,
                embed_scale: float = 1.0, embed_set: bool = False, post_scale: float = 1.0) -> Optional[torch.Tensor]:
    """One token-wise pass over the residual stream ``r`` (fp32 [T, W], updated in place):

        r += post_scale * post(y)          when a sub-layer output ``y`` [T, W] is given
        r += embed_scale * embed[ids]      when ``embed`` is given (``embed_set``: r is set to it instead)
        return nxt(r) as ``dtype``         (None: nothing is returned)

    ``ids`` None: row t of ``embed`` belongs to token t."""
    T, W = r.shape
    if r.dtype != torch.float32 or not r.is_contiguous():
        raise TypeError("the residual stream is a contiguous fp32 tensor")
    if not r.is_cuda:
        v = None
        if y is not None:
            v = _norm_ref(y.float(), post, eps) * post_scale
        if embed is not None:
            e = (embed if ids is None else embed[ids]).float() * embed_scale
            v = e if v is None else v + e
        if v is not None:
            r.copy_(v if embed_set else r + v)
        return None if nxt is None else _norm_ref(r, nxt, eps).to(dtype)
    code = _dtype_code(dtype)
    for t in (y, embed, *((post.weight, post.bias) if post else ()), *((nxt.weight, nxt.bias) if nxt else ())):
        if t is not None and t.dtype != dtype:
            raise TypeError(f"stream_norm: {t.dtype} operand beside {dtype} activations")
    if y is not None and y.stride(-1) != 1:
        y = y.contiguous()
    if embed is not None and not embed.is_contiguous():
        embed = embed.contiguous()
    x = None if nxt is None else torch.empty((T, W), dtype=dtype, device=r.device)
    emb = 0 if embed is None else (1 if embed_set else 2)
    rc = _native.lib().b200_stream_norm(
        r.data_ptr(), _native.ptr(y), 0 if y is None else y.stride(0), _KIND[post.kind] if y is not None else 0,
        _native.ptr(post.weight if y is not None else None), _native.ptr(post.bias if y is not None else None),
        float(post_scale), emb, _native.ptr(ids), _native.ptr(embed), 0 if embed is None else embed.shape[0],
        float(embed_scale), 0 if nxt is None else _KIND[nxt.kind], _native.ptr(nxt.weight if nxt else None),
        _native.ptr(nxt.bias if nxt else None), _native.ptr(x), T, W, post.groups if y is not None else 1,
        nxt.groups if nxt else 1, float(eps), code,
        _native.status_word(r.device).data_ptr(), _native.stream_ptr())
    _native.check(rc, "stream_norm")
    _native.count_launch()
    return x


class StreamMix:
    """How a sub-layer reads from and writes to S parallel streams (fp32): input sum_s read[s] x_s; afterwards
    x_t = sum_s mix[s, t] x_s + write[t] y."""
    __slots__ = ("read", "write", "mix")

    def __init__(self, read: torch.Tensor, write: torch.Tensor, mix: torch.Tensor):
        self.read, self.write, self.mix = read, write, mix


def stream_mix(r: torch.Tensor, y: Optional[torch.Tensor], post: Optional[NormSpec], joined: Optional[StreamMix],
               reader: Optional[StreamMix], nxt: Optional[NormSpec], eps: float, dtype: torch.dtype,
               embed: Optional[torch.Tensor] = None, ids: Optional[torch.Tensor] = None, embed_scale: float = 1.0,
               pos_table: Optional[torch.Tensor] = None, positions: Optional[torch.Tensor] = None,
               store: bool = True) -> Optional[torch.Tensor]:
    """One token-wise pass over ``r`` (fp32 [T, S, W], S parallel residual streams, updated in place):

        x_t = sum_s joined.mix[s, t] x_s + joined.write[t] post(y)      when a sub-layer output ``y`` is given
        x_t = embed_scale * embed[ids] + pos_table[positions]           when ``embed`` is given
        return nxt(sum_s reader.read[s] x_s) as ``dtype``               (reader None: the sum; nxt None: nothing)

    ``store`` False: the streams are not needed afterwards and may be left as they were."""
    T, S, W = r.shape
    if r.dtype != torch.float32 or not r.is_contiguous():
        raise TypeError("the residual streams are a contiguous fp32 tensor")
    if not r.is_cuda:
        x = r
        if embed is not None:
            e = (embed if ids is None else embed[ids]).float() * embed_scale
            if pos_table is not None:
                if positions.numel() and (int(positions.max()) >= pos_table.shape[0] or int(positions.min()) < 0):
                    raise IndexError("position outside the position table")
                e = e + pos_table[positions].float()
            x = e[:, None].expand(T, S, W)
        elif y is not None:
            x = torch.einsum("tsw,sz->tzw", r, joined.mix) + joined.write[:, None] * _norm_ref(y.float(), post, eps)[:, None]
        u = x.sum(1) if reader is None else torch.einsum("s,tsw->tw", reader.read, x)
        if store and x is not r:
            r.copy_(x)
        return None if nxt is None else _norm_ref(u, nxt, eps).to(dtype)
    if any(n is not None and n.groups > 1 for n in (post, nxt)):
        raise NotImplementedError("norms in groups on several streams")
    code = _dtype_code(dtype)
    for t in (y, embed, pos_table, *((post.weight, post.bias) if post else ()), *((nxt.weight, nxt.bias) if nxt else ())):
        if t is not None and t.dtype != dtype:
            raise TypeError(f"stream_mix: {t.dtype} operand beside {dtype} activations")
    for m in (joined, reader):
        if m is not None and not (m.read.dtype == m.write.dtype == m.mix.dtype == torch.float32):
            raise TypeError("stream_mix: the mixing weights are fp32")
    if y is not None and y.stride(-1) != 1:
        y = y.contiguous()
    if embed is not None and not embed.is_contiguous():
        embed = embed.contiguous()
    x = None if nxt is None else torch.empty((T, W), dtype=dtype, device=r.device)
    has = y is not None
    rc = _native.lib().b200_stream_mix(
        r.data_ptr(), _native.ptr(y), 0 if y is None else y.stride(0), _KIND[post.kind] if has else 0,
        _native.ptr(post.weight if has else None), _native.ptr(post.bias if has else None),
        _native.ptr(joined.mix if has else None), _native.ptr(joined.write if has else None), int(embed is not None),
        _native.ptr(ids), _native.ptr(embed), 0 if embed is None else embed.shape[0], float(embed_scale),
        _native.ptr(positions if pos_table is not None else None), _native.ptr(pos_table),
        0 if pos_table is None else pos_table.shape[0], _native.ptr(reader.read if reader else None),
        0 if nxt is None else _KIND[nxt.kind], _native.ptr(nxt.weight if nxt else None),
        _native.ptr(nxt.bias if nxt else None), _native.ptr(x), T, S, W, int(store), float(eps), code,
        _native.status_word(r.device).data_ptr(), _native.stream_ptr())
    _native.check(rc, "stream_mix")
    _native.count_launch()
    return x


def side_gate(a: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, offset: int) -> torch.Tensor:
    """gelu_tanh(a) * table[ids][:, offset : offset + D] with a [T, D]."""
    T, D = a.shape
    if not a.is_cuda:
        e = table[ids][:, offset:offset + D]
        return (F.gelu(a.float(), approximate="tanh") * e.float()).to(a.dtype)
    if table.dtype != a.dtype or not table.is_contiguous() or a.stride(1) != 1:
        raise TypeError("side_gate takes a dense table of the activations' type")
    out = torch.empty((T, D), dtype=a.dtype, device=a.device)
    rc = _native.lib().b200_side_gate(
        a.data_ptr(), a.stride(0), ids.data_ptr(), table.data_ptr(), table.shape[1], table.shape[0], int(offset),
        out.data_ptr(), T, D, _dtype_code(a.dtype), _native.status_word(a.device).data_ptr(), _native.stream_ptr())
    _native.check(rc, "side_gate")
    _native.count_launch()
    return out


def gated_head_norm(o: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """rms_norm(o) * weight * silu(z) per head: o [T, H, D] dense, z [T, H * D] (rows may be strided) ->
    [T, H * D]."""
    T, H, D = o.shape
    if not o.is_cuda:
        v = o.float()
        v = v * torch.rsqrt((v * v).mean(-1, keepdim=True) + eps) * weight.float()
        return (v * F.silu(z.reshape(T, H, D).float())).reshape(T, H * D).to(o.dtype)
    if not o.is_contiguous() or z.stride(1) != 1 or not (o.dtype == z.dtype == weight.dtype):
        raise TypeError("gated_head_norm takes dense heads and operands of one type")
    out = torch.empty((T, H * D), dtype=o.dtype, device=o.device)
    rc = _native.lib().b200_gated_head_norm(o.data_ptr(), z.data_ptr(), z.stride(0), weight.data_ptr(), out.data_ptr(),
                                            T, H, D, float(eps), _dtype_code(o.dtype), _native.stream_ptr())
    _native.check(rc, "gated_head_norm")
    _native.count_launch()
    return out
