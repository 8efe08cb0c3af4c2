"""Paged grouped-query attention with options: sliding window that keeps the first tokens of a sequence, capped
scores, a learned bias by distance, an attention sink, a gate per head on the output, value heads of another
size than the key heads, keys shared by several value heads.  And the pass in front of it: short convolution, q / k norm
(over all heads or head by head), rotary positions, factors by position, wide queries, cache write.

GPU tensors run the kernels of csrc/qkv_prep.cu and csrc/attention_variant.cu (fp32, odd sizes) or the tcgen05
kernels of csrc/attention_tc.cu, csrc/attention_decode_tc.cu and (keys above 128 dimensions) csrc/attention_wide.cu
(bf16); CPU tensors run the PyTorch definitions
below.  The reference's paged attention has the window and the mask (vllm_ascend/attention/attention_v1.py:1341-1472)."""
from __future__ import annotations

import ctypes
import math
from ctypes import c_void_p
from dataclasses import dataclass
from typing import Optional

import torch

from .. import _native
from ..ops import linear_attn as la
from ..ops import reference as ref


class _PrepArgs(ctypes.Structure):
    """QkvPrepArgs of csrc/qkv_prep.cu."""
    _fields_ = _native.struct_fields(
        pointers="qkv conv_w state cu slots has_init q_norm k_norm positions cos_sin slot_mapping q_out k_cache v_cache sums "
                 "mix q_scale",
        longs="qkv_stride state_rows cache_slots k_block k_tok k_head v_block v_tok v_head tokens",
        ints="num_seqs taps heads kv_heads dim vdim q_norm_dims k_norm_dims values_from_keys rot cos_rows block_size "
             "uniform phase dtype head_norm v_heads key_parts part_run out_heads q_scale_rows", floats="eps")


class _AttnArgs(ctypes.Structure):
    """AttnVariantArgs of csrc/attention.h."""
    _fields_ = _native.struct_fields(
        pointers="q k_cache v_cache out cu seq_lens block_table row_seq row_kv_len bias sink gate scratch",
        longs="q_stride out_stride gate_stride num_blocks tokens k_block k_tok k_head v_block v_tok v_head",
        ints="num_seqs max_blocks block_size heads kv_heads dim vdim window keep_first bias_len num_splits dtype key_heads "
             "out_f32", floats="scale softcap out_scale")


_ENTRY = [c_void_p, c_void_p, c_void_p]
for _name in ("b200_qkv_prep", "b200_attention_variant", "b200_attention_variant_prefill",
              "b200_attention_variant_decode", "b200_attention_wide_prefill", "b200_attention_wide_decode"):
    _native.register_signature(_name, _ENTRY)


def _launch(entry: str, args: ctypes.Structure, device, launches: int = 1) -> None:
    rc = getattr(_native.lib(), entry)(ctypes.addressof(args), _native.status_word(device).data_ptr(), _native.stream_ptr())
    _native.check(rc, entry[5:])
    _native.count_launch(launches)


@dataclass
class AttnOptions:
    scale: float
    window: int = 0                          # 0: all earlier tokens
    keep_first: int = 0                      # with a window: the first tokens that stay visible
    softcap: float = 0.0                     # 0: scores as they are
    bias: Optional[torch.Tensor] = None      # fp32 [H, n]: added to the score by distance (the last entry from n - 1 on)
    sink: Optional[torch.Tensor] = None      # fp32 [H]: exp(sink) joins the softmax denominator
    out_scale: float = 1.0                   # factor of the result
    out_f32: bool = False                    # the result is fp32 whatever the type of queries and caches

    @property
    def plain(self) -> bool:
        return not self.keep_first and not self.softcap and self.bias is None and self.sink is None


def distance_buckets(rows: int, largest: int, count: int) -> list[int]:
    """Bucket of every distance 0 .. count - 1 in a table of ``rows`` rows: one bucket each below rows / 2,
    logarithmic buckets up to ``largest`` from there on."""
    half = rows // 2
    out = []
    for n in range(count):
        if n < half:
            out.append(n)
        elif largest <= half or half == 0:
            out.append(rows - 1)
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(largest / half) * (rows - half))))
    return out


def distance_table(rel: torch.Tensor, largest: int, count: int) -> torch.Tensor:
    """rel [rows, H] -> fp32 [H, n] indexed by distance; from the first distance of the last bucket on (or from
    ``count`` - 1 on) the bias stays the same."""
    rows = rel.shape[0]
    idx = distance_buckets(rows, largest, max(1, min(count, max(largest, rows) + 1)))
    if rows - 1 in idx:
        idx = idx[:idx.index(rows - 1) + 1]
    return rel.float()[torch.tensor(idx, device=rel.device)].T.contiguous()


# ---------------------------------------------------------------- q / k / v in front of the attention
@dataclass
class PrepSpec:
    """What happens to the rows [q | k | v | rest] of a fused projection."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    eps: float
    q_norm: Optional[torch.Tensor]           # [heads * dim], [kv_heads * dim]; None: no norm
    k_norm: Optional[torch.Tensor]
    norm_dims: tuple                         # widths the means are over (all ranks' heads)
    values_from_keys: bool = False           # no v columns: the values are the keys before norm and rotation
    conv: Optional[torch.Tensor] = None      # [columns of q, k (and v), taps]
    rot_dims: int = 0
    cos_sin: Optional[torch.Tensor] = None   # fp32 [positions, rot_dims]
    head_norm: bool = False                  # every head by itself, q_norm and k_norm are [dim]; without convolution
    v_heads: Optional[int] = None            # value heads (None: kv_heads)
    # wide keys: a cache row holds key_parts projected keys side by side, and part c of an output head's query is the
    # sum of mix[head, g] q_g over the projected heads g with (g // part_run) % key_parts == c (mix None: identity)
    key_parts: int = 1
    part_run: int = 1
    mix: Optional[torch.Tensor] = None       # fp32 [output heads, heads]
    q_scale: Optional[torch.Tensor] = None   # fp32 [positions]: factor of the queries

    @property
    def values(self) -> int:
        return self.kv_heads if self.v_heads is None else self.v_heads

    @property
    def columns(self) -> int:
        return self.heads * self.dim + self.kv_heads * self.dim + (0 if self.values_from_keys else self.values * self.vdim)

    @property
    def key_heads(self) -> int:
        return self.kv_heads // self.key_parts

    @property
    def out_heads(self) -> int:
        return self.heads if self.mix is None else self.mix.shape[0]

    @property
    def spread(self) -> bool:
        """Head by head with options of ``qkv_spread_kernel``."""
        return self.q_norm is None or self.key_parts > 1 or self.mix is not None or self.q_scale is not None \
            or self.values != self.kv_heads


def _prep_ref(s: PrepSpec, qkv, meta, k_cache, v_cache, state, reduce_sums):
    T, nq, nk = qkv.shape[0], s.heads * s.dim, s.kv_heads * s.dim
    x = qkv[:, :s.columns]
    if s.conv is not None:
        slots, init = meta.state_slots, meta.has_initial_state
        if state is None:                    # one tap: nothing is kept
            x = (x.float() * s.conv.float()[:, 0]).to(x.dtype)
        else:
            x = la.causal_conv1d_ref(x, s.conv, None, state, meta.query_start_loc, slots, init, act=False)
    q, k = x[:, :nq].float(), x[:, nq:nq + nk].float()
    v = x[:, nq:nq + nk] if s.values_from_keys else x[:, nq + nk:]
    if s.q_norm is None:
        q, k = q.reshape(T, s.heads, s.dim), k.reshape(T, s.kv_heads, s.dim)
    elif s.head_norm:
        q, k = (ref.rms_norm(t.reshape(T, -1, s.dim), w.float(), s.eps)[0] for t, w in ((q, s.q_norm), (k, s.k_norm)))
    else:
        sums = torch.stack([(q * q).sum(-1), (k * k).sum(-1)], -1)
        if reduce_sums is not None:
            sums = reduce_sums(sums)
        inv = torch.rsqrt(sums / torch.tensor(s.norm_dims, dtype=torch.float32) + s.eps)
        q = (q * inv[:, :1] * s.q_norm.float()).view(T, s.heads, s.dim)
        k = (k * inv[:, 1:] * s.k_norm.float()).view(T, s.kv_heads, s.dim)
    if s.rot_dims:
        q = ref.apply_rope_interleaved(q, meta.positions, s.cos_sin, s.rot_dims)
        k = ref.apply_rope_interleaved(k, meta.positions, s.cos_sin, s.rot_dims)
    if s.q_scale is not None:
        q = q * s.q_scale[meta.positions][:, None, None]
    if s.key_parts > 1 or s.mix is not None:
        mix = torch.eye(s.heads) if s.mix is None else s.mix
        part = torch.nn.functional.one_hot(torch.arange(s.heads) // s.part_run % s.key_parts, s.key_parts).float()
        q = torch.einsum("og,gp,tgd->topd", mix, part, q).flatten(2)
        k = k.reshape(T, s.key_heads, s.key_parts * s.dim)
    keep = meta.slot_mapping >= 0
    slot = meta.slot_mapping[keep]
    bs = k_cache.shape[1]
    k_cache[slot // bs, slot % bs] = k[keep].to(k_cache.dtype)
    v_cache[slot // bs, slot % bs] = v.reshape(T, s.values, s.vdim)[keep].to(v_cache.dtype)
    return q.to(qkv.dtype)


def qkv_prep(s: PrepSpec, qkv: torch.Tensor, meta, k_cache: torch.Tensor, v_cache: torch.Tensor,
             state: Optional[torch.Tensor] = None, reduce_sums=None) -> torch.Tensor:
    """qkv [T, columns ...] -> q [T, output heads, key parts * dim]; keys and values go to their cache slots (slot < 0:
    not stored).
    ``state`` [slots, taps - 1, columns] holds the last convolution inputs of every sequence and is updated.
    ``reduce_sums`` (tensor parallelism) completes the sums of squares [T, 2] of q and k over the ranks."""
    if not qkv.is_cuda:
        return _prep_ref(s, qkv, meta, k_cache, v_cache, state, reduce_sums)
    T, dev, dt = qkv.shape[0], qkv.device, qkv.dtype
    taps = 0 if s.conv is None else s.conv.shape[1]
    same = [k_cache, v_cache] + [t for t in (s.q_norm, s.k_norm, s.conv, state) if t is not None]
    if dt not in (torch.bfloat16, torch.float32) or any(t.dtype != dt for t in same) or qkv.stride(1) != 1:
        raise TypeError("qkv_prep takes bf16 or fp32 rows with weights, state and caches of the same type")
    if k_cache.stride(3) != 1 or v_cache.stride(3) != 1 or qkv.shape[1] < s.columns:
        raise ValueError("qkv_prep: cache rows must be dense and the projection wide enough")
    if taps > 1 and (state is None or tuple(state.shape[1:]) != (taps - 1, s.columns) or not state.is_contiguous()):
        raise ValueError("qkv_prep: convolution state of another shape")
    widths = (s.dim, s.dim) if s.head_norm else (s.heads * s.dim, s.kv_heads * s.dim)
    if s.q_norm is not None and (s.q_norm.numel(), s.k_norm.numel()) != widths \
            or ((s.head_norm or s.q_norm is None) and (taps or reduce_sums is not None)):
        raise ValueError("qkv_prep: norm weights of another size, or a norm per head with a convolution")
    if s.spread and ((s.q_norm is not None and not s.head_norm) or s.values_from_keys or s.kv_heads % s.key_parts or any(
            t is not None and (t.dtype != torch.float32 or not t.is_contiguous()) for t in (s.mix, s.q_scale))):
        raise ValueError("qkv_prep: wide queries take norms per head or none, and dense fp32 factors")
    if s.mix is not None and s.mix.shape[1] != s.heads:
        raise ValueError("qkv_prep: the mixing matrix has a column per projected head")
    q = torch.empty((T, s.out_heads, s.key_parts * s.dim), dtype=dt, device=dev)
    if T == 0:
        return q
    B = meta.num_reqs
    a = _PrepArgs(
        qkv=qkv.data_ptr(), conv_w=_native.ptr(s.conv), state=_native.ptr(state), cu=meta.query_start_loc.data_ptr(),
        slots=_native.ptr(meta.state_slots), has_init=_native.ptr(meta.has_initial_state), q_norm=_native.ptr(s.q_norm),
        k_norm=_native.ptr(s.k_norm), positions=meta.positions.data_ptr(),
        cos_sin=_native.ptr(s.cos_sin) if s.rot_dims else None, slot_mapping=meta.slot_mapping.data_ptr(),
        q_out=q.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), qkv_stride=qkv.stride(0),
        state_rows=0 if state is None else state.shape[0], cache_slots=k_cache.shape[0] * k_cache.shape[1],
        k_block=k_cache.stride(0), k_tok=k_cache.stride(1), k_head=k_cache.stride(2), v_block=v_cache.stride(0),
        v_tok=v_cache.stride(1), v_head=v_cache.stride(2), tokens=T, num_seqs=B, taps=taps, heads=s.heads,
        kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, q_norm_dims=int(s.norm_dims[0]), k_norm_dims=int(s.norm_dims[1]),
        values_from_keys=int(s.values_from_keys), rot=s.rot_dims, cos_rows=s.cos_sin.shape[0] if s.rot_dims else 0,
        block_size=k_cache.shape[1], uniform=int(meta.max_query_len <= 1 and T == B), dtype=int(dt == torch.float32),
        head_norm=int(s.head_norm), eps=s.eps, mix=_native.ptr(s.mix), q_scale=_native.ptr(s.q_scale),
        v_heads=s.values, key_parts=s.key_parts if s.spread else 0, part_run=s.part_run, out_heads=s.out_heads,
        q_scale_rows=0 if s.q_scale is None else s.q_scale.shape[0])
    if reduce_sums is None:
        _launch("b200_qkv_prep", a, dev)
        return q
    sums = torch.empty((T, 2), dtype=torch.float32, device=dev)
    a.sums, a.phase = sums.data_ptr(), 1
    _launch("b200_qkv_prep", a, dev)
    sums = reduce_sums(sums).contiguous()
    a.sums, a.phase = sums.data_ptr(), 2
    _launch("b200_qkv_prep", a, dev)
    return q


# ---------------------------------------------------------------- attention
def _attention_ref(q, k_cache, v_cache, meta, o: AttnOptions, gate, out):
    T, H, _ = q.shape
    Hkv, Dv = v_cache.shape[2], v_cache.shape[3]
    owner = torch.arange(H, device=q.device) // (H // Hkv)
    key_owner = owner * k_cache.shape[2] // Hkv
    qsl, sls = meta.query_start_loc_cpu, meta.seq_lens_cpu
    for b in range(meta.num_reqs):
        qs, qe, sl = int(qsl[b]), int(qsl[b + 1]), int(sls[b])
        if qe <= qs:
            continue
        k = ref.gather_kv(k_cache, meta.block_table[b], sl).float()[:, key_owner]
        v = ref.gather_kv(v_cache, meta.block_table[b], sl).float()[:, owner]
        s = torch.einsum("qhd,khd->hqk", q[qs:qe].float(), k) * o.scale
        if o.softcap:
            s = o.softcap * torch.tanh(s / o.softcap)
        dist = torch.arange(sl - (qe - qs), sl)[:, None] - torch.arange(sl)[None, :]
        if o.bias is not None:
            s = s + o.bias[:, dist.clamp(0, o.bias.shape[1] - 1)]
        seen = dist >= 0
        if o.window:
            seen &= (dist < o.window) | (torch.arange(sl) < o.keep_first)[None, :]
        s = s.masked_fill(~seen[None], float("-inf"))
        if o.sink is not None:
            s = torch.cat([s, o.sink.view(H, 1, 1).expand(H, qe - qs, 1)], -1)
        p = torch.softmax(s, -1)[..., :sl]
        out[qs:qe] = (torch.einsum("hqk,khd->qhd", p, v) * o.out_scale).to(out.dtype)
    if gate is not None:
        out *= torch.sigmoid(gate.float())[:, :, None].to(out.dtype)
    return out


def _args(q, k_cache, v_cache, meta, o: AttnOptions, gate, out) -> _AttnArgs:
    for t, w in ((o.bias, 2), (o.sink, 1)):
        if t is not None and (t.dtype != torch.float32 or t.dim() != w or t.shape[0] != q.shape[1] or not t.is_contiguous()):
            raise TypeError("bias and sink are dense fp32 tensors over the heads")
    if any(t is not None and t.dtype != q.dtype for t in (k_cache, v_cache, gate)) or out.dtype != _out_dtype(q, o):
        raise TypeError("queries, caches, gate and output are of one type")
    if v_cache.shape[2] % k_cache.shape[2] or q.shape[1] % v_cache.shape[2] or q.shape[2] != k_cache.shape[3]:
        raise ValueError("value heads share key heads, and query heads value heads")
    if out.stride(2) != 1 or out.stride(1) != out.shape[2]:
        raise ValueError("heads of the output are dense")
    if gate is not None and gate.stride(1) != 1:
        gate = gate.contiguous()
    a = _AttnArgs(
        q=q.data_ptr(), k_cache=k_cache.data_ptr(), v_cache=v_cache.data_ptr(), out=out.data_ptr(),
        cu=meta.query_start_loc.data_ptr(), seq_lens=meta.seq_lens.data_ptr(), block_table=meta.block_table.data_ptr(),
        bias=_native.ptr(o.bias), sink=_native.ptr(o.sink), gate=_native.ptr(gate), q_stride=q.stride(0),
        out_stride=out.stride(0), gate_stride=0 if gate is None else gate.stride(0), num_blocks=k_cache.shape[0],
        tokens=q.shape[0], k_block=k_cache.stride(0), k_tok=k_cache.stride(1), k_head=k_cache.stride(2),
        v_block=v_cache.stride(0), v_tok=v_cache.stride(1), v_head=v_cache.stride(2), num_seqs=meta.num_reqs,
        max_blocks=meta.block_table.stride(0), block_size=k_cache.shape[1], heads=q.shape[1], kv_heads=v_cache.shape[2],
        dim=q.shape[2], vdim=v_cache.shape[3], window=o.window, keep_first=o.keep_first if o.window else 0,
        bias_len=0 if o.bias is None else o.bias.shape[1], num_splits=1, dtype=int(q.dtype == torch.float32),
        scale=o.scale, softcap=o.softcap, key_heads=k_cache.shape[2], out_f32=int(out.dtype == torch.float32),
        out_scale=o.out_scale)
    a.hold = gate                    # alive until the launch
    return a


def _out_dtype(q: torch.Tensor, o: AttnOptions) -> torch.dtype:
    return torch.float32 if o.out_f32 else q.dtype


def _new_out(q: torch.Tensor, v_cache: torch.Tensor, o: AttnOptions) -> torch.Tensor:
    return torch.empty((q.shape[0], q.shape[1], v_cache.shape[3]), dtype=_out_dtype(q, o), device=q.device)


def variant_attention_simple(q, k_cache, v_cache, meta, o: AttnOptions, gate=None, out=None) -> torch.Tensor:
    """CUDA-core kernel: any sizes, bf16 or fp32."""
    from .mla import _batch_rows
    T, H, _ = q.shape
    if q.stride(2) != 1 or q.stride(1) != q.shape[2] or k_cache.stride(3) != 1 or v_cache.stride(3) != 1:
        raise ValueError("heads and cache rows must be dense")
    if out is None:
        out = _new_out(q, v_cache, o)
    a = _args(q, k_cache, v_cache, meta, o, gate, out)
    row_seq, row_kv = _batch_rows(meta, T, q.device)
    a.row_seq, a.row_kv_len = row_seq.data_ptr(), row_kv.data_ptr()
    _launch("b200_attention_variant", a, q.device)
    return out


def _tma_ok(q, k_cache, v_cache, out) -> bool:
    """True when the tcgen05 kernels can load these tensors (TMA: 16-byte strides and bases)."""
    D, Dv, bs = q.shape[2], v_cache.shape[3], k_cache.shape[1]
    strides = [q.stride(0), out.stride(0), *k_cache.stride()[:3], *v_cache.stride()[:3]]
    return (q.dtype == torch.bfloat16 and D % 8 == 0 and Dv % 8 == 0 and D >= 8 and 8 <= Dv <= 128
            and q.shape[1] // v_cache.shape[2] <= 128 and bs >= 8 and (128 % bs == 0 or bs % 128 == 0)
            and all(x % 8 == 0 for x in strides) and all(t.data_ptr() % 16 == 0 for t in (q, k_cache, v_cache, out))
            and k_cache.stride(3) == v_cache.stride(3) == 1)


def _kernels(q, k_cache, v_cache, out, o: AttnOptions, gate=None) -> tuple[Optional[str], Optional[str]]:
    """(kernel for several rows per sequence, kernel for one): "tile" (keys up to 128 dimensions, all options), "wide"
    (wider or shared key rows) or None (CUDA cores)."""
    if not _tma_ok(q, k_cache, v_cache, out):
        return None, None
    D, H, Hv, Hk = q.shape[2], q.shape[1], v_cache.shape[2], k_cache.shape[2]
    plain, columns = o.plain and gate is None, H // Hk
    many = "tile" if D <= 128 else "wide" if D <= 512 and plain else None
    if plain and (D > 128 or Hk < Hv) and D <= 1024 and columns <= 32 and (2 + Hv // Hk) * (16 if columns <= 16 else 32) <= 512:
        return many, "wide"
    return many, "tile" if D <= 128 and H // Hv <= 16 else None


def decode_splits(num_seqs: int, kv_heads: int, o: AttnOptions, max_keys: int, device) -> int:
    """Splits of the key range of a decode batch: about one work item per SM, none below two tiles.  Depends on
    the batch size and the capacity only, so that a captured graph and an eager step agree."""
    from ..batch_invariant import is_batch_invariant
    if is_batch_invariant():
        return 1
    keys = min(max_keys, o.window + 127 + ((o.keep_first + 127) // 128) * 128) if o.window else max_keys
    tiles = (keys + 127) // 128
    sms = torch.cuda.get_device_properties(device).multi_processor_count
    return max(1, min((sms + num_seqs * kv_heads - 1) // (num_seqs * kv_heads), tiles // 2, 32))


def reserve_decode_scratch(device, max_seqs: int, heads: int, kv_heads: int, vdim: int, o: AttnOptions, max_keys: int) -> None:
    """Split-KV scratch of decode batches of up to ``max_seqs`` sequences, allocated before graphs are captured."""
    from .. import ops
    worst = 0
    for b in range(1, max_seqs + 1):
        n = decode_splits(b, kv_heads, o, max_keys, device)
        if n > 1:
            worst = max(worst, b * heads * n * (vdim + 1) * 4)
    if worst:
        ops.reserve_attention_scratch(device, worst)


def variant_attention_decode(q, k_cache, v_cache, meta, o: AttnOptions, gate=None, out=None, num_seqs=None,
                             num_splits: int = 0) -> torch.Tensor:
    """tcgen05 decode kernel: the first ``num_seqs`` sequences of the step, one query row each."""
    from .. import ops
    num_seqs = meta.num_reqs if num_seqs is None else num_seqs
    if out is None:
        out = _new_out(q, v_cache, o)
    a = _args(q, k_cache, v_cache, meta, o, gate, out)
    a.num_seqs = num_seqs
    a.num_splits = num_splits or decode_splits(num_seqs, a.kv_heads, o, meta.block_table.shape[1] * a.block_size, q.device)
    if a.num_splits > 1:
        a.scratch = ops._get_scratch(q.device, num_seqs * a.heads * a.num_splits * (a.vdim + 1) * 4).data_ptr()
    _launch("b200_attention_variant_decode", a, q.device, 2 if a.num_splits > 1 else 1)
    return out


def wide_attention_decode(q, k_cache, v_cache, meta, o: AttnOptions, out=None, num_seqs=None, num_splits: int = 0) -> torch.Tensor:
    """tcgen05 decode kernel for wide or shared key rows: the first ``num_seqs`` sequences, one query row each."""
    from .. import ops
    num_seqs = meta.num_reqs if num_seqs is None else num_seqs
    if out is None:
        out = _new_out(q, v_cache, o)
    a = _args(q, k_cache, v_cache, meta, o, None, out)
    a.num_seqs = num_seqs
    a.num_splits = num_splits or decode_splits(num_seqs, a.key_heads, o, meta.block_table.shape[1] * a.block_size, q.device)
    if a.num_splits > 1:
        a.scratch = ops._get_scratch(q.device, num_seqs * a.heads * a.num_splits * (a.vdim + 1) * 4).data_ptr()
    _launch("b200_attention_wide_decode", a, q.device, 2 if a.num_splits > 1 else 1)
    return out


def variant_attention_prefill(q, k_cache, v_cache, meta, o: AttnOptions, gate=None, out=None,
                              first_seq: int = 0, wide: bool = False) -> torch.Tensor:
    """tcgen05 tile kernel (``wide``: for keys of more than 128 dimensions): every sequence of the step from
    ``first_seq`` on, any number of query rows each."""
    if out is None:
        out = _new_out(q, v_cache, o)
    a = _args(q, k_cache, v_cache, meta, o, gate, out)
    a.num_seqs = meta.num_reqs - first_seq
    a.cu, a.seq_lens = a.cu + 4 * first_seq, a.seq_lens + 4 * first_seq
    a.block_table += 4 * first_seq * a.max_blocks
    _launch("b200_attention_wide_prefill" if wide else "b200_attention_variant_prefill", a, q.device)
    return out


def variant_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, meta, o: AttnOptions,
                      gate: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of every query row of the step over its sequence's paged keys: q [T, H, D] -> [T, H, Dv].
    ``gate`` [T, H]: head h's output is scaled by sigmoid(gate[:, h])."""
    T, H, _ = q.shape
    if out is None:
        out = _new_out(q, v_cache, o)
    if T == 0:
        return out
    if not q.is_cuda:
        return _attention_ref(q, k_cache, v_cache, meta, o, gate, out)
    many, one = _kernels(q, k_cache, v_cache, out, o, gate)
    # the leading sequences with one row stream their keys through the decode kernel
    nd = meta.num_reqs if meta.max_query_len <= 1 and T == meta.num_reqs else int(meta.num_decodes)
    if many is None and (one is None or nd < meta.num_reqs):          # no tensor-core kernel takes all rows
        return variant_attention_simple(q, k_cache, v_cache, meta, o, gate, out)
    if one == "wide" and nd:
        wide_attention_decode(q, k_cache, v_cache, meta, o, out, nd)
    elif one == "tile" and nd:
        variant_attention_decode(q, k_cache, v_cache, meta, o, gate, out, nd)
    else:
        nd = 0
    if nd < meta.num_reqs:
        variant_attention_prefill(q, k_cache, v_cache, meta, o, gate, out, nd, many == "wide")
    return out
