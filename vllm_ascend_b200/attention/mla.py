"""Latent attention (MLA): cache write and absorbed-weight attention, full or over a sliding window, with
an optional attention sink per head.

Cache layout contract: two paged tensors per layer, latent
``[num_blocks, block_size, 1, kv_lora_rank]`` and rope
``[num_blocks, block_size, 1, qk_rope_head_dim]``
(vllm_ascend/worker/model_runner_v1.py:3994-4069).  Attention is MQA over the
(latent ‖ rope) key, 512 + 64 wide in DeepSeek's models, with the latent as value
(vllm_ascend/attention/mla_v1.py:1373-1577).
"""
from __future__ import annotations

from typing import Optional

import torch

from ctypes import c_float, c_int, c_long, c_void_p

from .. import _native
from ..ops import reference as ref

_P, _I, _L, _F = c_void_p, c_int, c_long, c_float
_native.register_signature("b200_mla_attention", [_P, _L, _L, _P, _L, _L, _L, _I, _I, _I, _P, _P, _L, _I, _P, _P, _P, _P,
                                                  _I, _I, _P, _I, _P, _I, _F, _I, _P, _L, _L, _P, _P, _P, _P])
_native.register_signature("b200_latent_attention", [_P, _L, _L, _P, _L, _L, _L, _I, _I, _I, _P, _P, _L, _I, _P, _P, _P,
                                                     _I, _P, _F, _I, _P, _L, _L, _I, _P, _P])
_scratch: dict = {}
_MAX_SPLITS = 32


def _split_scratch(dev, numel: int) -> torch.Tensor:
    buf = _scratch.get(dev.index)
    if buf is None or buf.numel() < numel:
        buf = torch.empty(max(numel, 1 << 20), dtype=torch.float32, device=dev)
        _scratch[dev.index] = buf
    return buf


def _num_splits(dev, ctas: int, max_keys: int) -> int:
    """Splits of the key range that give about two CTAs per SM, at most one per 128-key tile."""
    from ..batch_invariant import is_batch_invariant
    if is_batch_invariant():
        return 1
    sms = torch.cuda.get_device_properties(dev).multi_processor_count
    tiles = max(1, (max_keys + 127) // 128)
    return max(1, min(tiles, (2 * sms + ctas - 1) // max(ctas, 1), _MAX_SPLITS))


def _tc_sizes_ok(q_lat: torch.Tensor, q_pe: torch.Tensor, lat_cache: torch.Tensor) -> bool:
    """True when the tcgen05 kernel takes these tensors (TMA: 16-byte strides and bases)."""
    H, dc, dr = q_lat.shape[1], q_lat.shape[2], q_pe.shape[2]
    strides = (q_lat.stride(0), q_lat.stride(1), q_pe.stride(0), q_pe.stride(1))
    return (q_lat.dtype == torch.bfloat16 and lat_cache.dtype == torch.bfloat16 and 8 <= dc <= 512 and 8 <= dr <= 64
            and dc % 8 == 0 and dr % 8 == 0 and q_lat.stride(2) == 1 and q_pe.stride(2) == 1 and H >= 1
            and all(x % 8 == 0 for x in strides) and q_lat.data_ptr() % 16 == 0 and q_pe.data_ptr() % 16 == 0
            and lat_cache.shape[1] in (8, 16, 32, 64, 128, 256, 512))


def latent_attention_tc(q_lat: torch.Tensor, q_pe: torch.Tensor, lat_cache: torch.Tensor, pe_cache: torch.Tensor,
                        block_table: torch.Tensor, scale: float, row_seq=None, row_kv_len=None, cu=None, seq_lens=None,
                        uniform: bool = False, window: int = 0, sink: Optional[torch.Tensor] = None,
                        num_splits: int = 0, max_kv_len: int = 0, out: Optional[torch.Tensor] = None,
                        lse_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """tcgen05 latent attention over query rows: q_lat [R, H, dc] (absorbed), q_pe [R, H, dr] -> [R, H, dc].

    Rows are described one by one (``row_seq`` / ``row_kv_len``: row r attends to the first ``row_kv_len[r]``
    tokens of block-table row ``row_seq[r]``) or as a batch (``cu`` / ``seq_lens``: sequence b owns rows
    cu[b]..cu[b+1), its last row sees ``seq_lens[b]`` tokens; ``uniform``: one row each).  ``window``: a row
    sees only the last ``window`` of its tokens.  ``out`` may be any [R, H, dc] view whose last dimension is
    dense.  ``lse_out`` (fp32 [R, H]) receives the log-sum-exp over the keys seen (-inf for a row without
    keys), for merging the results of context-parallel ranks."""
    R, H, dc = q_lat.shape
    dev = q_lat.device
    if out is None:
        out = torch.empty((R, H, dc), dtype=torch.bfloat16, device=dev)
    if num_splits <= 0:
        pack = cu is not None and not uniform
        nq = 32 if (H > 16 or pack) else 16
        hb = (H + nq - 1) // nq
        tok = nq // ((H + hb - 1) // hb) if pack else 1
        ctas = hb * ((R + tok - 1) // tok)
        keys = max_kv_len or 1024
        if window > 0:
            keys = min(keys, window + tok + 126)        # a window rarely starts on a tile border
        num_splits = _num_splits(dev, ctas, keys)
    if lse_out is not None:
        num_splits = max(2, num_splits)          # the split merge produces the log-sum-exp
    scratch = _split_scratch(dev, R * H * num_splits * (dc + 1)) if num_splits > 1 else None
    B = 0 if cu is None else cu.numel() - 1
    rc = _native.lib().b200_mla_attention(
        q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1), q_pe.data_ptr(), q_pe.stride(0), q_pe.stride(1), R, H, dc,
        q_pe.shape[2], lat_cache.data_ptr(), pe_cache.data_ptr(), lat_cache.shape[0], lat_cache.shape[1],
        _native.ptr(row_seq), _native.ptr(row_kv_len), _native.ptr(cu), _native.ptr(seq_lens), B, int(uniform),
        block_table.data_ptr(), block_table.stride(0), _native.ptr(sink), int(window), scale, num_splits,
        out.data_ptr(), out.stride(0), out.stride(1), _native.ptr(scratch), _native.ptr(lse_out),
        _native.status_word(dev).data_ptr(), _native.stream_ptr())
    _native.check(rc, "mla_attention")
    _native.count_launch(2 if num_splits > 1 else 1)
    return out


def mla_decode_native(q_cat: torch.Tensor, lat_cache: torch.Tensor, pe_cache: torch.Tensor,
                      row_seq: torch.Tensor, row_kv_len: torch.Tensor, block_table: torch.Tensor,
                      scale: float, num_splits: int = 0, max_kv_len: int = 0,
                      lse_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``latent_attention_tc`` over listed rows whose two query parts are concatenated:
    q_cat [R, H, dc + dr] = absorbed q_nope ‖ q_pe.  Returns o_lat [R, H, dc]."""
    dc = lat_cache.shape[-1]
    assert q_cat.dtype == torch.bfloat16 and q_cat.stride(2) == 1
    return latent_attention_tc(q_cat[..., :dc], q_cat[..., dc:], lat_cache, pe_cache, block_table, scale,
                               row_seq=row_seq, row_kv_len=row_kv_len, num_splits=num_splits, max_kv_len=max_kv_len,
                               lse_out=lse_out)


def latent_attention_simple(q_lat: torch.Tensor, q_pe: torch.Tensor, lat_cache: torch.Tensor, pe_cache: torch.Tensor,
                            row_seq: torch.Tensor, row_kv_len: torch.Tensor, block_table: torch.Tensor, scale: float,
                            window: int = 0, sink: Optional[torch.Tensor] = None,
                            out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """CUDA-core kernel for the sizes and types the tcgen05 kernel does not take (fp32, odd widths)."""
    R, H, dc = q_lat.shape
    if out is None:
        out = torch.empty((R, H, dc), dtype=q_lat.dtype, device=q_lat.device)
    if not (q_lat.dtype == q_pe.dtype == lat_cache.dtype == pe_cache.dtype == out.dtype) \
            or q_lat.dtype not in (torch.bfloat16, torch.float32):
        raise TypeError("latent attention takes bf16 or fp32 queries with a cache of the same type")
    rc = _native.lib().b200_latent_attention(
        q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1), q_pe.data_ptr(), q_pe.stride(0), q_pe.stride(1), R, H, dc,
        q_pe.shape[2], lat_cache.data_ptr(), pe_cache.data_ptr(), lat_cache.shape[0], lat_cache.shape[1],
        row_seq.data_ptr(), row_kv_len.data_ptr(), block_table.data_ptr(), block_table.stride(0), _native.ptr(sink),
        scale, int(window), out.data_ptr(), out.stride(0), out.stride(1), int(q_lat.dtype == torch.float32),
        _native.status_word(q_lat.device).data_ptr(), _native.stream_ptr())
    _native.check(rc, "latent_attention")
    _native.count_launch()
    return out


def _batch_rows(meta, T: int, device) -> tuple[torch.Tensor, torch.Tensor]:
    """(block-table row, visible key count) of every query row of a step, computed once per step."""
    key = (T, torch.cuda.is_current_stream_capturing())
    cached = getattr(meta, "_latent_rows", None)
    if cached is not None and cached[0] == key:
        return cached[1], cached[2]
    B = meta.num_reqs
    if meta.max_query_len == 1 and T == B:
        row_seq = torch.arange(T, dtype=torch.int32, device=device)
    else:
        q_lens = (meta.query_start_loc[1:B + 1] - meta.query_start_loc[:B]).long()
        row_seq = torch.repeat_interleave(torch.arange(B, device=device), q_lens, output_size=T).to(torch.int32)
    row_kv = (meta.positions[:T] + 1).to(torch.int32)
    meta._latent_rows = (key, row_seq, row_kv)
    return row_seq, row_kv


def reserve_mla_scratch(device, rows: int, heads: int, width: int = 512, max_keys: int = 0) -> None:
    """Allocate the split-KV scratch of decode batches of up to ``rows`` rows up front (before graph
    capture, whose batches all use it)."""
    hb = (heads + 31) // 32 if heads > 16 else 1
    worst = max(r * _num_splits(device, r * hb, max_keys or _MAX_SPLITS * 128) for r in range(1, rows + 1))
    _split_scratch(device, worst * heads * (width + 1))


def write_latent_cache(latent: torch.Tensor, k_pe: torch.Tensor, lat_cache: torch.Tensor,
                       pe_cache: torch.Tensor, slot_mapping: torch.Tensor) -> None:
    """Scatter the step's latents / rope keys into their cache slots; slot -1 = not stored.
    Written without data-dependent shapes so it can be captured into a CUDA graph: skipped
    tokens rewrite slot 0 with the value it already holds."""
    valid = (slot_mapping >= 0).unsqueeze(-1)
    idx = slot_mapping.clamp(min=0)
    lat_flat = lat_cache.view(-1, lat_cache.shape[-1])
    pe_flat = pe_cache.view(-1, pe_cache.shape[-1])
    lat_flat.index_copy_(0, idx, torch.where(valid, latent.to(lat_cache.dtype), lat_flat[idx]))
    pe_flat.index_copy_(0, idx, torch.where(valid, k_pe.to(pe_cache.dtype), pe_flat[idx]))


def mla_paged_attention(q_lat: torch.Tensor, q_pe: torch.Tensor, lat_cache: torch.Tensor,
                        pe_cache: torch.Tensor, meta, scale: float, window: int = 0,
                        sink: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q_lat [T,H,dc], q_pe [T,H,dr] -> o_lat [T,H,dc] (softmax over latent‖rope keys).  ``window`` > 0: a token
    sees itself and the window - 1 tokens before it; ``sink`` [H]: exp(sink) joins the softmax denominator."""
    T, H, dc = q_lat.shape
    from .. import envs
    if q_lat.is_cuda and envs.VLLM_B200_MLA_ATTN == "tcgen05" and T > 0:
        # a captured graph must carry a split count that suits any later sequence length
        max_kv = meta.block_table.shape[1] * lat_cache.shape[1] if torch.cuda.is_current_stream_capturing() \
            else meta.max_seq_len
        uniform = meta.max_query_len == 1 and T == meta.num_reqs
        if _tc_sizes_ok(q_lat, q_pe, lat_cache) and T + meta.num_reqs <= 65535:
            return latent_attention_tc(q_lat, q_pe, lat_cache, pe_cache, meta.block_table, scale,
                                       cu=meta.query_start_loc[:meta.num_reqs + 1], seq_lens=meta.seq_lens,
                                       uniform=uniform, window=window, sink=sink, max_kv_len=max_kv, out=out)
        row_seq, row_kv = _batch_rows(meta, T, q_lat.device)
        return latent_attention_simple(q_lat, q_pe, lat_cache, pe_cache, row_seq, row_kv, meta.block_table, scale,
                                       window, sink, out)
    if out is None:
        out = torch.empty(T, H, dc, dtype=q_lat.dtype, device=q_lat.device)
    qsl, sls = meta.query_start_loc_cpu, meta.seq_lens_cpu
    for b in range(meta.num_reqs):
        qs, qe = int(qsl[b]), int(qsl[b + 1])
        ql = qe - qs
        if ql <= 0:
            continue
        sl = int(sls[b])
        ctx = sl - ql
        lat = ref.gather_kv(lat_cache, meta.block_table[b], sl)[:, 0].float()   # [sl, dc]
        pe = ref.gather_kv(pe_cache, meta.block_table[b], sl)[:, 0].float()     # [sl, dr]
        s = (torch.einsum("qhc,kc->hqk", q_lat[qs:qe].float(), lat) +
             torch.einsum("qhr,kr->hqk", q_pe[qs:qe].float(), pe)) * scale
        kpos = torch.arange(sl, device=s.device)
        qpos = ctx + torch.arange(ql, device=s.device)
        seen = kpos[None, :] <= qpos[:, None]
        if window > 0:
            seen &= kpos[None, :] > qpos[:, None] - window
        s = s.masked_fill(~seen[None], float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.float().view(H, 1, 1).expand(H, ql, 1)], dim=-1)
        p = torch.softmax(s, dim=-1)[..., :sl]
        out[qs:qe] = torch.einsum("hqk,kc->qhc", p, lat).to(out.dtype)
    return out


class B200MLABackend:
    """Descriptor of the MLA backend (vllm_ascend/attention/mla_v1.py: cache of a 512-wide
    normalised latent plus a 64-wide RoPE key per token, MQA with absorbed up-projections)."""

    @staticmethod
    def get_name() -> str:
        return "B200_MLA"

    @staticmethod
    def get_kv_cache_shape(num_blocks: int, block_size: int, num_kv_heads: int, head_size: int) -> tuple:
        return (num_blocks, block_size, 1, head_size)

    @staticmethod
    def get_supported_block_size() -> list[int]:
        return [128]

    @staticmethod
    def get_impl_cls():
        from ..models.transformer import MLAAttention
        return MLAAttention
