"""The kernels of the Pegopel decoder, each alone, against the plain definitions: bf16 and fp32, sizes that are
no multiple of anything, page, window, kept-token and tile borders."""
import numpy as np
import pytest
import torch

import pegopel_oracle as po
from gpu_utils import make_paged_case
from vllm_ascend_b200.attention import variant as va
from vllm_ascend_b200.attention.metadata import AttentionMetadata
from vllm_ascend_b200.ops import reference as ref
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, StreamMix, stream_mix

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype, scale=1.0):
    err = float((got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().clamp_min(1e-6))
    assert err < scale * (2e-5 if dtype == torch.float32 else 1.2e-2), err


def rnd(g, *shape, dtype, std=1.0):
    return (torch.randn(*shape, generator=g) * std).to(dtype)


# ---------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,S", [(1, 1), (30, 3), (33, 2), (256, 4), (1000, 16), (4096, 2), (4096, 4)])
def test_stream_mix(dtype, W, S):
    g = torch.Generator().manual_seed(W + S)
    T, V, eps = 7, 20, 1e-4
    y, wn = rnd(g, T, W, dtype=dtype), rnd(g, W, dtype=dtype)
    table, pos = rnd(g, V, W, dtype=dtype), rnd(g, 12, W, dtype=dtype)
    ids, at = torch.randint(0, V, (T,), generator=g), torch.randint(0, 12, (T,), generator=g)
    a, b = (StreamMix(torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g)) for _ in "ab")
    cu = lambda m: StreamMix(*(getattr(m, n).cuda() for n in ("read", "write", "mix")))        # noqa: E731
    spec = NormSpec("rms", wn.cuda())
    r = torch.empty(T, S, W, device="cuda")
    x = stream_mix(r, None, None, None, cu(a), spec, eps, dtype, embed=table.cuda(), ids=ids.cuda(), embed_scale=3.0,
                   pos_table=pos.cuda(), positions=at.cuda())
    e = table.double()[ids] * 3 + pos.double()[at]
    st = e[None].repeat(S, 1, 1)
    close(r, st.transpose(0, 1), torch.float32)

    def out(streams, m):
        u = streams.sum(0) if m is None else torch.einsum("s,stw->tw", m.read.double(), streams)
        return po.rms_norm(u, wn.double(), eps)
    if W > 1:
        close(x, out(st, a), dtype, 5)
    st = torch.randn(S, T, W, generator=g).double()
    for reader in (b, None):
        r = st.transpose(0, 1).float().contiguous().cuda()
        x = stream_mix(r, y.cuda(), PLAIN, cu(a), reader and cu(reader), spec, eps, dtype)
        new = po.mix_streams(st.float().double(), y.double(), {"mix": a.mix.double(), "out": a.write.double()})
        close(r, new.transpose(0, 1), torch.float32)
        if W > 1:
            close(x, out(new, reader), dtype, 5)
    keep = r.clone()
    stream_mix(r, None, None, None, None, spec, eps, dtype)
    assert torch.equal(r, keep)


# ---------------------------------------------------------------- q / k / v preparation
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,vd,taps,rot,shared", [
    (6, 2, 16, 24, 4, 0, False), (8, 2, 48, 48, 0, 32, True), (3, 1, 9, 5, 3, 0, False), (5, 5, 7, 7, 0, 4, True),
    (4, 1, 40, 8, 2, 40, False), (2, 2, 24, 16, 9, 8, False), (40, 8, 128, 128, 4, 0, False), (64, 8, 128, 128, 3, 64, True),
    (1, 1, 1, 3, 1, 0, False), (24, 4, 64, 40, 1, 0, False)])
def test_qkv_prep_over_portions(dtype, H, G, d, vd, taps, rot, shared):
    """Sequences in portions shorter and longer than the taps and a tile, in changing order; caches in both
    layouts, pages in a scattered order."""
    g = torch.Generator().manual_seed(H * d + taps)
    eps, bs, lens, slots = 1e-5, 8, [50, 1, 35, 18], [4, 0, 2, 5]
    nq, nk, nv = H * d, G * d, 0 if shared else G * vd
    C = nq + nk + nv
    x = [rnd(g, n, C + 8, dtype=dtype) for n in lens]
    conv = rnd(g, C, taps, dtype=dtype) if taps else None
    qn, kn = rnd(g, nq, dtype=dtype) + 1, rnd(g, nk, dtype=dtype) + 1
    cos_sin = ref.build_cos_sin_cache(rot, 64, 1e4, None).cuda() if rot else None
    spec = va.PrepSpec(H, G, d, vd, eps, qn.cuda(), kn.cuda(), (nq, nk), shared, None if conv is None else conv.cuda(),
                       rot, cos_sin)
    pages = torch.randperm(40, generator=g).tolist()
    table = [pages[7 * i:7 * i + 7] for i in range(4)]
    state = torch.full((6, taps - 1, C), 7.0, dtype=dtype, device="cuda") if taps > 1 else None
    if G % 2:
        kc, vc = (torch.zeros(40, bs, G, w, dtype=dtype, device="cuda") for w in (d, vd))
    else:
        kc, vc = (torch.zeros(40, G, bs, w, dtype=dtype, device="cuda").permute(0, 2, 1, 3) for w in (d, vd))
    q, at, k = [[] for _ in lens], [0] * 4, 0
    while any(a < n for a, n in zip(at, lens)):
        todo = [i for i in (range(4) if k % 2 else range(3, -1, -1)) if at[i] < lens[i]]
        take = [1] * len(todo) if k % 3 == 2 else [min([1, 2, 17, 3, 16][(k + i) % 5], lens[i] - at[i]) for i in todo]
        cu = np.concatenate([[0], np.cumsum(take)]).astype(np.int32)
        place = [np.arange(at[i], at[i] + n) for i, n in zip(todo, take)]
        slot = np.concatenate([np.asarray(table[i])[p // bs] * bs + p % bs for i, p in zip(todo, place)])
        dev = lambda a, t: torch.as_tensor(np.asarray(a), dtype=t).cuda()                     # noqa: E731
        meta = AttentionMetadata(
            num_reqs=len(todo), num_actual_tokens=int(cu[-1]), max_query_len=max(take), max_seq_len=64,
            query_start_loc=dev(cu, torch.int32), seq_lens=None, block_table=None, slot_mapping=dev(slot, torch.int64),
            positions=dev(np.concatenate(place), torch.int64), query_start_loc_cpu=cu, seq_lens_cpu=None)
        meta.state_slots = dev([slots[i] for i in todo], torch.int32)
        meta.has_initial_state = dev([at[i] > 0 for i in todo], torch.int32)
        rows = torch.cat([x[i][at[i]:at[i] + n] for i, n in zip(todo, take)]).cuda()
        got = va.qkv_prep(spec, rows, meta, kc, vc, state)
        for j, i in enumerate(todo):
            q[i].append(got[cu[j]:cu[j + 1]].cpu())
            at[i] += take[j]
        k += 1
    for i, n in enumerate(lens):
        u = x[i][:, :C].double()
        if taps:
            u = po.short_conv(u, conv.double())
        raw = u[:, nq:nq + nk]
        wq, wk = po.rms_norm(u[:, :nq], qn.double(), eps).view(n, H, d), po.rms_norm(raw, kn.double(), eps).view(n, G, d)
        if rot:
            wq, wk = (torch.stack([po.rotate(t[p], p, rot, 1e4, None) for p in range(n)]) for t in (wq, wk))
        want_v = (raw if shared else u[:, nq + nk:]).reshape(n, G, vd)
        close(torch.cat(q[i]), wq, dtype)
        p = torch.arange(n)
        pg = torch.tensor(table[i])[p // bs]
        close(kc[pg.cuda(), (p % bs).cuda()], wk, dtype)
        close(vc[pg.cuda(), (p % bs).cuda()], want_v, dtype)


# ---------------------------------------------------------------- attention
def run_case(dtype, H, G, d, vd, bs, q_lens, ctx, window, keep, cap, buckets, largest, sink, gate, kernel, splits=0,
             layout="HND"):
    g = torch.Generator().manual_seed(H * d + window)
    q, k, v, meta = make_paged_case(q_lens, ctx, H, G, d, bs, dtype=dtype, layout=layout, tok_per_tile=1)[:4]
    v = torch.zeros(*k.shape[:3], vd) if layout == "NHD" else torch.zeros(k.shape[0], G, bs, vd).permute(0, 2, 1, 3)
    v.copy_(torch.randn(k.shape[0], bs, G, vd, generator=g))
    v = v.to(dtype).cuda()
    q, k = (q * 2).to(dtype), k.to(dtype)
    meta.num_decodes = int(np.argmax(np.append(np.diff(meta.query_start_loc_cpu), 9) > 1))
    pos = [np.arange(c, c + n) for c, n in zip(ctx, q_lens)]
    meta.positions = torch.from_numpy(np.concatenate(pos)).cuda()
    rel = torch.randn(buckets, H, generator=g) * 2 if buckets else None
    sk = {None: None, "zero": torch.zeros(H), "learned": torch.randn(H, generator=g) + 1}[sink]
    scale = d ** -0.5 * 2
    o = va.AttnOptions(scale, window, keep, cap, None if rel is None else va.distance_table(rel, largest, 4096).cuda(),
                       None if sk is None else sk.cuda())
    gt = rnd(g, q.shape[0], H + 3, dtype=dtype) if gate else None
    gd = None if gt is None else gt.cuda()[:, :H]
    if kernel == "simple":
        got = va.variant_attention_simple(q, k, v, meta, o, gd)
    elif kernel == "prefill":
        got = va.variant_attention_prefill(q, k, v, meta, o, gd)
    elif kernel == "decode":
        got = va.variant_attention_decode(q, k, v, meta, o, gd, num_splits=splits)
    else:
        got = va.variant_attention(q, k, v, meta, o, gd)
    cu = meta.query_start_loc_cpu
    for b, (n, c) in enumerate(zip(q_lens, ctx)):
        kb, vb = (ref.gather_kv(t, meta.block_table[b], c + n).double().cpu() for t in (k, v))
        qb = torch.zeros(c + n, H, d, dtype=torch.float64)
        qb[c:] = q[cu[b]:cu[b + 1]].double().cpu()
        want = po.attend(qb, kb, vb, scale, window or None, keep, cap or None, None if rel is None else rel.double(),
                         largest, None if sk is None else sk.double(), rows=range(c, c + n))[c:]
        if gt is not None:
            want = want * torch.sigmoid(gt[cu[b]:cu[b + 1], :H].double())[:, :, None]
        close(got[cu[b]:cu[b + 1]], want, dtype)


OPTIONS = {          # window, kept, cap, buckets, largest, sink, gate
    "plain": (0, 0, 0.0, 0, 0, None, False),
    "biased": (40, 0, 0.0, 16, 60, "learned", False),
    "gated": (24, 9, 3.0, 0, 0, "zero", True),
    "far": (200, 150, 0.0, 32, 400, "learned", True),
    "cap": (0, 0, 40.0, 0, 0, "zero", False),
    "all": (130, 5, 2.0, 8, 20, "learned", True),
    "one": (1, 1, 2.0, 2, 4, "zero", True),
}
MIXED = ([1, 1, 37, 2, 130, 5], [0, 301, 100, 63, 0, 255])
SINGLE = ([1] * 6, [0, 23, 39, 127, 128, 411])


@pytest.mark.parametrize("opts", sorted(OPTIONS))
@pytest.mark.parametrize("dtype,H,G,d,vd", [(torch.float32, 4, 2, 20, 33), (torch.bfloat16, 3, 1, 9, 70),
                                            (torch.float32, 2, 2, 128, 64), (torch.bfloat16, 2, 1, 192, 200)])
def test_cuda_core_attention(dtype, H, G, d, vd, opts):
    run_case(dtype, H, G, d, vd, 16, *MIXED, *OPTIONS[opts], "simple")


@pytest.mark.parametrize("opts", sorted(OPTIONS))
@pytest.mark.parametrize("H,G,d,vd,bs,layout", [(8, 2, 128, 128, 64, "HND"), (8, 8, 64, 64, 128, "NHD"), (6, 2, 40, 24, 16, "HND"),
                                                (20, 1, 24, 128, 64, "NHD"), (10, 2, 72, 8, 128, "HND"),
                                                (128, 1, 16, 56, 32, "NHD")])
def test_prefill_attention(H, G, d, vd, bs, layout, opts):
    run_case(torch.bfloat16, H, G, d, vd, bs, *MIXED, *OPTIONS[opts], "prefill", layout=layout)


@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("opts", sorted(OPTIONS))
@pytest.mark.parametrize("H,G,d,vd,bs,layout", [(8, 2, 128, 128, 64, "HND"), (8, 8, 64, 64, 128, "NHD"), (6, 2, 40, 24, 16, "HND"),
                                                (16, 1, 128, 48, 128, "NHD"), (10, 2, 72, 8, 256, "HND")])
def test_decode_attention(H, G, d, vd, bs, layout, opts, splits):
    run_case(torch.bfloat16, H, G, d, vd, bs, *SINGLE, *OPTIONS[opts], "decode", splits, layout)


@pytest.mark.parametrize("H,G,d,vd", [(8, 2, 64, 64), (24, 1, 32, 16), (6, 3, 24, 40)])
def test_mixed_batch_takes_both_kernels(H, G, d, vd):
    run_case(torch.bfloat16, H, G, d, vd, 64, *MIXED, *OPTIONS["all"], "any")


@pytest.mark.parametrize("kernel", ["prefill", "decode", "simple"])
def test_edges_of_window_and_kept_tokens(kernel):
    """One key stands out: just inside and just outside the window's edge and the kept tokens, at page and tile
    borders, it is seen or not."""
    H, d, bs, window, keep = 2, 32, 16, 40, 20
    dtype = torch.float32 if kernel == "simple" else torch.bfloat16
    for pos in (19, 59, 60, 61, 100, 127, 128, 170, 299):
        q, k, v, meta = make_paged_case([1], [pos], H, 1, d, bs, dtype=dtype, tok_per_tile=1)[:4]
        meta.positions = torch.tensor([pos]).cuda()
        meta.num_decodes = 1
        o = va.AttnOptions(1.0, window, keep)
        fn = {"prefill": va.variant_attention_prefill, "decode": va.variant_attention_decode,
              "simple": va.variant_attention_simple}[kernel]
        for j in {0, keep - 1, keep, keep + 1, pos - window - 1, pos - window, pos - window + 1, pos - 1, pos}:
            if not 0 <= j <= pos:
                continue
            kk, vv = torch.zeros_like(k), torch.zeros_like(v)
            page = int(meta.block_table[0, j // bs])
            kk[page, j % bs] = q[0, 0] * 16 / float((q[0, 0].float() ** 2).sum())
            vv[page, j % bs] = 1.0
            got = float(fn(q, kk, vv, meta, o)[0, 0, 0])
            assert (got > 0.9) if po.visible(pos, j, window, keep) else got == 0.0, (pos, j, got)
