"""The kernels the Dubizen decoder adds or extends, each alone, against the plain definitions: bf16 and fp32, sizes
that are multiples of a vector and sizes that are not, page, window and tile borders."""
import numpy as np
import pytest
import torch

import dubizen_oracle as do
from gpu_utils import make_paged_case
from pegopel_oracle import distance_bucket
from test_gpu_pegopel_ops import MIXED, SINGLE, close, rnd, run_case
from test_gpu_vofelix_ops import attend, paged, slot
from vllm_ascend_b200 import _native, ops
from vllm_ascend_b200.attention import mla, variant as va
from vllm_ascend_b200.attention.metadata import AttentionMetadata
from vllm_ascend_b200.ops import fused_moe, moe_native, reference as ref
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, stream_norm
from vofelix_oracle import rotate

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(autouse=True)
def no_status():
    yield
    torch.cuda.synchronize()
    _native.check_status(torch.device("cuda"))


# ---------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [2, 33, 88, 1000, 4096])
def test_output_norm_joins_the_stream_with_a_multiplier(dtype, W):
    g = torch.Generator().manual_seed(W)
    r, y, w = torch.randn(9, W, generator=g), rnd(g, 9, W, dtype=dtype) + 2, rnd(g, W, dtype=dtype)
    want = r.double() + 0.3 * do.output_norm(y.double(), w.double(), 1e-4)
    rc = r.cuda()
    x = stream_norm(rc, y.cuda(), NormSpec("layer", w.cuda()), PLAIN, 1e-4, dtype, post_scale=0.3)
    close(rc, want, torch.float32, 4)
    assert torch.equal(x, rc.to(dtype))
    x = stream_norm(rc, y.cuda(), NormSpec("layer", w.cuda()), NormSpec("layer", w.cuda()), 1e-4, dtype, post_scale=-0.3)
    close(rc, r, torch.float32, 4)
    if W > 2:
        close(x, do.output_norm(r.double(), w.double(), 1e-4), dtype, 4)


# ---------------------------------------------------------------- latent attention around its projections
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rq,dc,dr", [(27, 21, 6), (96, 72, 16), (1, 1, 2), (1536, 512, 64), (24, 136, 8), (40, 0, 16)])
def test_latent_prep(dtype, rq, dc, dr):
    g = torch.Generator().manual_seed(rq + dc)
    T, base, pad = 13, 5000.0, 5
    table = ref.build_cos_sin_cache(dr, 400, base, None, "cuda")
    down = rnd(g, T, rq + (dc + dr if dc else 0) + pad, dtype=dtype)
    qn, kn = rnd(g, rq, dtype=dtype), rnd(g, dc, dtype=dtype) if dc else None
    pos, slots = torch.randint(0, 400, (T,), generator=g), torch.randperm(40, generator=g)[:T]
    slots[3] = -1
    lat, pe = (torch.zeros(5, 8, 1, n or 4, dtype=dtype).cuda() for n in (dc, dr))
    cq = ops.latent_prep(down.cuda(), qn.cuda(), kn if kn is None else kn.cuda(), 1e-5, pos.cuda(), table, slots.cuda(), lat, pe)
    close(cq, do.rms_norm(down[:, :rq].double(), qn.double(), 1e-5), dtype)
    if not dc:
        assert not lat.any() and not pe.any()
        return
    for t in range(T):
        if slots[t] < 0:
            continue
        close(lat.view(-1, dc)[slots[t]], do.rms_norm(down[t, rq:rq + dc].double(), kn.double(), 1e-5), dtype)
        close(pe.view(-1, dr)[slots[t]], rotate(down[t, rq + dc:rq + dc + dr].double(), int(pos[t]), dr, base, None), dtype)
    assert int((lat.view(-1, dc).abs().sum(-1) > 0).sum()) == T - 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,dn,dr", [(5, 3, 11, 6), (300, 8, 24, 16), (1, 1, 1, 2), (2, 40, 128, 64), (700, 2, 12, 4)])
def test_latent_query(dtype, T, H, dn, dr):
    g = torch.Generator().manual_seed(T)
    table = ref.build_cos_sin_cache(dr, 900, 1e4, None, "cuda")
    q, pos = rnd(g, T, H, dn + dr, dtype=dtype), torch.randint(0, 900, (T,), generator=g)
    qc = q.cuda()
    nope = ops.latent_query(qc, pos.cuda(), table)
    assert torch.equal(nope.cpu(), q[..., :dn]) and torch.equal(qc[..., :dn].cpu(), q[..., :dn])
    for t in sorted({0, T // 2, T - 1}):
        close(qc[t, :, dn:], rotate(q[t, :, dn:].double(), int(pos[t]), dr, 1e4, None), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [(7, 104, 24, 64, [300, 64, 65, 1], [300, 64, 1, 1]), (3, 20, 6, 16, [40, 9, 200], [40, 1, 2]),
                                  (16, 512, 64, 128, [700, 129, 258], [1, 1, 1]), (5, 72, 16, 64, [500, 128], [2, 128])])
def test_latent_attention_over_everything(dtype, case):
    H, dc, dr, bs, lens, q_lens = case
    lat_c, pe_c, table, meta = paged(lens, q_lens, bs, dc, dr, dtype, dc)
    g = torch.Generator().manual_seed(dc)
    T, scale = sum(q_lens), 0.6 * (dc + dr) ** -0.5
    q_lat, q_pe = rnd(g, T, H, dc, dtype=dtype), rnd(g, T, H, dr, dtype=dtype)
    got = mla.mla_paged_attention(q_lat.cuda(), q_pe.cuda(), lat_c.cuda(), pe_c.cuda(), meta, scale).cpu()
    for b, (n, m) in enumerate(zip(lens, q_lens)):
        pages = table[b, :(n + bs - 1) // bs].long()
        lat, pe = lat_c[pages].reshape(-1, dc)[:n].double(), pe_c[pages].reshape(-1, dr)[:n].double()
        r0 = int(meta.query_start_loc_cpu[b])
        want = torch.stack([attend(q_lat[r0 + i].double(), q_pe[r0 + i].double(), lat, pe, 0, n - m + i, scale, None)
                            for i in range(m)])
        close(got[r0:r0 + m], want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [True, False])
def test_one_far_latent_that_stands_out(dtype, decode):
    """A key whose score towers over all others is found wherever it lies: first, at page and tile borders, last;
    and not when it lies behind the query."""
    H, dc, dr, bs, n = 6, 40, 8, 64, 1000
    q_lens = [1, 3] if decode else [7, 40]
    lat_c, pe_c, table, meta = paged([n, n], q_lens, bs, dc, dr, dtype, 1)
    q_lat, q_pe = torch.zeros(sum(q_lens), H, dc, dtype=dtype), torch.zeros(sum(q_lens), H, dr, dtype=dtype)
    q_pe[..., 0] = 1.0
    m = q_lens[1]
    for j in (0, 1, 63, 64, 127, 128, 500, 959, 960, n - m - 1, n - m, n - 2, n - 1):
        lc, pc = lat_c * 0.1, pe_c * 0.1
        blk, off = slot(table, bs, 1, j)
        pc[blk, off, 0, 0] = 40.0
        lc[blk, off, 0] = 5.0
        out = mla.mla_paged_attention(q_lat.cuda(), q_pe.cuda(), lc.cuda(), pc.cuda(), meta, 1.0).float().cpu()[q_lens[0]:]
        for i in range(m):
            seen = j <= n - m + i
            assert bool(((out[i] - 5.0).abs() < 0.05).all()) if seen else bool((out[i].abs() < 0.6).all()), (j, i)


# ---------------------------------------------------------------- paged attention with a norm per head
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,vd,rot,shared", [(6, 2, 9, 14, 0, False), (6, 2, 40, 24, 0, False), (4, 4, 64, 128, 32, False),
                                                 (1, 1, 1, 1, 0, False), (3, 1, 7, 7, 4, True), (16, 2, 128, 96, 0, False),
                                                 (2, 2, 256, 520, 256, False), (8, 2, 48, 48, 48, True), (2, 1, 300, 33, 10, False)])
def test_prep_with_a_norm_per_head(dtype, H, G, d, vd, rot, shared):
    g = torch.Generator().manual_seed(H * d)
    T, bs, eps = 21, 8, 1e-5
    nq, nk, nv = H * d, G * d, 0 if shared else G * vd
    x = rnd(g, T, nq + nk + nv + 8, dtype=dtype)
    qn, kn = rnd(g, d, dtype=dtype) + 1, rnd(g, d, dtype=dtype) + 1
    cs = ref.build_cos_sin_cache(rot, 64, 1e4, None).cuda() if rot else None
    spec = va.PrepSpec(H, G, d, vd, eps, qn.cuda(), kn.cuda(), (nq, nk), shared, rot_dims=rot, cos_sin=cs, head_norm=True)
    if G % 2:
        kc, vc = (torch.zeros(6, bs, G, w, dtype=dtype, device="cuda") for w in (d, vd))
    else:
        kc, vc = (torch.zeros(6, G, bs, w, dtype=dtype, device="cuda").permute(0, 2, 1, 3) for w in (d, vd))
    slots, pos = torch.randperm(48, generator=g)[:T], torch.randint(0, 64, (T,), generator=g)
    slots[5] = -1
    cu = np.array([0, T], dtype=np.int32)
    meta = AttentionMetadata(num_reqs=1, num_actual_tokens=T, max_query_len=T, max_seq_len=64,
                             query_start_loc=torch.from_numpy(cu).cuda(), seq_lens=None, block_table=None,
                             slot_mapping=slots.cuda(), positions=pos.cuda(), query_start_loc_cpu=cu, seq_lens_cpu=None)
    q = va.qkv_prep(spec, x.cuda(), meta, kc, vc)
    u = x.double()
    raw = u[:, nq:nq + nk].view(T, G, d)
    wq, wk = do.rms_norm(u[:, :nq].view(T, H, d), qn.double(), eps), do.rms_norm(raw, kn.double(), eps)
    if rot:
        wq, wk = (torch.stack([rotate(t[i], int(pos[i]), rot, 1e4, None) for i in range(T)]) for t in (wq, wk))
    want_v = raw if shared else u[:, nq + nk:nq + nk + nv].view(T, G, vd)
    close(q, wq, dtype)
    on = slots >= 0
    at = (slots[on].cuda() // bs, slots[on].cuda() % bs)
    close(kc[at], wk[on], dtype)
    close(vc[at], want_v[on], dtype)
    assert int((kc.abs().sum((2, 3)) > 0).sum()) == T - 1


BIASED = {"window": (40, 0, 0.0, 16, 60, None, False), "one": (1, 0, 0.0, 2, 4, None, False),
          "wide": (200, 0, 0.0, 32, 400, None, False), "everything": (0, 0, 0.0, 8, 20, None, False)}


@pytest.mark.parametrize("opts", sorted(BIASED))
@pytest.mark.parametrize("H,G,d,vd,bs,kernel,splits", [
    (6, 2, 40, 24, 16, "prefill", 0), (6, 2, 40, 24, 16, "decode", 1), (8, 2, 128, 96, 64, "decode", 3),
    (24, 1, 16, 40, 64, "any", 0), (6, 2, 40, 24, 64, "any", 0), (4, 2, 20, 33, 16, "simple", 0)])
def test_distance_bias_without_a_sink(H, G, d, vd, bs, kernel, splits, opts):
    dtype = torch.float32 if kernel == "simple" else torch.bfloat16
    run_case(dtype, H, G, d, vd, bs, *(SINGLE if kernel == "decode" else MIXED), *BIASED[opts], kernel, splits)


@pytest.mark.parametrize("kernel", ["prefill", "decode", "simple"])
def test_distance_buckets_and_window_edge(kernel):
    """All keys alike: the weights are those of the biases of the distances inside the window, and of no other."""
    H, d, bs, window, largest, rows = 3, 16, 16, 50, 33, 12
    dtype = torch.float32 if kernel == "simple" else torch.bfloat16
    rel = torch.randn(rows, H, generator=torch.Generator().manual_seed(2)) * 2
    fn = {"prefill": va.variant_attention_prefill, "decode": va.variant_attention_decode,
          "simple": va.variant_attention_simple}[kernel]
    for pos in (0, 3, 49, 50, 51, 127, 128, 200):
        q, k, v, meta = make_paged_case([1], [pos], H, 1, d, bs, dtype=dtype, tok_per_tile=1)[:4]
        meta.positions, meta.num_decodes = torch.tensor([pos]).cuda(), 1
        k.zero_()
        o = va.AttnOptions(1.0, window, bias=va.distance_table(rel, largest, window).cuda())
        got = fn(q, k, v, meta, o)
        seen = torch.arange(max(0, pos - window + 1), pos + 1)
        b = torch.stack([rel[distance_bucket(pos - int(j), rows, largest)] for j in seen]).double()
        vals = ref.gather_kv(v, meta.block_table[0], pos + 1).double().cpu()[seen, 0]
        close(got[0], torch.softmax(b, 0).T @ vals, dtype)


# ---------------------------------------------------------------- experts
@pytest.mark.parametrize("E,k,groups", [(16, 5, (4, 2)), (12, 3, (4, 2)), (9, 1, (9, 1)), (8, 8, (1, 1)), (300, 20, (30, 4))])
def test_router_with_best_group_and_negative_scores(E, k, groups):
    g = torch.Generator().manual_seed(E)
    z, corr = torch.randn(50, E, generator=g) * 2, torch.randn(E, generator=g) * 0.3 - 1.0
    w, ids = fused_moe.gating_topk(z.cuda(), k, "softmax", True, *groups, corr.cuda(), 1.7, "max")
    c = {"experts": E, "top": k, "scale": 1.7, "groups": dict(zip(("count", "keep"), groups))}
    for t in range(50):
        want = do.route(z[t].double(), corr, c)
        got = {int(e): float(v) for e, v in zip(ids[t].cpu(), w[t].cpu())}
        assert got.keys() == want.keys() and all(abs(got[e] - want[e]) < 1e-5 for e in want)


def test_router_logits_keep_32_bits():
    g = torch.Generator().manual_seed(1)
    x, w = rnd(g, 70, 1000, dtype=torch.bfloat16), rnd(g, 13, 1000, dtype=torch.bfloat16)
    got = ops.linear_fp32(x.cuda(), w.cuda())
    assert got.dtype == torch.float32
    close(got, x.double() @ w.double().T, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,H,I,shared,gate", [
    (7, 9, 2, 38, 13, True, True), (64, 24, 5, 128, 72, True, True), (300, 4, 4, 72, 24, False, False), (1, 1, 1, 24, 1, True, True),
    (500, 16, 4, 256, 136, True, False), (33, 8, 1, 40, 128, True, True), (2, 64, 8, 512, 384, True, True)])
def test_experts_and_shared_expert(dtype, T, E, k, H, I, shared, gate):
    g = torch.Generator().manual_seed(T + E)
    x, w13, w2 = rnd(g, T, H, dtype=dtype), rnd(g, E, 2 * I, H, dtype=dtype, std=H ** -0.5), rnd(g, E, H, I, dtype=dtype, std=I ** -0.5)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).to(torch.int32)
    tw = torch.rand(T, k, generator=g)
    s = rnd(g, T, H, dtype=dtype) if shared else None
    sg = rnd(g, 1, H, dtype=dtype, std=H ** -0.5) if gate else None
    cu = lambda t: None if t is None else t.cuda()                                         # noqa: E731
    got = fused_moe.fused_experts(x.cuda(), w13.cuda(), w2.cuda(), tw.cuda(), ids.cuda(), shared=cu(s), shared_gate=cu(sg))
    want = torch.zeros(T, H, dtype=torch.float64)
    for e in range(E):
        t, j = (ids == e).nonzero(as_tuple=True)
        y = do.expert(x[t].double(), {"gate": w13[e, :I].double(), "up": w13[e, I:].double(), "down": w2[e].double()})
        want.index_add_(0, t, tw[t, j, None].double() * y)
    if shared:
        want += s.double() if sg is None else torch.sigmoid(x.double() @ sg[0].double())[:, None] * s.double()
    close(got, want, dtype, 1.5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_product_on_the_cuda_cores_with_empty_and_uneven_groups(dtype):
    g = torch.Generator().manual_seed(5)
    counts, N, K = [0, 1, 31, 32, 33, 0, 70, 0], 37, 45
    off = torch.tensor([0] + list(np.cumsum(counts)), dtype=torch.int32).cuda()
    rows = sum(counts)
    a, w = rnd(g, 50, K, dtype=dtype), rnd(g, len(counts), N, K, dtype=dtype)
    src = torch.randint(0, 50, (rows,), generator=g).to(torch.int32)
    got = moe_native.grouped_linear_simple(a.cuda(), w.cuda(), off, False, rows, src.cuda())
    e = torch.repeat_interleave(torch.arange(len(counts)), torch.tensor(counts))
    close(got, torch.einsum("rk,rnk->rn", a[src.long()].double(), w[e].double()), dtype)


@pytest.mark.parametrize("M,I,K", [(1, 8, 64), (70, 72, 136), (300, 200, 512), (5, 136, 72)])
def test_gate_and_up_product_of_any_width(M, I, K):
    g = torch.Generator().manual_seed(I)
    x, w = rnd(g, M, K, dtype=torch.bfloat16), rnd(g, 2 * I, K, dtype=torch.bfloat16, std=K ** -0.5)
    want = do.silu(x.double() @ w[:I].double().T) * (x.double() @ w[I:].double().T)
    close(ops.linear_swiglu(x.cuda(), w.cuda()), want, torch.bfloat16)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("I", [1, 35, 64, 1000])
def test_activations(dtype, I):
    x = rnd(torch.Generator().manual_seed(I), 9, I, dtype=dtype, std=3.0)
    close(ops.activation(x.cuda(), "gelu"), do.gelu_erf(x.double()), dtype)
    x = rnd(torch.Generator().manual_seed(I), 9, 2 * I, dtype=dtype, std=3.0)
    close(ops.silu_and_mul(x.cuda()), do.silu(x[:, :I].double()) * x[:, I:].double(), dtype)
