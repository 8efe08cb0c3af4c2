"""The kernels the Nevotar decoder adds or extends, each alone, against the plain definitions: bf16 and fp32, sizes that
are multiples of a vector and sizes that are not, page, window, tile and chunk borders."""
import numpy as np
import pytest
import torch

import nevotar_oracle as no
from dubizen_oracle import rotate_halves
from gpu_utils import make_paged_case
from test_gpu_pegopel_ops import MIXED, SINGLE, close, rnd
from vllm_ascend_b200 import _native, ops
from vllm_ascend_b200.attention import variant as va
from vllm_ascend_b200.ops import fused_moe
from vllm_ascend_b200.ops import linear_attn as la
from vllm_ascend_b200.ops import linear_recurrence as lr
from vllm_ascend_b200.ops import reference as ref
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, stream_norm

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(autouse=True)
def no_status():
    yield
    torch.cuda.synchronize()
    _native.check_status(torch.device("cuda"))


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


# ---------------------------------------------------------------- norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,groups", [(24, 24), (45, 5), (256, 2), (1000, 8), (4096, 4), (4096, 1), (4096, 32), (96, 3)])
def test_stream_norm_in_groups(dtype, W, groups):
    g = gen(W + groups)
    r, y, w, table = torch.randn(9, W, generator=g), rnd(g, 9, W, dtype=dtype), rnd(g, W, dtype=dtype), rnd(g, 5, W, dtype=dtype)
    ids = torch.randint(0, 5, (9,), generator=g)
    n = NormSpec("rms", w.cuda(), None, groups)
    rc = torch.empty(9, W, device="cuda")
    x = stream_norm(rc, None, None, n, 1e-4, dtype, embed=table.cuda(), ids=ids.cuda(), embed_set=True)
    close(x, no.group_norm(table[ids].double(), w.double(), 1e-4, groups), dtype, 4)
    rc = r.cuda()
    x = stream_norm(rc, y.cuda(), PLAIN, n, 1e-4, dtype)
    close(rc, r.double() + y.double(), torch.float32)
    close(x, no.group_norm(r.double() + y.double(), w.double(), 1e-4, groups), dtype, 4)
    stream_norm(rc, y.cuda(), n, None, 1e-4, dtype)                  # behind a sub-layer as well
    close(rc, r.double() + y.double() + no.group_norm(y.double(), w.double(), 1e-4, groups), torch.float32, 4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("groups,size", [(1, 1), (4, 9), (3, 64), (2, 200), (8, 128), (1, 4096), (2, 5000), (1, 1031)])
def test_group_norm_with_gate_and_shared_weights(dtype, groups, size):
    g = gen(groups * size)
    T, C = 11, groups * size
    y, z, w = rnd(g, T, C + 8, dtype=dtype), rnd(g, T, C + 24, dtype=dtype), rnd(g, C, dtype=dtype)
    yc, zc = y.cuda()[:, :C], z.cuda()[:, 8:C + 8]
    out = torch.zeros(T, C + 16, dtype=dtype, device="cuda")
    lr.group_norm(yc, w.cuda(), groups, 1e-4, zc, 0.7, out[:, 8:C + 8])
    want = 0.7 * no.group_norm(y[:, :C].double() * no.silu(z[:, 8:C + 8].double()), w.double(), 1e-4, groups)
    close(out[:, 8:C + 8], want, dtype, 3)
    assert not out[:, :8].any() and not out[:, C + 8:].any()
    close(lr.group_norm(yc, w.cuda()[:size], groups, 1e-4), no.group_norm(y[:, :C].double(), w[:size].double().repeat(groups), 1e-4, groups),
          dtype, 3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D", [(1, 1), (3, 11), (6, 56), (16, 128), (2, 512)])
def test_map_difference(dtype, H, D):
    g = gen(D)
    o = torch.randn(7, 2 * H, D, generator=g)
    o[:, 1::2] = o[:, 0::2] + 0.1 * o[:, 1::2]                       # maps that almost cancel
    want = o[:, 0::2].double() - 0.95 * o[:, 1::2].double()
    want = want / torch.sqrt((want ** 2).mean(-1, keepdim=True) + 1e-4) * 0.6
    close(lr.map_difference(o.cuda(), 0.95, 1e-4, 0.6, dtype), want.reshape(7, -1), dtype, 2)


# ---------------------------------------------------------------- recurrences
PLANS = [[1, 2, 17, 3, 16], [1], [64], [8, 9, 7]]


def run_portions(lens, plan, step):
    """Sequences of the given lengths in portions, in batches of changing order; ``step(seqs, rows, cu, later, uniform)``
    -> outputs of the step's rows.  Returns the outputs per sequence."""
    got, at, k = [[] for _ in lens], [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        todo = [i for i in (range(len(lens)) if k % 2 else reversed(range(len(lens)))) if at[i] < lens[i]]
        take = [min(plan[(k + i) % len(plan)], lens[i] - at[i]) for i in todo]
        if k % 3 == 2:
            take = [1] * len(todo)
        cu = np.concatenate([[0], np.cumsum(take)]).astype(np.int32)
        y = step(todo, [slice(at[i], at[i] + n) for i, n in zip(todo, take)], torch.from_numpy(cu).cuda(),
                 torch.tensor([at[i] > 0 for i in todo], dtype=torch.int32).cuda(), max(take) == 1).cpu()
        for j, i in enumerate(todo):
            got[i].append(y[cu[j]:cu[j + 1]])
            at[i] += take[j]
        k += 1
    return [torch.cat(x) for x in got]


@pytest.mark.parametrize("plan", PLANS)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,P", [(6, 3, 9, 5), (8, 2, 48, 32), (1, 1, 1, 1), (4, 1, 128, 64), (4, 4, 256, 24), (2, 1, 72, 136),
                                     (8, 8, 64, 128)])
def test_state_space(dtype, H, G, N, P, plan):
    g = gen(H * N)
    lens, slots, inner = [50, 1, 35, 18], [4, 0, 2, 5], H * P
    C = inner + 2 * G * N
    pad = (8 - (C + H) % 8) % 8
    rows = [rnd(g, n, C + H + pad, dtype=dtype) for n in lens]
    A, dtb, D = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    sp = lr.StateSpace(A.cuda(), dtb.cuda(), D.cuda(), G)
    state = torch.full((6, H, N, P), 7.0, device="cuda")              # stale contents

    def step(seqs, parts, cu, later, uniform):
        x = torch.cat([rows[i][s] for i, s in zip(seqs, parts)]).cuda()
        return lr.state_space(sp, x[:, :C], x[:, C:C + H], state, cu, torch.tensor([slots[i] for i in seqs], dtype=torch.int32).cuda(),
                              later, uniform=uniform)
    got = run_portions(lens, plan, step)
    for i, n in enumerate(lens):
        r = rows[i].double()
        y, S = no.state_space(r[:, :inner].reshape(n, H, P), r[:, inner:inner + G * N].reshape(n, G, N),
                              r[:, inner + G * N:C].reshape(n, G, N), no.softplus(r[:, C:C + H] + dtb.double()), A.double(), D.double())
        close(got[i], y.reshape(n, inner), dtype, 2)
        close(state[slots[i]], S, torch.float32, 2)
    assert bool((state[[1, 3]] == 7.0).all())


@pytest.mark.parametrize("plan", PLANS)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,P", [(3, 9, 13), (4, 48, 64), (1, 1, 1), (2, 128, 128), (2, 136, 72), (3, 64, 24), (1, 256, 264)])
def test_forget_recurrence(dtype, H, D, P, plan):
    g = gen(D + P)
    lens, slots, n0, n1 = [50, 1, 35, 18], [4, 0, 2, 5], H * D, H * P
    width = (2 * n0 + n1 + 7) // 8 * 8
    rows = [rnd(g, n, width, dtype=dtype, std=2.0) for n in lens]
    fb, nw = rnd(g, n0, dtype=dtype, std=3.0), rnd(g, P, dtype=dtype)
    low = torch.rand(n0, generator=g).to(dtype)
    state = torch.full((6, H, D, P), 7.0, device="cuda")

    def step(seqs, parts, cu, later, uniform):
        x = torch.cat([rows[i][s] for i, s in zip(seqs, parts)]).cuda()
        return lr.forget_recurrence(x[:, :n0], x[:, n0:2 * n0], x[:, 2 * n0:2 * n0 + n1], fb.cuda(), low.cuda(), state, cu,
                                    torch.tensor([slots[i] for i in seqs], dtype=torch.int32).cuda(), later, nw.cuda(), 1e-4,
                                    uniform=uniform)
    got = run_portions(lens, plan, step)
    for i, n in enumerate(lens):
        r = rows[i].double()
        gate = low.double() + (1 - low.double()) / (1 + torch.exp(-(r[:, n0:2 * n0] + fb.double())))
        o, S = no.forget_recurrence(no.silu(r[:, :n0]).view(n, H, D), gate.view(n, H, D), r[:, 2 * n0:2 * n0 + n1].reshape(n, H, P))
        close(got[i], no.rms_norm(o, nw.double(), 1e-4).reshape(n, n1), dtype, 6)
        close(state[slots[i]], S, torch.float32, 2)
    assert bool((state[[1, 3]] == 7.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,N,P", [(4, 4, 64, 64), (6, 2, 20, 11)])
def test_gated_linear_attention_on_the_gpu(dtype, H, G, N, P):
    g = gen(N)
    cu_h = [0, 33, 34, 34, 60]
    T = cu_h[-1]
    q, k, v, dec = rnd(g, T, G, N, dtype=dtype), rnd(g, T, G, N, dtype=dtype), rnd(g, T, H, P, dtype=dtype), -torch.rand(T, H, generator=g)
    cu, slots, init = torch.tensor(cu_h, dtype=torch.int32), torch.tensor([2, 0, 3, 1], dtype=torch.int32), torch.tensor([1, 0, 1, 1], dtype=torch.int32)
    state = torch.randn(5, H, N, P, generator=g)
    want_state = state.clone()
    want = la.gated_linear_attention_ref(q.double(), k.double(), v.double(), dec, want_state, cu, slots, init)
    sc = state.cuda()
    got = la.gated_linear_attention(q.cuda(), k.cuda(), v.cuda(), dec.cuda(), sc, cu.cuda(), slots.cuda(), init.cuda(), cu_cpu=cu_h)
    close(got, want, dtype, 2)
    close(sc, want_state, torch.float32, 4)


# ---------------------------------------------------------------- in front of the attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,vd,rot,temp,norm,kind", [
    (6, 3, 10, 7, 6, False, True, "talk"), (8, 4, 64, 64, 64, False, True, "talk"), (10, 5, 32, 40, 16, True, True, "talk"),
    (4, 2, 48, 96, 0, True, False, "maps"), (3, 1, 7, 11, 0, True, False, "maps"), (1, 1, 1, 1, 0, False, False, "maps"),
    (8, 2, 128, 128, 128, True, False, "plain"), (16, 4, 128, 128, 128, False, True, "talk"), (2, 1, 2, 3, 2, False, True, "talk")])
def test_wide_queries(dtype, H, G, d, vd, rot, temp, norm, kind):
    g = gen(H * d)
    T, bs, eps = 21, 8, 1e-5
    nq, nk = (H, G) if kind != "maps" else (2 * H, 2 * G)
    x = rnd(g, T, nq * d + nk * d + G * vd + 8, dtype=dtype)
    qn, kn = (rnd(g, d, dtype=dtype) + 1 for _ in "qk") if norm else (None, None)
    mix = torch.randn(H, H, generator=g) if kind == "talk" else None
    table = 1 + torch.rand(64, generator=g) if temp else None
    cs = ref.build_cos_sin_cache(rot, 64, 1e4, None).cuda() if rot else None
    cu_ = lambda t: None if t is None else t.cuda()                                             # noqa: E731
    parts = {"talk": G, "maps": 2, "plain": 1}[kind]
    spec = va.PrepSpec(nq, nk, d, vd, eps, cu_(qn), cu_(kn), (nq * d, nk * d), rot_dims=rot, cos_sin=cs, head_norm=norm, v_heads=G,
                       key_parts=parts, part_run=H // G if kind == "talk" else 1, mix=cu_(mix), q_scale=cu_(table))
    kc, vc = torch.zeros(6, bs, nk // parts, parts * d, dtype=dtype, device="cuda"), ops.alloc_kv_cache(6, bs, G, vd, dtype, "cuda")
    slot = torch.randperm(48, generator=g)[:T]
    slot[4] = -1
    pos = torch.randint(0, 64, (T,), generator=g)

    class Meta:
        num_reqs, max_query_len = 1, T
        query_start_loc = torch.tensor([0, T], dtype=torch.int32).cuda()
        slot_mapping, positions, state_slots, has_initial_state = slot.cuda(), pos.cuda(), None, None
    got = va.qkv_prep(spec, x.cuda(), Meta, kc, vc)
    q, k, v = (t.double().view(T, -1, n) for t, n in ((x[:, :nq * d], d), (x[:, nq * d:(nq + nk) * d], d),
                                                     (x[:, (nq + nk) * d:(nq + nk) * d + G * vd], vd)))
    if norm:
        q, k = no.rms_norm(q, qn.double(), eps), no.rms_norm(k, kn.double(), eps)
    if rot:             # the kernel's pairs are (2i, 2i + 1)
        order = torch.arange(d)
        order[:rot] = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])
        back = torch.argsort(order)
        q, k = (torch.stack([rotate_halves(t[i][:, order], int(pos[i]), rot, 1e4)[:, back] for i in range(T)]) for t in (q, k))
    if temp:
        q = q * table.double()[pos][:, None, None]
    want = torch.zeros(T, spec.out_heads, parts, d, dtype=torch.float64)
    for oh in range(spec.out_heads):
        for h in range(nq):
            c = h // (H // G) if kind == "talk" else h % parts
            f = float(mix[oh, h]) if kind == "talk" else float(oh == h)
            want[:, oh, c] += f * q[:, h]
    close(got, want.flatten(2), dtype, 2)
    for t in range(T):
        if slot[t] >= 0:
            b, o = int(slot[t]) // bs, int(slot[t]) % bs
            close(kc[b, o].reshape(nk, d), k[t], dtype, 2)
            close(vc[b, o], v[t], dtype)
    assert int((kc.flatten(2).abs().sum(-1) > 0).sum()) == T - 1


# ---------------------------------------------------------------- attention over wide or shared keys
def run_wide(dtype, H, Hv, Hk, d, vd, bs, q_lens, ctx, window, kernel, splits=1, layout="HND", f32=False, scale=None, factor=0.7):
    g = gen(H * d + window)
    q, _, _, meta = make_paged_case(q_lens, ctx, H, Hk, d, bs, dtype=dtype, layout=layout, tok_per_tile=1)[:4]
    meta.num_decodes = next((i for i, n in enumerate(q_lens) if n > 1), len(q_lens))
    meta.positions = torch.cat([torch.arange(c, c + n) for c, n in zip(ctx, q_lens)]).cuda()
    nb = int(meta.block_table.max()) + 1
    k, v = (ops.alloc_kv_cache(nb, bs, h, w, dtype, "cuda", layout) for h, w in ((Hk, d), (Hv, vd)))
    for t in (k, v):
        t.copy_(rnd(g, *t.shape, dtype=dtype).cuda())
    scale = d ** -0.5 * 2 if scale is None else scale
    o = va.AttnOptions(scale, window, out_scale=factor, out_f32=f32)
    buf = torch.zeros(q.shape[0], H * vd + 24, dtype=torch.float32 if f32 else dtype, device="cuda")
    out = buf[:, 8:8 + H * vd].unflatten(1, (H, vd))
    if kernel == "prefill":
        va.variant_attention_prefill(q, k, v, meta, o, None, out, wide=d > 128)
    elif kernel == "decode":
        va.wide_attention_decode(q, k, v, meta, o, out, num_splits=splits)
    elif kernel == "simple":
        va.variant_attention_simple(q, k, v, meta, o, None, out)
    else:
        va.variant_attention(q, k, v, meta, o, None, out)
    cu = meta.query_start_loc_cpu
    for b, (n, c) in enumerate(zip(q_lens, ctx)):
        kb, vb = (ref.gather_kv(t, meta.block_table[b], c + n).double().cpu() for t in (k, v))
        own = torch.arange(H) // (H // Hv)
        kb, vb = kb[:, own * Hk // Hv], vb[:, own]
        for i in range(n):
            p = c + i
            lo = max(0, p - window + 1) if window else 0
            s = torch.einsum("hd,jhd->hj", q[cu[b] + i].double().cpu(), kb[lo:p + 1]) * scale
            close(out[cu[b] + i], factor * torch.einsum("hj,jhv->hv", no.softmax_rows(s), vb[lo:p + 1]), dtype)
    assert not buf[:, :8].any() and not buf[:, 8 + H * vd:].any()


WIDE = [(8, 4, 1, 256, 64, 64, "HND"), (10, 5, 1, 160, 40, 16, "NHD"), (12, 3, 3, 192, 56, 128, "HND"), (16, 4, 1, 512, 128, 64, "HND"),
        (6, 2, 1, 136, 8, 32, "NHD"), (8, 8, 1, 448, 24, 256, "HND"), (4, 2, 2, 384, 128, 64, "NHD"), (12, 6, 2, 320, 72, 64, "HND")]


@pytest.mark.parametrize("window", [0, 1, 70, 136, 300])
@pytest.mark.parametrize("H,Hv,Hk,d,vd,bs,layout", WIDE)
def test_wide_prefill_attention(H, Hv, Hk, d, vd, bs, layout, window):
    run_wide(torch.bfloat16, H, Hv, Hk, d, vd, bs, *MIXED, window, "prefill", layout=layout, f32=window == 70)


@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("window", [0, 1, 70, 300])
@pytest.mark.parametrize("H,Hv,Hk,d,vd,bs,layout", WIDE + [(32, 4, 1, 1024, 128, 64, "HND"), (24, 12, 1, 96, 16, 64, "NHD"),
                                                           (4, 4, 1, 24, 120, 64, "HND")])
def test_wide_decode_attention(H, Hv, Hk, d, vd, bs, layout, window, splits):
    run_wide(torch.bfloat16, H, Hv, Hk, d, vd, bs, *SINGLE, window, "decode", splits, layout, f32=window == 70)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,Hv,Hk,d,vd", [(8, 4, 1, 256, 64), (6, 3, 1, 30, 7), (6, 2, 2, 14, 11), (18, 9, 1, 576, 8), (4, 2, 1, 1600, 40)])
def test_cuda_core_attention_over_shared_keys(dtype, H, Hv, Hk, d, vd):
    run_wide(dtype, H, Hv, Hk, d, vd, 16, *MIXED, 40, "simple", f32=dtype == torch.float32)
    run_wide(dtype, H, Hv, Hk, d, vd, 16, [1, 5], [33, 20], 0, "simple", f32=True)


@pytest.mark.parametrize("H,Hv,Hk,d,vd", [(8, 4, 1, 256, 64), (8, 4, 4, 96, 96), (8, 4, 1, 64, 16), (40, 1, 1, 16, 16), (18, 9, 1, 576, 8),
                                          (48, 4, 1, 160, 24)])
def test_mixed_batches_choose_their_kernels(H, Hv, Hk, d, vd):
    for lens, ctx in (MIXED, SINGLE, ([40, 3], [0, 130])):
        run_wide(torch.bfloat16, H, Hv, Hk, d, vd, 64, lens, ctx, 130, "any", f32=H == 8)


@pytest.mark.parametrize("kernel", ["prefill", "decode", "simple"])
def test_one_key_inside_and_outside_the_window(kernel):
    """A key whose score towers over all others, at the window's edge and at page and tile borders: seen or not."""
    H, Hv, d, vd, bs, window = 8, 4, 256, 64, 64, 136
    dtype = torch.float32 if kernel == "simple" else torch.bfloat16
    for pos in (135, 136, 137, 200, 255, 256, 300):
        q, _, _, meta = make_paged_case([1], [pos], H, 1, d, bs, dtype=dtype, tok_per_tile=1)[:4]
        meta.num_decodes, meta.positions = 1, torch.tensor([pos]).cuda()
        nb = int(meta.block_table.max()) + 1
        o = va.AttnOptions(1.0, window)
        fn = {"prefill": lambda *a: va.variant_attention_prefill(*a, wide=True), "decode": va.wide_attention_decode,
              "simple": va.variant_attention_simple}[kernel]
        for j in {0, pos - window - 1, pos - window, pos - window + 1, 63, 64, 127, 128, pos - 1, pos}:
            if not 0 <= j <= pos:
                continue
            k, v = torch.zeros(nb, bs, 1, d, dtype=dtype, device="cuda"), torch.zeros(nb, bs, Hv, vd, dtype=dtype, device="cuda")
            page = int(meta.block_table[0, j // bs])
            k[page, j % bs] = q[0, 0] * 16 / float((q[0, 0].float() ** 2).sum())
            v[page, j % bs] = 1.0
            got = float(fn(q, k, v, meta, o)[0, 0, 0])
            assert (got > 0.9) if pos - j < window else got == 0.0, (pos, j, got)


# ---------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,H,ff,shared", [(37, 7, 3, 45, 13, 11), (300, 16, 1, 256, 64, 128), (5, 24, 5, 128, 72, 48),
                                                 (1, 1, 1, 24, 1, 0), (700, 8, 2, 64, 136, 256), (64, 300, 4, 96, 8, 40)])
def test_experts_on_weighted_inputs(dtype, T, E, top, H, ff, shared):
    g = gen(T)
    mats = {}
    for name, n in [(f"e{e}", ff) for e in range(E)] + ([("shared", shared)] if shared else []):
        for part in ("gate", "up", "down"):
            rows, cols = (H, n) if part == "down" else (n, H)
            mats[f"{name}.{part}"] = (torch.randn(rows, cols, generator=g) * 2 * cols ** -0.5).to(dtype)
    x, router = rnd(g, T, H, dtype=dtype), (torch.randn(E, H, generator=g) * 3 * H ** -0.5).to(dtype)
    z = ops.linear_fp32(x.cuda(), router.cuda())
    w, ids = fused_moe.gating_topk(z, top, "sigmoid", renorm=False)
    s = None
    if shared:
        s = torch.nn.functional.linear(ops.linear_swiglu(x.cuda(), torch.cat([mats["shared.gate"], mats["shared.up"]]).cuda(), limit=1.1),
                                       mats["shared.down"].cuda())
        close(s, no.clamped_expert(x.double(), {k: t.double() for k, t in no.sub(mats, "shared.").items()}, 1.1), dtype, 2)
    got = fused_moe.fused_experts(x.cuda(), torch.stack([torch.cat([mats[f"e{e}.gate"], mats[f"e{e}.up"]]) for e in range(E)]).cuda(),
                                  torch.stack([mats[f"e{e}.down"] for e in range(E)]).cuda(), w, ids, shared=s, limit=0.8,
                                  weight_input=True)
    d = {k: t.double() for k, t in mats.items()}
    want = torch.zeros(T, H, dtype=torch.float64)
    for t in range(T):
        chosen = no.route(z[t].double().cpu(), top)
        assert sorted(chosen) == sorted(int(e) for e in ids[t])
        for e, f in chosen.items():
            want[t] += no.clamped_expert(f * x[t].double(), no.sub(d, f"e{e}."), 0.8)
        if shared:
            want[t] += no.clamped_expert(x[t].double(), no.sub(d, "shared."), 1.1)
    close(got, want, dtype, 2)


@pytest.mark.parametrize("M", [3, 130, 1024])
@pytest.mark.parametrize("I,K", [(128, 256), (48, 128), (384, 512)])
def test_clamped_gate_in_the_product(M, I, K):
    g = gen(M + I)
    x, w = rnd(g, M, K, dtype=torch.bfloat16), rnd(g, 2 * I, K, dtype=torch.bfloat16, std=2 * K ** -0.5)
    want = no.clamped_expert(x.double(), {"gate": w[:I].double(), "up": w[I:].double(), "down": torch.eye(I).double()}, 1.5)
    close(ops.linear_swiglu(x.cuda(), w.cuda(), limit=1.5), want, torch.bfloat16)
    plain = no.silu(x.double() @ w[:I].double().T) * (x.double() @ w[I:].double().T)
    close(ops.linear_swiglu(x.cuda(), w.cuda()), plain, torch.bfloat16)
    if I % 128 == 0:
        close(ops.linear_swiglu(x.cuda(), w.cuda(), two_cta=True, limit=1.5), want, torch.bfloat16)
