"""The kernels of the Vofelix decoder, each alone, against the plain definitions: bf16 and fp32, sizes that
are no multiple of anything, page, window and tile borders."""
import numpy as np
import pytest
import torch

import vofelix_oracle as vo
from vllm_ascend_b200 import ops
from vllm_ascend_b200.attention import mla
from vllm_ascend_b200.attention.metadata import AttentionMetadata
from vllm_ascend_b200.ops import linear_attn as la
from vllm_ascend_b200.ops import reference as ref
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, gated_head_norm, side_gate, stream_norm

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, dtype, scale=1.0):
    err = float((got.double().cpu() - want.double().cpu()).abs().max() / want.double().abs().max().clamp_min(1e-6))
    assert err < scale * (2e-5 if dtype == torch.float32 else 1.2e-2), err


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, dtype, std=1.0):
    return (torch.randn(*shape, generator=g) * std).to(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [1, 30, 33, 256, 1000, 4096])
def test_stream_norm(dtype, W):
    g = gen(W)
    T, V, eps = 9, 20, 1e-4
    w1, b1, w2, b2 = (rnd(g, W, dtype=dtype) for _ in range(4))
    table, ids = rnd(g, V, W, dtype=dtype), torch.randint(0, V, (T,), generator=g)
    y = rnd(g, T, W, dtype=dtype) + 3
    r0 = torch.randn(T, W, generator=g) * 2 + 1
    d = lambda t: t.double()                                                       # noqa: E731
    c = lambda t: t.cuda()                                                         # noqa: E731
    ln1, ln2, rms = NormSpec("layer", c(w1), c(b1)), NormSpec("layer", c(w2), c(b2)), NormSpec("rms", c(w1))
    r = c(torch.empty(T, W))
    x = stream_norm(r, None, None, ln2, eps, dtype, embed=c(table), ids=c(ids), embed_scale=5.0, embed_set=True)
    want = d(table)[ids] * 5.0
    close(r, want, torch.float32)
    if W > 1:
        close(x, vo.layer_norm(want, d(w2), d(b2), eps), dtype)
    r = c(r0)
    x = stream_norm(r, c(y), ln1, PLAIN, eps, dtype)
    want = d(r0) + vo.layer_norm(d(y), d(w1), d(b1), eps)
    close(r, want, torch.float32, 2)
    close(x, want, dtype)
    r = c(r0)
    x = stream_norm(r, c(y), rms, ln2, eps, dtype, embed=c(table), ids=c(ids), embed_scale=0.5)
    want = d(r0) + vo.rms_norm(d(y), d(w1), eps) + d(table)[ids] * 0.5
    close(r, want, torch.float32, 2)
    if W > 1:
        close(x, vo.layer_norm(want, d(w2), d(b2), eps), dtype)
    r = c(r0)
    assert stream_norm(r, c(y), PLAIN, None, eps, dtype) is None
    close(r, d(r0) + d(y), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,slot", [(1, 2), (24, 1), (18, 3), (256, 0)])
def test_side_gate_and_activation(dtype, D, slot):
    g = gen(D)
    a, table = rnd(g, 7, D, dtype=dtype), rnd(g, 11, 4 * D, dtype=dtype)
    ids = torch.randint(0, 11, (7,), generator=g)
    got = side_gate(a.cuda(), ids.cuda(), table.cuda(), slot * D)
    close(got, vo.gelu_tanh(a.double()) * table.double()[ids][:, slot * D:(slot + 1) * D], dtype)
    x = rnd(g, 5, 2 * D, dtype=dtype)
    got = ops.activation(x.cuda(), "gelu_tanh", gated=True)
    close(got, vo.gelu_tanh(x[:, :D].double()) * x[:, D:].double(), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D", [(1, 1), (3, 20), (4, 128), (2, 45)])
def test_gated_head_norm(dtype, H, D):
    g = gen(D)
    o, z, w = rnd(g, 6, H, D, dtype=dtype), rnd(g, 6, 2 * H * D, dtype=dtype), rnd(g, D, dtype=dtype)
    got = gated_head_norm(o.cuda(), z.cuda()[:, H * D:], w.cuda(), 1e-5)
    want = vo.rms_norm(o.double(), w.double(), 1e-5) * vo.silu(z[:, H * D:].double()).view(6, H, D)
    close(got, want.reshape(6, H * D), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("K,C", [(1, 40), (2, 64), (3, 50), (4, 136), (4, 7), (7, 33)])
def test_short_convolution_over_portions(dtype, K, C):
    """Sequences cut into portions shorter and longer than the taps and than a tile of tokens, in a batch of
    changing order, with the gates in the same launch."""
    g = gen(K * 100 + C)
    H, lens = 3, [50, 1, 35, 18]
    x = [rnd(g, n, C, dtype=dtype) for n in lens]
    ba = [rnd(g, n, 2 * H, dtype=dtype, std=3.0) for n in lens]
    w = rnd(g, C, K, dtype=dtype)
    A, dt = torch.randn(H, generator=g), torch.randn(H, generator=g)
    state = torch.full((6, K - 1, C), 7.0, dtype=dtype, device="cuda")          # stale contents
    slots = [4, 0, 2, 5]
    got, beta, decay = ([[] for _ in lens] for _ in range(3))
    at, k = [0] * 4, 0
    while any(a < n for a, n in zip(at, lens)):
        todo = [i for i in (range(4) if k % 2 else range(3, -1, -1)) if at[i] < lens[i]]
        take = [min([1, 2, 17, 3, 16][(k + i) % 5], lens[i] - at[i]) for i in todo]
        if k % 3 == 2:
            take = [1] * len(todo)
        cu = np.concatenate([[0], np.cumsum(take)]).astype(np.int32)
        xs = torch.cat([x[i][at[i]:at[i] + n] for i, n in zip(todo, take)]).cuda()
        bs = torch.cat([ba[i][at[i]:at[i] + n] for i, n in zip(todo, take)]).cuda()
        y, be, de = la.causal_conv1d(
            xs, w.cuda(), None, state, torch.from_numpy(cu).cuda(),
            torch.tensor([slots[i] for i in todo], dtype=torch.int32).cuda(),
            torch.tensor([at[i] > 0 for i in todo], dtype=torch.int32).cuda(), uniform=max(take) == 1,
            gates=(bs, A.cuda(), dt.cuda()))
        for j, i in enumerate(todo):
            for dst, src in ((got, y), (beta, be), (decay, de)):
                dst[i].append(src[cu[j]:cu[j + 1]].cpu())
            at[i] += take[j]
        k += 1
    for i in range(4):
        close(torch.cat(got[i]), vo.silu(vo.short_conv(x[i].double(), w.double())), dtype)
        close(torch.cat(beta[i]), torch.sigmoid(ba[i][:, :H].double()), torch.float32)
        close(torch.cat(decay[i]), -torch.exp(A.double()) * vo.softplus(ba[i][:, H:].double() + dt.double()),
              torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,Hk,d,vd", [(4, 2, 12, 20), (1, 1, 1, 1), (6, 2, 40, 48), (3, 3, 64, 5), (4, 4, 128, 128),
                                       (2, 1, 96, 64), (2, 2, 200, 72), (3, 1, 33, 130)])
def test_delta_rule_over_portions(dtype, H, Hk, d, vd):
    g = gen(d * 1000 + vd)
    lens, slots = [37, 5], [2, 0]
    q, k = ([rnd(g, n, Hk, d, dtype=dtype) + 0.1 for n in lens] for _ in range(2))
    v = [rnd(g, n, H, vd, dtype=dtype) for n in lens]
    beta = [torch.rand(n, H, generator=g) for n in lens]
    logg = [-torch.rand(n, H, generator=g) for n in lens]
    state = torch.full((3, H, d, vd), 9.0, device="cuda")
    owner = [h // (H // Hk) for h in range(H)]
    for sizes in ([(37, 5)], [(2, 0), (1, 1), (1, 1), (3, 3), (30, 0)], [(1, 1)] * 5 + [(32, 0)]):
        got, at = [[], []], [0, 0]
        for pair in sizes:
            todo = [i for i in (1, 0) if pair[i]]
            cu = np.concatenate([[0], np.cumsum([pair[i] for i in todo])]).astype(np.int32)
            part = lambda t: torch.cat([t[i][at[i]:at[i] + pair[i]] for i in todo]).cuda()      # noqa: E731
            o = la.gated_delta_rule(part(q), part(k), part(v), part(logg), part(beta), state, torch.from_numpy(cu).cuda(),
                                    torch.tensor([slots[i] for i in todo], dtype=torch.int32).cuda(),
                                    torch.tensor([at[i] > 0 for i in todo], dtype=torch.int32).cuda(), d ** -0.5,
                                    uniform=all(pair[i] == 1 for i in todo))
            for j, i in enumerate(todo):
                got[i].append(o[cu[j]:cu[j + 1]].cpu())
                at[i] += pair[i]
        assert at == lens
        for i in range(2):
            want, S = vo.delta_scan(vo.unit(q[i].double())[:, owner] * d ** -0.5, vo.unit(k[i].double())[:, owner],
                                    v[i].double(), beta[i].double(), torch.exp(logg[i].double()))
            close(torch.cat(got[i]), want, dtype)
            close(state[slots[i]], S, torch.float32, 4)
    assert bool((state[1] == 9.0).all())                     # nobody's slot


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,Hk,d,vd", [(4, 2, 12, 20), (6, 2, 40, 48), (4, 4, 128, 128), (2, 2, 200, 72), (3, 1, 33, 130),
                                       (2, 1, 256, 128), (3, 3, 16, 4)])
def test_delta_decode_with_the_gated_norm(dtype, H, Hk, d, vd):
    g = gen(d + vd)
    B, owner = 5, [h // (H // Hk) for h in range(H)]
    q, k = (rnd(g, B, Hk, d, dtype=dtype) for _ in range(2))
    v, z, w = rnd(g, B, H, vd, dtype=dtype), rnd(g, B, 2 * H * vd, dtype=dtype), rnd(g, vd, dtype=dtype)
    beta, logg = torch.rand(B, H, generator=g), -torch.rand(B, H, generator=g)
    S0 = torch.randn(B + 1, H, d, vd, generator=g)
    state, slots, init = S0.cuda(), [3, 0, 5, 1, 2], [1, 0, 1, 1, 0]
    i32 = lambda t: torch.tensor(t, dtype=torch.int32).cuda()                           # noqa: E731
    got = la.gated_delta_rule(q.cuda(), k.cuda(), v.cuda(), logg.cuda(), beta.cuda(), state, i32(list(range(B + 1))),
                              i32(slots), i32(init), d ** -0.5, uniform=True,
                              gate=(z.cuda()[:, H * vd:], w.cuda(), 1e-5))
    for b in range(B):
        o, S = vo.delta_scan(vo.unit(q[b:b + 1].double())[:, owner] * d ** -0.5, vo.unit(k[b:b + 1].double())[:, owner],
                             v[b:b + 1].double(), beta[b:b + 1].double(), torch.exp(logg[b:b + 1].double()),
                             S0[slots[b]].double() if init[b] else None)
        want = vo.rms_norm(o[0], w.double(), 1e-5) * vo.silu(z[b, H * vd:].double()).view(H, vd)
        close(got[b], want.reshape(-1), dtype, 1.5)
        close(state[slots[b]], S, torch.float32, 4)
    assert torch.equal(state[4].cpu(), S0[4])


# ---------------------------------------------------------------- latent attention
def paged(lens, q_lens, bs, dc, dr, dtype, seed):
    """Latent / rotated-key caches with shuffled pages and the step's metadata."""
    g = gen(seed)
    nb = [(n + bs - 1) // bs for n in lens]
    perm = (torch.randperm(sum(nb), generator=g) + 1).to(torch.int32)
    table = torch.zeros(len(lens), max(nb) + 1, dtype=torch.int32)
    lat_c = rnd(g, sum(nb) + 1, bs, 1, dc, dtype=dtype)
    pe_c = rnd(g, sum(nb) + 1, bs, 1, dr, dtype=dtype)
    o = 0
    for b, n in enumerate(nb):
        table[b, :n] = perm[o:o + n]
        o += n
    cu = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32)
    pos = torch.cat([torch.arange(n - m, n) for n, m in zip(lens, q_lens)])
    sl = np.asarray(lens, dtype=np.int32)
    meta = AttentionMetadata(
        num_reqs=len(lens), num_actual_tokens=int(cu[-1]), max_query_len=max(q_lens), max_seq_len=max(lens),
        query_start_loc=torch.from_numpy(cu).cuda(), seq_lens=torch.from_numpy(sl).cuda(), block_table=table.cuda(),
        slot_mapping=None, positions=pos.cuda(), query_start_loc_cpu=cu, seq_lens_cpu=sl)
    return lat_c, pe_c, table, meta


def slot(table, bs, b, j):
    return int(table[b, j // bs]), j % bs


def attend(q_lat, q_pe, lat, pe, first, last, scale, sink):
    s = (q_lat @ lat[first:last + 1].T + q_pe @ pe[first:last + 1].T) * scale
    top = s.max(-1, keepdim=True).values if sink is None else torch.maximum(s.max(-1, keepdim=True).values, sink[:, None])
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True) + (0 if sink is None else torch.exp(sink[:, None] - top))
    return (e / den) @ lat[first:last + 1]


CASES = [  # H, dc, dr, block, window, lens, q_lens
    (7, 104, 24, 64, 50, [300, 49, 50, 51, 1], [300, 49, 50, 51, 1]),
    (7, 104, 24, 64, 50, [300, 178, 129, 1, 77], [1, 1, 1, 1, 1]),
    (3, 20, 6, 16, 7, [40, 9, 200], [40, 1, 2]),
    (16, 512, 64, 128, 130, [700, 131, 258], [37, 131, 1]),
    (32, 512, 64, 128, 0, [500, 100], [1, 1]),
    (20, 136, 64, 16, 33, [90, 300], [90, 3]),
    (17, 264, 24, 32, 1, [64, 5], [64, 5]),
    (1, 8, 8, 64, 128, [257, 600], [257, 1]),
    (5, 200, 8, 128, 600, [1500, 30], [1, 1]),
    (2, 600, 100, 16, 40, [70], [70]),
    (40, 64, 32, 64, 200, [450, 210], [5, 210]),
]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink_on", [True, False])
@pytest.mark.parametrize("case", range(len(CASES)))
def test_latent_attention_window_and_sink(dtype, sink_on, case):
    H, dc, dr, bs, window, lens, q_lens = CASES[case]
    lat_c, pe_c, table, meta = paged(lens, q_lens, bs, dc, dr, dtype, case)
    g = gen(case + 100)
    T, scale = sum(q_lens), 0.6 * (dc + dr) ** -0.5
    q_lat, q_pe = rnd(g, T, H, dc, dtype=dtype), rnd(g, T, H, dr, dtype=dtype)
    sink = torch.randn(H, generator=g) * 3 + 1 if sink_on else None
    got = mla.mla_paged_attention(q_lat.cuda(), q_pe.cuda(), lat_c.cuda(), pe_c.cuda(), meta, scale, window=window,
                                  sink=None if sink is None else sink.cuda()).cpu()
    for b, (n, m) in enumerate(zip(lens, q_lens)):
        pages = table[b, :(n + bs - 1) // bs].long()
        lat, pe = lat_c[pages].reshape(-1, dc)[:n].double(), pe_c[pages].reshape(-1, dr)[:n].double()
        r0 = int(meta.query_start_loc_cpu[b])
        want = torch.stack([attend(q_lat[r0 + i].double(), q_pe[r0 + i].double(), lat, pe,
                                   max(0, n - m + i - window + 1) if window else 0, n - m + i, scale,
                                   None if sink is None else sink.double()) for i in range(m)])
        close(got[r0:r0 + m], want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 127, 128, 129, 300])
def test_one_key_that_stands_out(dtype, decode, window):
    """A key whose score towers over all others is found just inside the window, and is invisible one place
    further back, wherever the place falls within pages and key tiles."""
    H, dc, dr, bs = 6, 40, 8, 64
    for n in (window + 1, 128 + window, 400):
        lens, q_lens = [n, 330], ([1, 1] if decode else [min(n, 5), 330])
        lat_c, pe_c, table, meta = paged(lens, q_lens, bs, dc, dr, dtype, n)
        lat_c *= 0.1
        pe_c *= 0.1
        T = sum(q_lens)
        q_lat, q_pe = torch.zeros(T, H, dc, dtype=dtype), torch.zeros(T, H, dr, dtype=dtype)
        q_pe[..., 0] = 1.0
        for back, seen in ((window - 1, True), (window, False)):
            j = n - 1 - back
            if j < 0:
                continue
            pc, lc = pe_c.clone(), lat_c.clone()
            blk, off = slot(table, bs, 0, j)
            pc[blk, off, 0, 0] = 40.0
            lc[blk, off, 0] = 5.0
            out = mla.mla_paged_attention(q_lat.cuda(), q_pe.cuda(), lc.cuda(), pc.cuda(), meta, 1.0, window=window,
                                          sink=torch.zeros(H, device="cuda")).float().cpu()
            last = out[q_lens[0] - 1]
            assert bool(((last - 5.0).abs() < 0.05).all()) if seen else bool((last.abs() < 0.6).all()), (n, back)


def test_a_sink_far_above_or_below_the_scores():
    lat_c, pe_c, table, meta = paged([300], [1], 64, 64, 16, torch.bfloat16, 1)
    q_lat, q_pe = torch.zeros(1, 4, 64, dtype=torch.bfloat16), torch.zeros(1, 4, 16, dtype=torch.bfloat16)
    sink = torch.tensor([-300.0, 0.0, 5.7, 300.0])
    out = mla.mla_paged_attention(q_lat.cuda(), q_pe.cuda(), lat_c.cuda(), pe_c.cuda(), meta, 1.0, window=128,
                                  sink=sink.cuda()).float().cpu()[0]
    pages = table[0, :5].long()
    mean = lat_c[pages].reshape(-1, 64)[172:300].float().mean(0)
    for h, share in enumerate([1.0, 128 / 129, 128 / (128 + float(torch.exp(sink[2]))), 0.0]):
        assert float((out[h] - mean * share).abs().max()) < 2e-2 * float(mean.abs().max()) + 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dn,dr,dc", [(3, 11, 6, 20), (5, 56, 24, 120), (2, 8, 2, 8)])
def test_latent_preprocess(dtype, H, dn, dr, dc):
    g = gen(dc)
    T, base = 13, 5000.0
    sc = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    table = ref.build_cos_sin_cache(dr, 400, base, {"rope_type": "yarn_interp", "factor": 4.0, "beta_fast": 8.0,
                                                    "beta_slow": 1.0, "original_max_position_embeddings": 64}, "cuda")
    q, kv, w = rnd(g, T, H, dn + dr, dtype=dtype), rnd(g, T, dc + dr, dtype=dtype), rnd(g, dc, dtype=dtype)
    pos = torch.randint(0, 400, (T,), generator=g)
    slots = torch.randperm(40, generator=g)[:T]
    slots[3] = -1
    lat, pe = torch.zeros(5, 8, 1, dc, dtype=dtype).cuda(), torch.zeros(5, 8, 1, dr, dtype=dtype).cuda()
    qc = q.cuda()
    ops.mla_preprocess(qc, kv.cuda(), w.cuda(), 1e-5, pos.cuda(), table, slots.cuda(), lat, pe, dn, dr)
    for t in range(T):
        p = int(pos[t])
        close(qc[t, :, dn:], vo.rotate(q[t, :, dn:].double(), p, dr, base, sc), dtype)
        assert torch.equal(qc[t, :, :dn].cpu(), q[t, :, :dn])
        if slots[t] >= 0:
            close(lat.view(-1, dc)[slots[t]], vo.rms_norm(kv[t, :dc].double(), w.double(), 1e-5), dtype)
            close(pe.view(-1, dr)[slots[t]], vo.rotate(kv[t, dc:].double(), p, dr, base, sc), dtype)
    assert int((lat.view(-1, dc).abs().sum(-1) > 0).sum()) == T - 1
