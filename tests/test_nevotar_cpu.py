"""Nevotar on the CPU engine (fp32) against the plain definitions: configuration, loading, cache and state handling,
scheduling, generation, the replay program."""
import io
import json
import sys

import numpy as np
import pytest
import torch

import nevotar_cases as nc
import nevotar_oracle as no
from vllm_ascend_b200.attention import variant as va
from vllm_ascend_b200.config import ModelConfig, get_model_config
from vllm_ascend_b200.engine.replay import TraceReplayer, make_replay_engine
from vllm_ascend_b200.models.hgrn2 import HGRN2Mixer
from vllm_ascend_b200.models.parallel_mixer import ParallelMixer
from vllm_ascend_b200.ops import fused_moe
from vllm_ascend_b200.ops import linear_recurrence as lr
from vllm_ascend_b200.ops.stream import NormSpec, stream_norm

TOL = 1e-4


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = nc.CONFIGS[name]()
            w = nc.weights(cfg, seed=ord(name))
            made[name] = (cfg, w, nc.save(tmp_path_factory.mktemp("nevotar") / name, cfg, w))
        return made[name]
    return get


def engine(path, max_tokens=256, page=16):
    return TraceReplayer(make_replay_engine(path, "float32", max_tokens, page=page, device="cpu"))


def test_config_reader():
    m = ModelConfig.from_hf_dict(nc.CONFIGS["B"]())
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_hidden_layers) == ("Nevotar", 128, 264, 4)
    assert (m.norm_type, m.norm_groups, m.pre_norm, m.sandwich_norm, m.tie_word_embeddings) == ("rms", 4, True, False, True)
    a, b, c, d = (m.layer_config(i) for i in range(4))
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.sliding_window, a.attention_multiplier,
            a.rotary_dims, a.rope_theta, a.parallel_scales) == (10, 5, 32, 40, 70, 0.2, 16, 2e5, (0.45, 0.9))
    assert a.attn_talk and a.qk_norm and not a.qk_norm_full and a.attention_bias and not a.attention_out_bias and a.rope_half_split
    assert a.mamba_config == {"n_heads": 8, "d_head": 24, "n_groups": 4, "d_state": 40, "d_conv": 4, "norm_groups": 8}
    assert (a.num_experts, a.num_experts_per_tok, a.moe_intermediate_size, a.expert_limit, a.shared_expert_intermediate_size,
            a.shared_expert_limit) == (24, 5, 72, 2.0, 48, 3.0)
    assert a.scoring_func == "sigmoid" and not a.norm_topk_prob and a.moe_weight_input and a.router_fp32
    assert (b.attn_map_diff, b.attn_query_temp, b.head_dim, b.v_head_dim, b.sliding_window) == (0.2, (0.25, 50), 96, 56, None)
    assert not b.qk_norm and not b.attn_talk and d.attn_query_temp is None and d.num_experts == 0 or m.num_experts
    assert (c.linear_num_value_heads, c.linear_key_head_dim, c.linear_value_head_dim) == (6, 40, 32)
    assert m.is_hybrid and m.keeps_sequence_state and [m.is_linear_layer(i) for i in range(4)] == [False, False, True, False]
    e = ModelConfig.from_hf_dict(nc.CONFIGS["E"]())
    assert [p.get("weights_of") for p in e.layer_plan] == [None, None, None, 0, 2, 1, 1, None]
    chain = nc.CONFIGS["E"]()
    chain["layers"][6]["weights_of"] = 5
    assert ModelConfig.from_hf_dict(chain).layer_plan[6]["weights_of"] == 1
    alone = nc.config(50, 16, 1, [nc.parallel((2, 1, 8, 8, 1.0, 4, (1e4, 8)), (2, 8, 4, 1, 3, 1), (1.0, 1.0))])
    assert ModelConfig.from_hf_dict(alone).keeps_sequence_state


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][3].update(weights_of=1), lambda c: c["layers"][3].update(weights_of=8),
    lambda c: c["layers"][3].update(weights_of=3), lambda c: c["norm"].update(groups=7),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), lambda c: c["layers"][1]["mixer"]["right"].update(groups=3),
    lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=5), lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26),
    lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][2]["mixer"].update(q_temp={"coef": 1.0, "every": 1.5}), lambda c: c["layers"][0].update(type="delta")])
def test_configurations_that_do_not_fit_are_refused(change):
    c = nc.CONFIGS["E"]()
    change(c)
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(c)


# ---------------------------------------------------------------- mechanisms
def test_norm_in_groups():
    g = torch.Generator().manual_seed(1)
    r, y, w = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g), torch.randn(12, generator=g)
    for groups in (1, 2, 3, 12):
        rr = r.clone()
        x = stream_norm(rr, y, NormSpec("plain"), NormSpec("rms", w, None, groups), 1e-3, torch.float32)
        torch.testing.assert_close(rr, r + y)
        torch.testing.assert_close(x.double(), no.group_norm((r + y).double(), w.double(), 1e-3, groups), rtol=1e-5, atol=1e-5)
    with pytest.raises(ValueError):
        NormSpec("rms", w, None, 5)
    with pytest.raises(ValueError):
        NormSpec("layer", w, None, 2)


def test_norms_of_read_outs():
    g = torch.Generator().manual_seed(2)
    y, z, w = (torch.randn(4, 24, generator=g) for _ in range(3))
    got = lr.group_norm(y, w[0], 3, 1e-3, z, 0.5)
    want = no.group_norm(y.double() * no.silu(z.double()), w[0].double(), 1e-3, 3) * 0.5
    torch.testing.assert_close(got.double(), want, rtol=1e-5, atol=1e-5)
    got = lr.group_norm(y, w[0, :6], 4, 1e-3)                     # one weight for all parts
    torch.testing.assert_close(got.double(), no.group_norm(y.double(), w[0, :6].double().repeat(4), 1e-3, 4), rtol=1e-5, atol=1e-5)
    o = torch.randn(4, 6, 5, generator=g)
    d = o[:, 0::2].double() - 0.7 * o[:, 1::2].double()
    want = no.group_norm(d.reshape(4, 15), torch.ones(15).double(), 1e-3, 3) * 0.4
    torch.testing.assert_close(lr.map_difference(o, 0.7, 1e-3, 0.4, torch.float32).double(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("top,shared", [(1, True), (3, False), (7, True)])
def test_experts_on_weighted_inputs(top, shared):
    g = torch.Generator().manual_seed(top)
    E, H, ff, T = 7, 10, 6, 9
    p = {f"e{e}.{n}": torch.randn(*((H, ff) if n == "down" else (ff, H)), generator=g) for e in range(E) for n in ("gate", "up", "down")}
    p["router"], x = torch.randn(E, H, generator=g), torch.randn(T, H, generator=g)
    c = {"router": {"top": top}, "expert": {"limit": 0.8}}
    s = None
    if shared:
        p.update({"shared." + n: torch.randn(*((H, ff) if n == "down" else (ff, H)), generator=g) for n in ("gate", "up", "down")})
        c["shared"] = {"limit": 1.1}
        s = no.clamped_expert(x, no.sub(p, "shared."), 1.1)
    w, ids = fused_moe.gating_topk_ref(x @ p["router"].T, top, "sigmoid", renorm=False)
    got = fused_moe.fused_experts(x, torch.stack([torch.cat([p[f"e{e}.gate"], p[f"e{e}.up"]]) for e in range(E)]),
                                  torch.stack([p[f"e{e}.down"] for e in range(E)]), w, ids, shared=s, limit=0.8, weight_input=True)
    want = no.mixture(x.double(), {k: t.double() for k, t in p.items()}, c)
    torch.testing.assert_close(got.double(), want, rtol=1e-4, atol=1e-4)
    out = fused_moe.fused_experts(x, torch.stack([torch.cat([p[f"e{e}.gate"], p[f"e{e}.up"]]) for e in range(E)]),
                                  torch.stack([p[f"e{e}.down"] for e in range(E)]), w, ids, shared=s, limit=0.8)
    assert float((out - want).abs().max()) > 1e-2                  # weighting the outputs is something else


def _scan_portions(run, T, sizes):
    """``run(rows, first)`` over consecutive portions of the given sizes (repeated)."""
    out, at, k = [], 0, 0
    while at < T:
        n = min(sizes[k % len(sizes)], T - at)
        out.append(run(slice(at, at + n), at > 0))
        at, k = at + n, k + 1
    return torch.cat(out)


@pytest.mark.parametrize("sizes", [[40], [1], [2, 3], [17, 1]])
def test_recurrences_over_portions(sizes):
    g = torch.Generator().manual_seed(4)
    T, H, G, N, P, D = 40, 6, 2, 5, 3, 4
    one, slot = torch.tensor([1], dtype=torch.int32), torch.tensor([2], dtype=torch.int32)
    xbc, dt = torch.randn(T, H * P + 2 * G * N, generator=g), torch.randn(T, H, generator=g) * 2
    sp = lr.StateSpace(torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g), G)
    state = torch.full((4, H, N, P), 9.0)                          # stale

    def cu(rows):
        return torch.tensor([0, rows.stop - rows.start], dtype=torch.int32)
    got = _scan_portions(lambda r, later: lr.state_space(sp, xbc[r], dt[r], state, cu(r), slot, one * int(later)), T, sizes)
    x, B, C = xbc[:, :H * P].view(T, H, P), xbc[:, H * P:H * P + G * N].view(T, G, N), xbc[:, H * P + G * N:].view(T, G, N)
    y, S = no.state_space(*(t.double() for t in (x, B, C)), no.softplus(dt.double() + sp.dt_bias.double()), sp.A_log.double(),
                          sp.D.double())
    torch.testing.assert_close(got.double().view(T, H, P), y, rtol=1e-4, atol=1e-4)
    torch.testing.assert_close(state[2].double(), S, rtol=1e-4, atol=1e-4)
    assert bool((state[[0, 1, 3]] == 9.0).all())
    q, f, v = torch.randn(T, H * D, generator=g), torch.randn(T, H * D, generator=g) * 3, torch.randn(T, H * P, generator=g)
    fb, low, nw = torch.randn(H * D, generator=g), torch.rand(H * D, generator=g), torch.randn(P, generator=g)
    state = torch.full((4, H, D, P), 9.0)
    got = _scan_portions(lambda r, later: lr.forget_recurrence(q[r], f[r], v[r], fb, low, state, cu(r), slot, one * int(later),
                                                               nw, 1e-4), T, sizes)
    gate = low.double() + (1 - low.double()) * torch.sigmoid(f.double() + fb.double())
    o, S = no.forget_recurrence(no.silu(q.double()).view(T, H, D), gate.view(T, H, D), v.double().view(T, H, P))
    torch.testing.assert_close(got.double(), no.rms_norm(o, nw.double(), 1e-4).reshape(T, -1), rtol=2e-4, atol=2e-4)
    torch.testing.assert_close(state[2].double(), S, rtol=1e-4, atol=1e-4)


def test_wide_queries_are_mixed_scores():
    """Products of wide queries with all key heads side by side are the mixed scores; with two maps each map's own."""
    g = torch.Generator().manual_seed(5)
    H, G, d, T = 6, 3, 4, 2
    spec = va.PrepSpec(H, G, d, 2, 1e-5, None, None, (0, 0), v_heads=G, key_parts=G, part_run=H // G,
                       mix=torch.randn(H, H, generator=g))

    class Meta:
        slot_mapping = torch.arange(T)
        positions = torch.arange(T)
    qkv = torch.randn(T, H * d + G * d + G * 2, generator=g)
    kc, vc = torch.zeros(1, T, 1, G * d), torch.zeros(1, T, G, 2)
    q = va.qkv_prep(spec, qkv, Meta, kc, vc)
    assert tuple(q.shape) == (T, H, G * d)
    k = qkv[:, H * d:H * d + G * d].view(T, G, d)
    s = torch.einsum("thd,jhd->htj", qkv[:, :H * d].view(T, H, d), k[:, torch.arange(H) // (H // G)])
    torch.testing.assert_close(torch.einsum("thd,jd->htj", q, kc[0, :, 0]), torch.einsum("hg,gtj->htj", spec.mix, s))
    two = va.PrepSpec(4, 4, d, 2, 1e-5, None, None, (0, 0), v_heads=2, key_parts=2, q_scale=torch.tensor([1.0, 3.0]))
    qkv, kc, vc = torch.randn(T, 8 * d + 4, generator=g), torch.zeros(1, T, 2, 2 * d), torch.zeros(1, T, 2, 2)
    q = va.qkv_prep(two, qkv, Meta, kc, vc).view(T, 2, 2, 2 * d)
    raw, k = qkv[:, :4 * d].view(T, 2, 2, d), qkv[:, 4 * d:8 * d].view(T, 2, 2, d)
    torch.testing.assert_close(torch.einsum("thmd,jhd->hmtj", q, kc[0]),
                               torch.einsum("thmd,jhmd->hmtj", raw * torch.tensor([1.0, 3.0]).view(2, 1, 1, 1), k))


# ---------------------------------------------------------------- engine
@pytest.mark.parametrize("name", sorted(nc.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_definition(cases, name):
    cfg, w, path = cases(name)
    ids = nc.tokens(cfg, 61, 1)
    want = nc.reference(cfg, w, ids)
    rp = engine(path)
    for sizes in ([61], [1], [2, 3], [2], [16, 1, 15, 17], [40, 1]):
        got = nc.replay(rp, nc.alone("r", nc.cut(ids, sizes)))["r"]
        assert nc.error(got, want) < TOL, sizes
    assert rp.scheduler.pool.num_free_blocks == rp.scheduler.pool.num_blocks - 1
    assert len(rp.scheduler._free_rows) == 4 and not rp.scheduler.running


@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(cases, name):
    cfg, w, path = cases(name)
    ids = {i: nc.tokens(cfg, n, 10 + k) for k, (i, n) in enumerate(
        [("a", 40), ("b", 1), ("c", 23), ("d", 33), ("e", 18), ("f", 29)])}
    queue = {i: nc.cut(t, s) for (i, t), s in zip(ids.items(), ([9, 1, 1], [1], [23], [2], [5, 1], [1, 12]))}
    rp = engine(path, max_tokens=144)                 # room for what lives at once, not for all
    got = nc.replay(rp, nc.interleave(queue, 3))
    for i, t in ids.items():
        assert nc.error(got[i], nc.reference(cfg, w, t)) < TOL, i


def test_an_id_that_comes_back_is_a_new_request(cases):
    cfg, w, path = cases("E")
    rp = engine(path)
    for seed in (1, 2, 3):
        ids = nc.tokens(cfg, 20, seed)
        assert nc.error(nc.replay(rp, nc.alone("r", nc.cut(ids, [7])))["r"], nc.reference(cfg, w, ids)) < TOL


def test_layers_that_share_weights_have_caches_of_their_own(cases):
    cfg, _, path = cases("E")
    run = engine(path).runner
    m = run.model
    assert len(m.layers) == 8 and len(m.unique_layers) == 4
    assert m.layers[3] is m.layers[0] and m.layers[4] is m.layers[2] and m.layers[5] is m.layers[6] is m.layers[1]
    assert len({t.data_ptr() for c in run.kv_caches for t in c}) == sum(len(c) for c in run.kv_caches)
    kinds = [[(tuple(t.shape[1:]), t.dtype) for t in c] for c in run.kv_caches]
    assert kinds[1] == kinds[5] == kinds[6] and kinds[1][2:] == [((4, 96), torch.float32), ((4, 16, 16), torch.float32)]
    assert kinds[2] == [((16, 4, 32), torch.float32), ((16, 4, 32), torch.float32)] and kinds[1][0][0] == (16, 1, 48)
    per_token = 3 * (48 + 2 * 16) + 2 * (4 * 32 + 4 * 32)           # three parallel layers, two with maps
    assert run.kv_bytes_per_block() == 16 * 4 * per_token
    state = 5 * 4 * (3 * (4 * 96 + 4 * 16 * 16) + 2 * (1 + 4 * 32 * 24) + (1 + 2 * 16 * 48))
    assert run.state_bytes() == state


def test_mistakes_would_show(cases):
    """What the comparisons would notice: each mistake, planted in the definition, is far outside the tolerance."""
    cfg, w, _ = cases("A")
    ids = nc.tokens(cfg, 30, 1)
    want = nc.reference(cfg, w, ids)

    def planted(change):
        c, ww = json.loads(json.dumps(cfg)), dict(w)
        change(c, ww)
        return nc.error(no.forward(c, ww, ids), want)
    far = 50 * TOL

    def mixer(c, i):
        return c["layers"][i]["mixer"]
    for off in (-1, 1):
        assert planted(lambda c, x: [mixer(c, i)["left"]["mask"].update(size=11 + off) for i in (0, 4)]) > far
        assert planted(lambda c, x: [mixer(c, i)["q_temp"].update(every=9 + off) for i in (1, 3)]) > far
    for name in ("l0.mix.left.q.b", "l0.mix.left.k.b", "l0.mix.left.v.b", "l0.mix.left.q.norm", "l0.mix.left.talk",
                 "l0.mix.right.conv", "l0.mix.right.conv.b", "l0.mix.right.dt_bias", "l0.mix.right.A_log", "l0.mix.right.D",
                 "l0.mix.right.norm", "l1.mix.q.b", "l1.mix.v.b", "l1.mix.lq1", "l1.mix.lk2", "l2.mix.f.b", "l2.mix.lower",
                 "l2.mix.norm", "l0.norm1", "l1.norm2", "final.norm", "l0.mlp.router"):
        assert planted(lambda c, x: x.update({name: torch.roll(w[name], 1, 0)})) > far, name
    assert planted(lambda c, x: x.update({"l0.mix.left.talk": w["l0.mix.left.talk"].T.contiguous()})) > far
    assert planted(lambda c, x: [mixer(c, i).update(diff=0.4) for i in (1, 3)]) > far
    assert planted(lambda c, x: [mixer(c, i).pop("q_temp") for i in (1, 3)]) > far
    assert planted(lambda c, x: [mixer(c, i)["left"]["rot"].update(dims=8) for i in (0, 4)]) > far
    assert planted(lambda c, x: [mixer(c, i).update(right_scale=0.36) for i in (0, 4)]) > far
    assert planted(lambda c, x: [mixer(c, i)["right"].update(norm_groups=1) for i in (0, 4)]) > far
    assert planted(lambda c, x: c["layers"][0]["mlp"]["expert"].update(limit=1.4)) > far
    assert planted(lambda c, x: c["layers"][2]["mlp"]["shared"].update(limit=0.6)) > far
    assert planted(lambda c, x: c["layers"][0]["mlp"]["router"].update(top=2)) > far
    assert planted(lambda c, x: c["norm"].update(groups=3)) > far
    for attr, wrong in (("softplus", lambda z: torch.relu(z)), ("query_temperature", lambda p, c, e: 1 + c * float(np.log((p + 1) / e + 1))),
                        ("route", lambda z, top: {e: v / sum(kept.values()) for kept in [no_route(z, top)] for e, v in kept.items()})):
        old = getattr(no, attr)
        no_route = no.route
        try:
            setattr(no, attr, wrong)
            assert nc.error(no.forward(cfg, w, ids), want) > far, attr
        finally:
            setattr(no, attr, old)


@pytest.mark.parametrize("decoded", [False, True])
def test_one_far_key_that_stands_out(tmp_path, decoded):
    """A query of the last token meets the first token's key, a hundred positions away, in one of the two maps with a
    score far above all others."""
    cfg = nc.config(40, 32, 2, [nc.maps(2, 1, 8, 8, 1.0, 0.3)])
    w = nc.weights(cfg, seed=3)
    first, last = 5, 9
    ids = [first] + [t if t not in (first, last) else 11 for t in nc.tokens(cfg, 99, 4)] + [last]
    x = no.group_norm(w["embed"].double()[[first, last]], w["l0.norm1"].double(), 1e-5, 2)
    key = x[0] @ w["l0.mix.k"].double().T + w["l0.mix.k.b"].double()
    q = w["l0.mix.q"].double().view(2, 2, 8, 32)
    q[:, 0] += 4.0 * key[:8, None] * (x[1] / (x[1] @ x[1]))[None]
    w["l0.mix.q"] = q.reshape(32, 32).to(torch.bfloat16)
    got = nc.replay(engine(nc.save(tmp_path / "far", cfg, w)), nc.alone("r", nc.cut(ids, [100, 1] if decoded else [101])))["r"]
    want = nc.reference(cfg, w, ids)
    assert nc.error(got, want) < TOL
    other = [(first + 1) % 40] + ids[1:]              # without that key the last position reads something else
    assert nc.error(nc.reference(cfg, w, other)[-1:], want[-1:]) > 0.05


@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("pos", [15, 16, 17, 40])
def test_key_just_inside_and_just_outside_a_window(tmp_path, pos, decoded):
    """Changing the token at the window's far edge changes what the attention side reads, the one before it nothing."""
    size = 16
    cfg = nc.config(40, 32, 1, [nc.parallel((4, 2, 8, 8, 0.05, size, (1e4, 4)), (2, 4, 4, 1, 2, 1), (1.0, 0.0))])
    w = nc.weights(cfg, seed=8)
    path = nc.save(tmp_path / "edge", cfg, w)
    ids = nc.tokens(cfg, pos + 1, 6)
    pieces = nc.cut(ids, [pos, 1] if decoded else [pos + 1])
    base = nc.replay(engine(path), nc.alone("r", pieces))["r"][-1:]
    assert nc.error(base, nc.reference(cfg, w, ids)[-1:]) < TOL
    for j, seen in ((pos - size, False), (pos - size + 1, True)):
        if j < 0:
            continue
        other = list(ids)
        other[j] = (ids[j] + 7) % 40
        got = nc.replay(engine(path), nc.alone("r", nc.cut(other, [pos, 1] if decoded else [pos + 1])))["r"][-1:]
        assert (nc.error(got, base) > 1e-3) if seen else (nc.error(got, base) < 1e-6), j


def test_long_decoding(cases):
    cfg, w, path = cases("A")
    ids = nc.tokens(cfg, 150, 8)
    got = nc.replay(engine(path), nc.alone("r", nc.cut(ids, [4] + [1] * 150)))["r"]
    assert nc.error(got, nc.reference(cfg, w, ids)) < TOL


def test_layer_hook_sees_the_stream_after_every_layer(cases):
    cfg, w, path = cases("E")
    ids = nc.tokens(cfg, 12, 4)
    streams, seen = [], []
    no.forward(cfg, w, ids, collect=streams)
    rp = engine(path)
    m = rp.runner.model
    m.layer_hook = lambda run: seen.append((run, m.stream.clone()))
    nc.replay(rp, nc.alone("r", [ids]))
    assert [r for r, _ in seen] == list(range(len(streams)))
    for (_, a), b in zip(seen, streams):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)


def test_greedy_generation_through_the_engine(cases):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("B")
    prompts = [nc.tokens(cfg, n, 20 + n) for n in (13, 2, 9, 5, 7)]
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=64, max_num_seqs=3, max_num_batched_tokens=6)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p) + list(o.outputs[0].token_ids)
        lg = no.forward(cfg, w, seq)
        assert [int(t) for t in lg[len(p) - 1:-1].argmax(-1)] == seq[len(p):]


def test_checkpoint_errors(cases, tmp_path):
    cfg, w, _ = cases("A")
    short = {k: t for k, t in w.items() if k != "l0.mix.right.conv.b"}
    with pytest.raises(ValueError, match="conv.b"):
        engine(nc.save(tmp_path / "missing", cfg, short))
    with pytest.raises(ValueError, match="unexpected"):       # a layer that uses another's weights has none
        engine(nc.save(tmp_path / "extra", cfg, {**w, "l3.mix.q": w["l1.mix.q"].clone()}))
    for name in ("l0.mix.left.q", "l0.mix.left.talk", "l0.mix.right.in", "l0.mix.right.conv", "l0.mix.right.o", "l1.mix.lq1",
                 "l1.mix.o", "l2.mix.lower", "l2.mix.f", "l2.mix.norm", "l0.mlp.e0.gate", "l0.norm1"):
        wrong = w[name][..., :-1].clone()
        with pytest.raises((ValueError, RuntimeError)):
            engine(nc.save(tmp_path / name, cfg, {**w, name: wrong}))


def test_random_weights_and_parameter_names():
    from vllm_ascend_b200 import LLM, SamplingParams
    llm = LLM(get_model_config("tiny-nevotar"), device="cpu", max_model_len=64, max_num_seqs=2, max_num_batched_tokens=32)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 3
    model = llm.engine.runner.model
    assert [type(L.self_attn) for L in model.layers[::2]] == [ParallelMixer, HGRN2Mixer]
    params = dict(model.named_parameters())
    assert len(params) == len(list(model.named_parameters()))
    before = model.layers[0].self_attn.out_weight.clone()
    model.load_weights((n, t.clone()) for n, t in params.items())
    assert torch.equal(before, model.layers[0].self_attn.out_weight)
    side = model.layers[0].self_attn                              # the mixers' weights are views of the fused ones
    side.right.in_proj.weight.fill_(1.5)
    side.right.out_proj.weight.fill_(2.5)
    assert float(side.in_proj.weight[side.split].max()) == 1.5 and float(side.out_weight[:, side.inner:].min()) == 2.5


def test_states_are_not_cached_by_prefix_or_speculated(cases):
    from vllm_ascend_b200 import LLM
    _, _, path = cases("E")
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=64, max_num_seqs=2, max_num_batched_tokens=32,
              enable_prefix_caching=True)
    assert not llm.cfg.cache.enable_prefix_caching


def test_replay_program(cases, tmp_path, monkeypatch, capsys):
    from vllm_ascend_b200.entrypoints import trace_run
    cfg, w, path = cases("A")
    ids = nc.tokens(cfg, 11, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:8], "want": [7, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[8:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": ids[:3], "want": [0]},
                                     {"id": "a", "tokens": ids[10:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    args = ["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]
    assert trace_run.main(args) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = nc.reference(cfg, w, ids)
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4")).view(2, -1)
    assert nc.error(first, want[[7, 2]]) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    last = torch.from_numpy(np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4")).view(2, -1)
    assert nc.error(last, torch.stack([want[0], want[10]])) < TOL
