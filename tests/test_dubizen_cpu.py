"""Dubizen on the CPU engine (fp32) against the plain definitions: configuration, loading, cache handling,
scheduling, generation, the replay program."""
import io
import json
import sys

import numpy as np
import pytest
import torch

import dubizen_cases as dc
import dubizen_oracle as do
from vllm_ascend_b200.config import ModelConfig, get_model_config
from vllm_ascend_b200.engine.replay import TraceReplayer, make_replay_engine
from vllm_ascend_b200.models.layers import PlainMLP
from vllm_ascend_b200.models.transformer import SparseMoeBlock
from vllm_ascend_b200.ops import fused_moe
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, stream_norm

TOL = 1e-4


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = dc.CONFIGS[name]()
            w = dc.weights(cfg, seed=ord(name))
            made[name] = (cfg, w, dc.save(tmp_path_factory.mktemp("dubizen") / name, cfg, w))
        return made[name]
    return get


def engine(path, max_tokens=256, page=16):
    return TraceReplayer(make_replay_engine(path, "float32", max_tokens, page=page, device="cpu"))


def test_config_reader():
    m = ModelConfig.from_hf_dict(dc.CONFIGS["B"]())
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_hidden_layers) == ("Dubizen", 128, 264, 4)
    assert (m.norm_type, m.norm_bias, m.pre_norm, m.sandwich_norm, m.residual_multiplier, m.tie_word_embeddings) \
        == ("layer", False, False, True, 0.4, True)
    a, b, c, d = (m.layer_config(i) for i in range(4))
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.sliding_window, a.attn_distance_max,
            a.attention_multiplier, a.rotary_dims) == (6, 2, 40, 24, 70, 100, 0.15, 0)
    assert a.qk_norm and not a.qk_norm_full and a.attention_bias and a.attention_out_bias and not a.attention_sink
    assert (a.num_experts, a.num_experts_per_tok, a.moe_intermediate_size, a.n_group, a.topk_group, a.moe_group_score,
            a.routed_scaling_factor, a.shared_expert_intermediate_size) == (24, 5, 72, 6, 3, "max", 3.0, 48)
    assert a.e_score_correction_bias and a.shared_expert_gate and a.router_fp32 and a.scoring_func == "softmax"
    assert (b.q_lora_rank, b.kv_lora_rank, b.qk_nope_head_dim, b.qk_rope_head_dim, b.v_head_dim, b.rope_theta,
            b.latent_kv_from) == (96, 72, 24, 16, 40, 5e5, None)
    assert (b.intermediate_size, b.mlp_gated, b.hidden_act, b.is_moe) == (112, False, "gelu", False)
    assert b.rope_half_split and not b.attention_sink and b.sliding_window is None
    assert (c.latent_kv_from, c.q_lora_rank, c.n_group) == (1, 48, 4) and not m.layer_plan[3]["mlp"]
    assert m.is_moe and [m.is_moe_layer(i) for i in range(4)] == [True, False, True, False]
    assert not m.keeps_sequence_state and not m.is_hybrid
    plain = ModelConfig.from_hf_dict(dc.CONFIGS["C"]()).layer_config(0)
    assert (plain.n_group, plain.topk_group, plain.shared_expert_intermediate_size) == (1, 1, 0)


@pytest.mark.parametrize("layer,change", [
    (2, {"mixer": {"kv_from": 0}}),            # no latents there
    (2, {"mixer": {"kv_from": 2}}),            # its own
    (2, {"mixer": {"kv_from": 3}}),            # a later layer
    (2, {"mixer": {"kv_rank": 80}}),           # latents of another size
    (2, {"mixer": {"rot": {"base": 1e4, "dims": 16}}}),
    (1, {"mixer": {"rot": {"base": 1e4, "dims": 8}}}),
    (0, {"mixer": {"kv_heads": 4}}),
    (0, {"type": "delta"}),
    (0, {"mlp": {"kind": "moe2"}}),
    (0, {"mlp": {"router": {"experts": 24, "top": 5, "groups": {"count": 5, "keep": 1}}}}),
    (0, {"mlp": {"router": {"experts": 24, "top": 5, "groups": {"count": 6, "keep": 1}}}}),
])
def test_configurations_that_do_not_fit_are_refused(layer, change):
    c = dc.CONFIGS["B"]()
    for k, v in change.items():
        if isinstance(v, dict):
            c["layers"][layer][k].update(v)
        else:
            c["layers"][layer][k] = v
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(c)


def test_stream_norm_definition_with_a_multiplier_and_no_bias():
    g = torch.Generator().manual_seed(1)
    r, y, w = torch.randn(5, 12, generator=g), torch.randn(5, 12, generator=g) + 3, torch.randn(12, generator=g)
    want = r.double() + 0.3 * do.output_norm(y.double(), w.double(), 1e-3)
    x = stream_norm(r, y, NormSpec("layer", w), PLAIN, 1e-3, torch.float32, post_scale=0.3)
    torch.testing.assert_close(r.double(), want, rtol=1e-5, atol=1e-5)
    assert torch.equal(x, r)


@pytest.mark.parametrize("groups,top", [((4, 2), 3), ((1, 1), 5), ((6, 1), 2), ((12, 3), 3), ((3, 3), 12)])
def test_router_definition(groups, top):
    g = torch.Generator().manual_seed(7)
    z, corr = torch.randn(40, 12, generator=g) * 2, torch.randn(12, generator=g) * 0.5 - 0.6
    w, ids = fused_moe.gating_topk_ref(z, top, "softmax", True, *groups, corr, 2.5, "max")
    c = {"experts": 12, "top": top, "scale": 2.5, "groups": dict(zip(("count", "keep"), groups))}
    for t in range(40):
        want = do.route(z[t].double(), corr, c)
        got = {int(e): float(v) for e, v in zip(ids[t], w[t])}
        assert got.keys() == want.keys()
        assert all(abs(got[e] - want[e]) < 1e-5 for e in want)
    with pytest.raises(ValueError):
        fused_moe.gating_topk_ref(z, 2, n_group=2, group_score="mean")


def test_expert_groups_by_best_or_by_best_two():
    """A group with one strong expert against a group with two good ones: the two scores disagree."""
    z = torch.log(torch.tensor([[0.4, 0.01, 0.3, 0.29]]))
    zero = torch.zeros(4)
    best = [fused_moe.gating_topk_ref(z, 1, n_group=2, topk_group=1, bias=zero, group_score=s)[1].tolist()
            for s in ("max", "top2", None)]
    assert best == [[[0]], [[2]], [[2]]]


@pytest.mark.parametrize("name", sorted(dc.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_definition(cases, name):
    cfg, w, path = cases(name)
    ids = dc.tokens(cfg, 61, 1)
    want = dc.reference(cfg, w, ids)
    rp = engine(path)
    for sizes in ([61], [1], [2, 3], [2], [16, 1, 15, 17], [40, 1]):
        got = dc.replay(rp, dc.alone("r", dc.cut(ids, sizes)))["r"]
        assert dc.error(got, want) < TOL, sizes
    assert rp.scheduler.pool.num_free_blocks == rp.scheduler.pool.num_blocks - 1
    assert len(rp.scheduler._free_rows) == 4 and not rp.scheduler.running


@pytest.mark.parametrize("name", ["A", "B", "E"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(cases, name):
    cfg, w, path = cases(name)
    ids = {i: dc.tokens(cfg, n, 10 + k) for k, (i, n) in enumerate(
        [("a", 40), ("b", 1), ("c", 23), ("d", 33), ("e", 18), ("f", 29)])}
    queue = {i: dc.cut(t, s) for (i, t), s in zip(ids.items(), ([9, 1, 1], [1], [23], [2], [5, 1], [1, 12]))}
    rp = engine(path, max_tokens=144)                 # room for what lives at once, not for all
    got = dc.replay(rp, dc.interleave(queue, 3))
    for i, t in ids.items():
        assert dc.error(got[i], dc.reference(cfg, w, t)) < TOL, i


def test_layers_share_one_cache(cases):
    _, _, path = cases("E")
    run = engine(path).runner
    shared = [tuple(t.data_ptr() for t in c) for c in run.kv_caches]
    assert shared[3] == shared[0] and shared[4] == shared[2] and len(set(shared)) == 3
    # 4 bytes of: latents and rotated keys twice, keys and values once
    assert run.kv_bytes_per_block() == 16 * 4 * ((40 + 8) + 2 * (32 + 32) + (104 + 16))


def test_mistakes_would_show(cases):
    """What the comparisons would notice: each mistake, planted in the definition, is far outside the tolerance."""
    cfg, w, _ = cases("A")
    ids = dc.tokens(cfg, 30, 1)
    want = dc.reference(cfg, w, ids)

    def planted(change):
        c, ww = json.loads(json.dumps(cfg)), dict(w)
        change(c, ww)
        return dc.error(do.forward(c, ww, ids), want)
    far = 50 * TOL
    for off in (-1, 1):
        for layer, size in ((1, 11), (3, 5)):
            assert planted(lambda c, x: c["layers"][layer]["mixer"]["mask"].update(size=size + off)) > far
    for name in ("l1.mix.rel", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l1.mix.o.b", "l1.mix.k.norm", "l0.mix.dq.norm",
                 "l0.mix.dkv.norm", "l0.mlp.correction", "l0.norm1", "l2.norm2"):
        assert planted(lambda c, x: x.update({name: torch.roll(w[name], 1, 0)})) > far, name
    assert planted(lambda c, x: c["layers"][1]["mixer"].update(bias_max=12)) > far
    assert planted(lambda c, x: c["layers"][0]["mixer"]["rot"].update(base=9e3)) > far
    assert planted(lambda c, x: c["layers"][0]["mixer"].update(scale=0.31)) > far
    assert planted(lambda c, x: c["layers"][0]["mlp"]["router"].update(scale=1.6)) > far
    assert planted(lambda c, x: c["layers"][0]["mlp"]["router"]["groups"].update(keep=3)) > far
    assert planted(lambda c, x: c["layers"][0]["mlp"]["router"].update(top=2)) > far
    assert planted(lambda c, x: c["layers"][3]["mlp"].pop("shared")) > far
    assert planted(lambda c, x: x.update({"l0.mlp.shared.sg": -w["l0.mlp.shared.sg"]})) > far
    assert planted(lambda c, x: c.update(residual_mult=0.61)) > far
    assert planted(lambda c, x: c["norm"].update(eps=1e-2)) > far
    # rotary pairs (2i, 2i + 1) instead of (i, i + half)
    old = do.rotate_halves
    try:
        from vofelix_oracle import rotate
        do.rotate_halves = lambda x, pos, dims, base: rotate(x, pos, dims, base, None)
        assert dc.error(do.forward(cfg, w, ids), want) > far
    finally:
        do.rotate_halves = old


@pytest.mark.parametrize("decoded", [False, True])
def test_one_far_key_that_stands_out(tmp_path, decoded):
    """The last token's query meets the first token's key with a score far above all others, a hundred positions
    apart: latent attention finds it, also through the layer that shares the latents."""
    cfg = dc.config(40, 32, [dc.latent(2, 8, 4, 8, 16, 24, 1.0), dc.latent(2, 8, 4, 8, 16, 24, 1.0, kv_from=0)], mult=0.6)
    w = dc.weights(cfg, seed=3)
    first, last = 5, 9
    ids = [first] + [t if t not in (first, last) else 11 for t in dc.tokens(cfg, 99, 4)] + [last]
    # unrotated key of the first token along its own latent; the last token's query along that key
    x = w["embed"].double()
    lat = do.rms_norm(x[first] @ w["l0.mix.dkv"][:16].double().T, w["l0.mix.dkv.norm"].double(), 1e-5)
    cq = do.rms_norm(x[last] @ w["l0.mix.dq"].double().T, w["l0.mix.dq.norm"].double(), 1e-5)
    uq = w["l0.mix.uq"].double().view(2, 12, 24)
    key = w["l0.mix.uk"].double().view(2, 8, 16) @ lat
    uq[:, :8] += 1.5 * key[:, :, None] * (cq / (cq @ cq))[None, None]
    w["l0.mix.uq"] = uq.reshape(24, 24).to(torch.bfloat16)
    got = dc.replay(engine(dc.save(tmp_path / "far", cfg, w)), dc.alone("r", dc.cut(ids, [100, 1] if decoded else [101])))["r"]
    want = dc.reference(cfg, w, ids)
    assert dc.error(got, want) < TOL
    other = [(first + 1) % 40] + ids[1:]              # without that key the last position reads something else
    assert dc.error(dc.reference(cfg, w, other)[-1:], want[-1:]) > 0.05


def test_long_decoding(cases):
    cfg, w, path = cases("A")
    ids = dc.tokens(cfg, 150, 8)
    got = dc.replay(engine(path), dc.alone("r", dc.cut(ids, [4] + [1] * 150)))["r"]
    assert dc.error(got, dc.reference(cfg, w, ids)) < TOL


def test_layer_hook_sees_the_stream_after_every_layer(cases):
    cfg, w, path = cases("B")
    ids = dc.tokens(cfg, 12, 4)
    streams, seen = [], []
    do.forward(cfg, w, ids, collect=streams)
    rp = engine(path)
    m = rp.runner.model
    m.layer_hook = lambda run: seen.append((run, m.stream.clone()))
    got = dc.replay(rp, dc.alone("r", [ids]))["r"]
    assert [r for r, _ in seen] == list(range(len(streams)))
    for (_, a), b in zip(seen, streams):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)
    assert dc.error(got, dc.reference(cfg, w, ids)) < TOL


@pytest.mark.parametrize("buckets", [2, 40])
def test_bias_table_of_any_size(tmp_path, buckets):
    cfg = dc.CONFIGS["B"]()
    w = dc.weights(cfg, seed=4, buckets=buckets)
    ids = dc.tokens(cfg, 80, 3)
    got = dc.replay(engine(dc.save(tmp_path / "m", cfg, w)), dc.alone("r", dc.cut(ids, [50, 1])))["r"]
    assert dc.error(got, dc.reference(cfg, w, ids)) < TOL


def test_greedy_generation_through_the_engine(cases):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("B")
    prompts = [dc.tokens(cfg, n, 20 + n) for n in (13, 2, 9, 5, 7)]
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=64, max_num_seqs=3, max_num_batched_tokens=6)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p) + list(o.outputs[0].token_ids)
        lg = do.forward(cfg, w, seq)
        assert [int(t) for t in lg[len(p) - 1:-1].argmax(-1)] == seq[len(p):]


def test_prefix_caching_keeps_shared_latents(cases):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("E")
    head = dc.tokens(cfg, 40, 2)
    prompts = [head + dc.tokens(cfg, n, n) for n in (5, 9)]
    sp = SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True)
    kw = dict(dtype="float32", device="cpu", max_model_len=96, max_num_seqs=2, max_num_batched_tokens=64, block_size=16)
    plain, cached = LLM(path, **kw), LLM(path, enable_prefix_caching=True, **kw)
    for p in prompts:
        assert cached.generate([p], sp)[0].outputs[0].token_ids == plain.generate([p], sp)[0].outputs[0].token_ids


def test_checkpoint_errors(cases, tmp_path):
    cfg, w, _ = cases("A")
    short = {k: t for k, t in w.items() if k != "l0.mlp.e4.up"}
    with pytest.raises(ValueError, match="e4.up"):
        engine(dc.save(tmp_path / "missing", cfg, short))
    with pytest.raises(ValueError, match="unexpected"):
        engine(dc.save(tmp_path / "extra", cfg, {**w, "l2.mix.dkv": w["l0.mix.dkv"].clone()}))
    for name in ("l0.mix.dkv", "l0.mix.uq", "l0.mlp.e0.gate", "l0.mlp.correction", "l1.mix.q.norm", "l1.mix.o.b", "l1.mix.rel"):
        wrong = w[name][..., :-1].clone()
        with pytest.raises((ValueError, RuntimeError)):
            engine(dc.save(tmp_path / name, cfg, {**w, name: wrong}))


def test_random_weights_and_parameter_names():
    from vllm_ascend_b200 import LLM, SamplingParams
    llm = LLM(get_model_config("tiny-dubizen"), device="cpu", max_model_len=64, max_num_seqs=2, max_num_batched_tokens=32)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 3
    model = llm.engine.runner.model
    kinds = [type(L.mlp) for L in model.layers]
    assert kinds == [PlainMLP, SparseMoeBlock, type(None)]
    params = dict(model.named_parameters())
    assert len(params) == len(list(model.named_parameters()))
    held = {t.data_ptr() for t in params.values()}
    for L in model.layers:                     # every weight the forward pass reads is among them
        a = L.self_attn
        if hasattr(a, "down_proj"):
            assert a.q_a_proj.weight.data_ptr() == a.down_proj.weight.data_ptr() and a.q_a_proj.weight.data_ptr() in held
    model.load_weights((n, t.clone()) for n, t in params.items())


def test_replay_program(cases, tmp_path, monkeypatch, capsys):
    from vllm_ascend_b200.entrypoints import trace_run
    cfg, w, path = cases("A")
    ids = dc.tokens(cfg, 11, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:8], "want": [7, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[8:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": ids[:3], "want": [0]},
                                     {"id": "a", "tokens": ids[10:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    args = ["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]
    assert trace_run.main(args) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = dc.reference(cfg, w, ids)
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4")).view(2, -1)
    assert dc.error(first, want[[7, 2]]) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    last = torch.from_numpy(np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4")).view(2, -1)
    assert dc.error(last, torch.stack([want[0], want[10]])) < TOL
