"""Vofelix on the CPU engine (fp32) against the plain definitions: configuration, loading, cache and state
handling, scheduling, generation, the replay program."""
import io
import json
import math
import sys

import numpy as np
import pytest
import torch

import vofelix_cases as vc
import vofelix_oracle as vo
from vllm_ascend_b200.config import ModelConfig, get_model_config
from vllm_ascend_b200.engine.replay import TraceReplayer, make_replay_engine
from vllm_ascend_b200.layer_plan import run_order
from vllm_ascend_b200.ops import reference as ref

TOL = 1e-4


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = vc.CONFIGS[name]()
            w = vc.weights(cfg, seed=ord(name))
            made[name] = (cfg, w, vc.save(tmp_path_factory.mktemp("vofelix") / name, cfg, w))
        return made[name]
    return get


def engine(path, max_tokens=256, page=16):
    return TraceReplayer(make_replay_engine(path, "float32", max_tokens, page=page, device="cpu"))


def test_config_reader_and_layer_order():
    cfg = vc.CONFIGS["B"]()
    m = ModelConfig.from_hf_dict(cfg)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_hidden_layers) == ("Vofelix", 128, 264, 5)
    a = m.layer_config(0)
    assert (a.num_attention_heads, a.qk_nope_head_dim, a.qk_rope_head_dim, a.v_head_dim, a.kv_lora_rank,
            a.sliding_window, a.intermediate_size, a.attention_multiplier) == (8, 32, 16, 24, 72, 50, 96, 0.5)
    assert m.layer_config(2).kv_lora_rank == 200 and m.layer_config(2).rope_scaling is None
    d = m.layer_config(3)
    assert (d.linear_num_value_heads, d.linear_num_key_heads, d.linear_key_head_dim, d.linear_value_head_dim,
            d.linear_conv_kernel_dim) == (6, 3, 72, 32, 2)
    assert m.is_hybrid and m.is_linear_layer(1) and not m.is_linear_layer(2)
    assert run_order(5, m.layer_loop) == ([0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4], {4, 7})
    for loop in (None, (0, 5, 1), (2, 3, 4), (0, 2, 2)):
        c = vc.config(10, 8, [vc.delta(1, 1, 8, 8, 2)] * 5, loop)
        assert run_order(5, loop) == vo.layer_order(c)
    for bad in ({"type": "mamba"}, {"mlp": {"kind": "moe", "ff": 8}}):
        c = vc.CONFIGS["A"]()
        c["layers"][0].update(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(c)
    c = vc.CONFIGS["A"]()
    c["loop"]["stop"] = 9
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(c)


@pytest.mark.parametrize("dims,base,scaling", [
    (8, 10000.0, None), (16, 5e5, (8.0, 512, 8.0, 1.0)), (64, 1e4, (3.0, 64, 4.0, 2.0)), (2, 100.0, (2.0, 32, 4.0, 1.0)),
    (12, 1e6, (4.0, 4096, 1.0, 1.0)), (6, 10.0, (16.0, 100000, 32.0, 1.0))])
def test_rotary_table(dims, base, scaling):
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    kw = None if sc is None else {"rope_type": "yarn_interp", "factor": sc["factor"], "beta_fast": sc["fast"],
                                  "original_max_position_embeddings": sc["original"], "beta_slow": sc["slow"]}
    table = ref.build_cos_sin_cache(dims, 700, base, kw)
    x = torch.randn(700, 1, dims, generator=torch.Generator().manual_seed(0))
    got = ref.apply_rope_interleaved(x, torch.arange(700), table, dims)
    for p in (0, 1, 7, 511, 699):
        want = vo.rotate(x[p, 0].double(), p, dims, base, sc)
        torch.testing.assert_close(got[p, 0].double(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("name", sorted(vc.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_definition(cases, name):
    cfg, w, path = cases(name)
    ids = vc.tokens(cfg, 61, 1)
    want = vc.reference(cfg, w, ids)
    rp = engine(path)
    for sizes in ([61], [1], [2, 3], [2], [16, 1, 15, 17], [40, 1]):
        got = vc.replay(rp, vc.alone("r", vc.cut(ids, sizes)))["r"]
        assert vc.error(got, want) < TOL, sizes
    assert rp.scheduler.pool.num_free_blocks == rp.scheduler.pool.num_blocks - 1
    assert len(rp.scheduler._free_rows) == 4 and not rp.scheduler.running


@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(cases, name):
    cfg, w, path = cases(name)
    ids = {i: vc.tokens(cfg, n, 10 + k) for k, (i, n) in enumerate(
        [("a", 40), ("b", 1), ("c", 23), ("d", 33), ("e", 18), ("f", 29)])}
    queue = {i: vc.cut(t, s) for (i, t), s in zip(ids.items(), ([9, 1, 1], [1], [23], [2], [5, 1], [1, 12]))}
    rng = np.random.default_rng(3)
    steps, live, waiting = [], [], list(queue)
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for i in list(live):
            if rng.random() < 0.25 and len(live) > 1:
                continue                              # left out of this step
            piece = queue[i].pop(0)
            step.append((i, piece, not queue[i]))
            if not queue[i]:
                live.remove(i)
        if step:
            steps.append(step)
    rp = engine(path, max_tokens=144)                 # room for what lives at once, not for all
    got = vc.replay(rp, steps)
    for i, t in ids.items():
        assert vc.error(got[i], vc.reference(cfg, w, t)) < TOL, i


def test_state_slot_of_a_finished_request_starts_from_zero(cases):
    cfg, w, path = cases("A")
    rp = engine(path, max_tokens=64)
    a, b = vc.tokens(cfg, 30, 5), vc.tokens(cfg, 2, 6)
    vc.replay(rp, vc.alone("x", [a]))
    got = vc.replay(rp, vc.alone("y", [b[:1], b[1:]]))["y"]
    assert vc.error(got, vc.reference(cfg, w, b)) < TOL
    # the same through a pool with one request's worth of pages
    with pytest.raises(RuntimeError):
        vc.replay(rp, [[("p", a, False), ("q", a, False), ("s", a, False)]])


def test_window_edge_shows_in_the_logits(cases):
    """The tests above would notice a window that is one token off, a sink left out, a pass without the
    embedding, a state that is lost: each mistake, planted in the definition, is far outside the tolerance."""
    cfg, w, _ = cases("A")
    ids = vc.tokens(cfg, 30, 1)
    want = vc.reference(cfg, w, ids)

    def planted(change):
        c, ww = json.loads(json.dumps(cfg)), dict(w)
        change(c, ww)
        return vc.error(vo.forward(c, ww, ids), want)
    far = 100 * TOL
    for off in (-1, 1):
        assert planted(lambda c, x: c["layers"][1]["mixer"]["mask"].update(size=7 + off)) > far
    assert planted(lambda c, x: x.update({"l1.mix.sink": torch.full_like(w["l1.mix.sink"], -1e4)})) > far
    assert planted(lambda c, x: c["loop"].update(times=1)) > far
    assert planted(lambda c, x: x.update({"l0.mix.k.conv": torch.roll(w["l0.mix.k.conv"], 1, -1)})) > far
    assert planted(lambda c, x: x.update({"side.embed": torch.roll(w["side.embed"], 1, -1)})) > far
    assert planted(lambda c, x: c["layers"][1]["mixer"]["rot"].update(base=9000.0)) > far / 10


def test_long_decoding(cases):
    cfg, w, path = cases("D")
    ids = vc.tokens(cfg, 200, 8)
    rp = engine(path)
    got = vc.replay(rp, vc.alone("r", vc.cut(ids, [4] + [1] * 200)))["r"]
    assert vc.error(got, vc.reference(cfg, w, ids)) < TOL


def test_layer_hook_sees_the_stream_after_every_run(cases):
    cfg, w, path = cases("A")
    ids = vc.tokens(cfg, 12, 4)
    streams = []
    vo.forward(cfg, w, ids, collect=streams)
    rp = engine(path)
    m, seen = rp.runner.model, []
    m.layer_hook = seen.append
    vc.replay(rp, vc.alone("r", [ids]))
    assert seen == list(range(len(streams))) == list(range(len(m.layers)))


def greedy(cfg, w, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(vo.forward(cfg, w, seq)[-1].argmax()))
    return seq[len(prompt):]


def test_greedy_generation_through_the_engine(cases):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("A")
    prompts = [vc.tokens(cfg, n, 20 + n) for n in (13, 2, 9, 5, 7)]
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=64, max_num_seqs=3, max_num_batched_tokens=6)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == greedy(cfg, w, p, 5)


def test_checkpoint_errors(cases, tmp_path):
    cfg, w, _ = cases("A")
    short = {k: t for k, t in w.items() if k != "l1.mix.sink"}
    with pytest.raises(ValueError, match="sink"):
        engine(vc.save(tmp_path / "missing", cfg, short))
    with pytest.raises(ValueError, match="unexpected"):
        engine(vc.save(tmp_path / "extra", cfg, {**w, "l0.mix.zz": w["embed"].clone()}))
    with pytest.raises(ValueError, match="shape"):
        engine(vc.save(tmp_path / "shape", cfg, {**w, "l0.mix.norm": w["l0.mix.norm"][:1]}))


def test_random_weights_and_parameter_names(cases):
    m = get_model_config("tiny-vofelix")
    from vllm_ascend_b200 import LLM, SamplingParams
    llm = LLM(m, device="cpu", max_model_len=64, max_num_seqs=2, max_num_batched_tokens=32)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 3
    model = llm.engine.runner.model
    params = dict(model.named_parameters())
    assert len(params) == len(list(model.named_parameters()))
    model.load_weights((n, t.clone()) for n, t in params.items())


def test_replay_program(cases, tmp_path, monkeypatch, capsys):
    from vllm_ascend_b200.entrypoints import trace_run
    cfg, w, path = cases("A")
    ids = vc.tokens(cfg, 11, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:8], "want": [7, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[8:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": ids[:3], "want": [0]},
                                     {"id": "a", "tokens": ids[10:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    args = ["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]
    assert trace_run.main(args) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = vc.reference(cfg, w, ids)
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4")).view(2, -1)
    assert vc.error(first, want[[7, 2]]) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    last = torch.from_numpy(np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4")).view(2, -1)
    assert vc.error(last, torch.stack([want[0], want[10]])) < TOL


def test_softplus_and_gates():
    from vllm_ascend_b200.ops.linear_attn import delta_gates_ref
    ba = torch.tensor([[0.3, -2.0, 25.0, -40.0]])
    A, dt = torch.tensor([0.5, -1.0]), torch.tensor([0.1, 0.2])
    beta, g = delta_gates_ref(ba, A, dt)
    want = [-math.exp(0.5) * float(vo.softplus(torch.tensor(25.1, dtype=torch.float64))),
            -math.exp(-1.0) * math.log1p(math.exp(-39.8))]
    np.testing.assert_allclose(g[0].numpy(), want, rtol=1e-5)
    np.testing.assert_allclose(beta[0].numpy(), [1 / (1 + math.exp(-0.3)), 1 / (1 + math.exp(2.0))], rtol=1e-6)
