"""Pegopel on the CPU engine (fp32) against the plain definitions: configuration, loading, cache and state
handling, scheduling, generation, the replay program."""
import io
import json
import sys

import numpy as np
import pytest
import torch

import pegopel_cases as pc
import pegopel_oracle as po
from vllm_ascend_b200.attention import variant as va
from vllm_ascend_b200.config import ModelConfig, get_model_config
from vllm_ascend_b200.engine.replay import TraceReplayer, make_replay_engine
from vllm_ascend_b200.layer_plan import run_order
from vllm_ascend_b200.ops.stream import PLAIN, NormSpec, StreamMix, stream_mix

TOL = 1e-4


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = pc.CONFIGS[name]()
            w = pc.weights(cfg, seed=ord(name))
            made[name] = (cfg, w, pc.save(tmp_path_factory.mktemp("pegopel") / name, cfg, w))
        return made[name]
    return get


def engine(path, max_tokens=256, page=16):
    return TraceReplayer(make_replay_engine(path, "float32", max_tokens, page=page, device="cpu"))


def test_config_reader_and_layer_order():
    cfg = pc.CONFIGS["B"]()
    m = ModelConfig.from_hf_dict(cfg)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.num_hidden_layers) == ("Pegopel", 128, 264, 4)
    assert (m.residual_streams, m.learned_positions, m.tie_word_embeddings, m.layer_loop) == (2, 400, True, (1, 4, 2))
    a, b = m.layer_config(0), m.layer_config(1)
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.sliding_window, a.attn_keep_first,
            a.attention_multiplier, a.attn_softcap, a.rotary_dims, a.rope_theta, a.intermediate_size) \
        == (8, 2, 32, 32, 50, 9, 0.3, 8.0, 24, 5e5, 96)
    assert a.attn_values_from_keys and a.attn_head_gate and a.attn_sink_value == 0.0 and not a.attn_conv_kernel
    assert (b.attn_conv_kernel, b.attn_distance_max, b.head_dim, b.v_head_dim, b.sliding_window) == (4, 64, 40, 24, 70)
    assert b.attention_sink and not b.attn_head_gate and b.rotary_dims == 0 and b.attn_softcap is None
    assert m.layer_config(3).rope_scaling is None and a.rope_scaling["factor"] == 8.0
    assert m.keeps_sequence_state and not m.is_hybrid and not any(m.is_linear_layer(i) for i in range(4))
    only = ModelConfig.from_hf_dict(pc.config(9, 8, [pc.gated(1, 1, 8, 4, 1, 1.0, 2.0, 4)], 2))
    assert not only.keeps_sequence_state
    for loop in (None, (0, 5, 1), (2, 3, 4), (0, 2, 2)):
        c = pc.config(10, 8, [pc.biased(1, 1, 8, 8, 2, 4, 20, 1.0)] * 5, 2, loop)
        assert run_order(5, loop)[0] == po.layer_order(c)
    for change in (dict(type="delta"), dict(mlp={"kind": "moe", "ff": 8})):
        c = pc.CONFIGS["A"]()
        c["layers"][0].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(c)
    for layer, change in ((0, dict(kv_heads=4)), (1, dict(vdim=9)), (1, dict(rot={"base": 1e4, "dims": 12}))):
        c = pc.CONFIGS["A"]()
        c["layers"][layer]["mixer"].update(change)
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(c)


@pytest.mark.parametrize("rows,largest", [(12, 50), (32, 128), (2, 9), (16, 4000), (64, 33), (6, 6)])
def test_distance_table_reaches_every_bucket(rows, largest):
    rel = torch.randn(rows, 3)
    t = va.distance_table(rel, largest, 100000)
    for n in range(2 * largest + 10):
        assert torch.equal(t[:, min(n, t.shape[1] - 1)], rel[po.distance_bucket(n, rows, largest)]), n
    short = va.distance_table(rel, largest, 5)          # a window of 5 never asks for more
    assert torch.equal(short[:, :5], t[:, :short.shape[1]][:, :5]) and short.shape[1] <= 5


def test_stream_mix_definition():
    g = torch.Generator().manual_seed(1)
    S, T, W = 3, 5, 8
    st = torch.randn(S, T, W, generator=g).double()
    y, wn = torch.randn(T, W, generator=g), torch.randn(W, generator=g)
    a, b = (StreamMix(torch.randn(S, generator=g), torch.randn(S, generator=g), torch.randn(S, S, generator=g)) for _ in "ab")
    r = st.transpose(0, 1).float().contiguous()
    x = stream_mix(r, y, PLAIN, a, b, NormSpec("rms", wn), 1e-5, torch.float32)
    new = po.mix_streams(st.float().double(), y.double(), {"mix": a.mix.double(), "out": a.write.double()})
    torch.testing.assert_close(r.double(), new.transpose(0, 1), rtol=1e-5, atol=1e-5)
    u = torch.einsum("s,stw->tw", b.read.double(), new)
    torch.testing.assert_close(x.double(), po.rms_norm(u, wn.double(), 1e-5), rtol=1e-4, atol=1e-4)
    with pytest.raises(IndexError):
        stream_mix(r, None, None, None, b, NormSpec("rms", wn), 1e-5, torch.float32, embed=y,
                   pos_table=torch.zeros(4, W), positions=torch.arange(T))


@pytest.mark.parametrize("name", sorted(pc.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_definition(cases, name):
    cfg, w, path = cases(name)
    ids = pc.tokens(cfg, 61, 1)
    want = pc.reference(cfg, w, ids)
    rp = engine(path)
    for sizes in ([61], [1], [2, 3], [2], [16, 1, 15, 17], [40, 1]):
        got = pc.replay(rp, pc.alone("r", pc.cut(ids, sizes)))["r"]
        assert pc.error(got, want) < TOL, sizes
    assert rp.scheduler.pool.num_free_blocks == rp.scheduler.pool.num_blocks - 1
    assert len(rp.scheduler._free_rows) == 4 and not rp.scheduler.running


@pytest.mark.parametrize("name", ["A", "B"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(cases, name):
    cfg, w, path = cases(name)
    ids = {i: pc.tokens(cfg, n, 10 + k) for k, (i, n) in enumerate(
        [("a", 40), ("b", 1), ("c", 23), ("d", 33), ("e", 18), ("f", 29)])}
    queue = {i: pc.cut(t, s) for (i, t), s in zip(ids.items(), ([9, 1, 1], [1], [23], [2], [5, 1], [1, 12]))}
    rp = engine(path, max_tokens=144)                 # room for what lives at once, not for all
    got = pc.replay(rp, pc.interleave(queue, 3))
    for i, t in ids.items():
        assert pc.error(got[i], pc.reference(cfg, w, t)) < TOL, i


def test_state_slot_of_a_finished_request_starts_from_zero(cases):
    cfg, w, path = cases("A")
    rp = engine(path, max_tokens=64)
    a, b = pc.tokens(cfg, 30, 5), pc.tokens(cfg, 3, 6)
    pc.replay(rp, pc.alone("x", [a]))
    got = pc.replay(rp, pc.alone("y", [b[:1], b[1:]]))["y"]
    assert pc.error(got, pc.reference(cfg, w, b)) < TOL


def test_mistakes_would_show(cases):
    """What the comparisons would notice: each mistake, planted in the definition, is far outside the tolerance."""
    cfg, w, _ = cases("A")
    ids = pc.tokens(cfg, 30, 1)
    want = pc.reference(cfg, w, ids)

    def planted(change):
        c, ww = json.loads(json.dumps(cfg)), dict(w)
        change(c, ww)
        return pc.error(po.forward(c, ww, ids), want)
    far = 50 * TOL
    for off in (-1, 1):
        for layer, size in ((0, 11), (1, 7), (2, 5)):
            assert planted(lambda c, x: c["layers"][layer]["mixer"]["mask"].update(size=size + off)) > far
        assert planted(lambda c, x: c["layers"][1]["mixer"]["mask"].update(keep_first=2 + off)) > far
    assert planted(lambda c, x: x.update({"l0.mix.sink": torch.full_like(w["l0.mix.sink"], -1e4)})) > far
    assert planted(lambda c, x: x.update({"l0.mix.rel": torch.roll(w["l0.mix.rel"], 1, 0)})) > far
    assert planted(lambda c, x: c["layers"][0]["mixer"].update(bias_max=12)) > far
    assert planted(lambda c, x: c["layers"][1]["mixer"].update(softcap=9.0)) > far
    assert planted(lambda c, x: c["layers"][1]["mixer"]["rot"].update(dims=4)) > far
    assert planted(lambda c, x: x.update({"l1.mix.g": -w["l1.mix.g"]})) > far
    assert planted(lambda c, x: x.update({"l1.mix.k.norm": torch.roll(w["l1.mix.k.norm"], 1)})) > far
    assert planted(lambda c, x: c["loop"].update(times=1)) > far
    assert planted(lambda c, x: x.update({"l2.mix.k.conv": torch.roll(w["l2.mix.k.conv"], 1, -1)})) > far
    assert planted(lambda c, x: x.update({"l0.hc1.mix": w["l0.hc1.mix"].T.contiguous()})) > far
    assert planted(lambda c, x: x.update({"pos": torch.roll(w["pos"], 1, 0)})) > far


def test_long_decoding(cases):
    cfg, w, path = cases("A")
    ids = pc.tokens(cfg, 150, 8)
    got = pc.replay(engine(path), pc.alone("r", pc.cut(ids, [4] + [1] * 150)))["r"]
    assert pc.error(got, pc.reference(cfg, w, ids)) < TOL


def test_layer_hook_sees_the_sum_of_the_streams_after_every_run(cases):
    cfg, w, path = cases("A")
    ids = pc.tokens(cfg, 12, 4)
    streams, seen = [], []
    po.forward(cfg, w, ids, collect=streams)
    rp = engine(path)
    m = rp.runner.model
    m.layer_hook = lambda run: seen.append((run, m.stream.clone()))
    got = pc.replay(rp, pc.alone("r", [ids]))["r"]
    assert [r for r, _ in seen] == list(range(len(streams)))
    for (_, a), b in zip(seen, streams):
        torch.testing.assert_close(a.double(), b, rtol=1e-4, atol=1e-4)
    assert pc.error(got, pc.reference(cfg, w, ids)) < TOL


def test_positions_end_with_their_table(cases, tmp_path):
    cfg = dict(pc.CONFIGS["D"](), max_positions=20)
    w = pc.weights(cfg, seed=2)
    rp = engine(pc.save(tmp_path / "short", cfg, w), max_tokens=64)
    ids = pc.tokens(cfg, 21, 3)
    got = pc.replay(rp, [[("r", ids[:20], False)]])["r"]
    assert pc.error(got, pc.reference(cfg, w, ids[:20])) < TOL
    with pytest.raises(ValueError):
        pc.replay(rp, [[("r", ids[20:], False)]])


def test_one_stream_without_weights_is_a_plain_residual_sum(tmp_path):
    cfg = pc.CONFIGS["C"]()
    w = pc.weights(cfg, seed=3)
    one = {k: (torch.ones_like(t) if ".hc" in k else t) for k, t in w.items()}
    ids = pc.tokens(cfg, 20, 3)
    bare = {k: t for k, t in w.items() if ".hc" not in k}
    del cfg["streams"]
    rp = engine(pc.save(tmp_path / "bare", cfg, bare))
    got = pc.replay(rp, pc.alone("r", [ids]))["r"]
    assert pc.error(got, po.forward(dict(cfg, streams=1), one, ids)) < TOL


@pytest.mark.parametrize("buckets", [2, 40])
def test_bias_table_of_any_size(tmp_path, buckets):
    cfg = pc.CONFIGS["B"]()
    w = pc.weights(cfg, seed=4, buckets=buckets)
    ids = pc.tokens(cfg, 80, 3)
    got = pc.replay(engine(pc.save(tmp_path / "m", cfg, w)), pc.alone("r", pc.cut(ids, [50, 1])))["r"]
    assert pc.error(got, pc.reference(cfg, w, ids)) < TOL


def test_greedy_generation_through_the_engine(cases):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("A")
    prompts = [pc.tokens(cfg, n, 20 + n) for n in (13, 2, 9, 5, 7)]
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=64, max_num_seqs=3, max_num_batched_tokens=6)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p) + list(o.outputs[0].token_ids)
        lg = po.forward(cfg, w, seq)
        assert [int(t) for t in lg[len(p) - 1:-1].argmax(-1)] == seq[len(p):]


def test_checkpoint_errors(cases, tmp_path):
    cfg, w, _ = cases("A")
    short = {k: t for k, t in w.items() if k != "l0.hc2.out"}
    with pytest.raises(ValueError, match="hc2.out"):
        engine(pc.save(tmp_path / "missing", cfg, short))
    with pytest.raises(ValueError, match="unexpected"):
        engine(pc.save(tmp_path / "extra", cfg, {**w, "l1.mix.v": w["embed"].clone()}))
    with pytest.raises(ValueError, match="shape"):
        engine(pc.save(tmp_path / "shape", cfg, {**w, "l0.mix.sink": w["l0.mix.sink"][:1].clone()}))
    with pytest.raises(ValueError, match="shape"):
        engine(pc.save(tmp_path / "rel", cfg, {**w, "l0.mix.rel": w["l0.mix.rel"][:, :1].clone()}))


def test_random_weights_and_parameter_names():
    from vllm_ascend_b200 import LLM, SamplingParams
    llm = LLM(get_model_config("tiny-pegopel"), device="cpu", max_model_len=64, max_num_seqs=2, max_num_batched_tokens=32)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 3
    model = llm.engine.runner.model
    params = dict(model.named_parameters())
    assert len(params) == len(list(model.named_parameters()))
    model.load_weights((n, t.clone()) for n, t in params.items())
    with pytest.raises(ValueError, match="speculative"):
        LLM(get_model_config("tiny-pegopel"), device="cpu", max_model_len=64,
            speculative_config={"method": "ngram", "num_speculative_tokens": 2})


def test_replay_program(cases, tmp_path, monkeypatch, capsys):
    from vllm_ascend_b200.entrypoints import trace_run
    cfg, w, path = cases("A")
    ids = pc.tokens(cfg, 11, 2)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:8], "want": [7, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ids[8:10], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": ids[:3], "want": [0]},
                                     {"id": "a", "tokens": ids[10:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    args = ["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]
    assert trace_run.main(args) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = pc.reference(cfg, w, ids)
    first = torch.from_numpy(np.fromfile(tmp_path / "o" / "0.f32", dtype="<f4")).view(2, -1)
    assert pc.error(first, want[[7, 2]]) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    last = torch.from_numpy(np.fromfile(tmp_path / "o" / "2.f32", dtype="<f4")).view(2, -1)
    assert pc.error(last, torch.stack([want[0], want[10]])) < TOL
