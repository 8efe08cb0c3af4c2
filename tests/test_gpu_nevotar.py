"""Nevotar on the GPU engine, fp32 and bf16, against the plain definitions: prompts, portions, decoding
(graph replay included), mixed batches, reused pages and slots, generation."""
import pytest

import nevotar_cases as nc
import nevotar_oracle as no

pytestmark = pytest.mark.gpu
DTYPES = ["bfloat16", "float32"]


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


def engine(path, dtype, max_tokens=256, page=64):
    from vllm_ascend_b200.engine.replay import TraceReplayer, make_replay_engine
    return TraceReplayer(make_replay_engine(path, dtype, max_tokens, page=page))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(nc.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_definition(cases, name, dtype):
    cfg, w, path = cases(name)
    ids = nc.tokens(cfg, 170, 1)
    rp = engine(path, dtype)
    assert rp.runner.capture_sizes == [1, 2, 4]
    for sizes in ([170], [1], [2, 3], [2], [64, 1, 63, 65], [140, 1]):
        got = nc.replay(rp, nc.alone("r", nc.cut(ids, sizes)))["r"]
        nc.check(got, cfg, w, ids, dtype, sizes)
    assert rp.runner.stats["graph_replays"] > 150
    assert rp.scheduler.pool.num_free_blocks == rp.scheduler.pool.num_blocks - 1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "E"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(cases, name, dtype):
    cfg, w, path = cases(name)
    ids = {i: nc.tokens(cfg, n, 10 + k) for k, (i, n) in enumerate(
        [("a", 90), ("b", 1), ("c", 70), ("d", 33), ("e", 66), ("f", 129), ("g", 7)])}
    sizes = ([40, 1, 1, 2], [1], [70], [2, 1], [5, 1], [1, 64], [3])
    rp = engine(path, dtype, max_tokens=16 * 32, page=16)
    got = nc.replay(rp, nc.interleave({i: nc.cut(t, s) for (i, t), s in zip(ids.items(), sizes)}, 7))
    nc.check_all([(got[i], t) for i, t in ids.items()], cfg, w, dtype)


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("E", "bfloat16")])
def test_long_decoding(cases, name, dtype):
    cfg, w, path = cases(name)
    ids = nc.tokens(cfg, 300, 8)
    rp = engine(path, dtype, max_tokens=320, page=16)
    nc.check(nc.replay(rp, nc.alone("r", nc.cut(ids, [4] + [1] * 300)))["r"], cfg, w, ids, dtype)


@pytest.mark.parametrize("async_scheduling", [True, False])
def test_greedy_generation_through_the_engine(cases, async_scheduling):
    from vllm_ascend_b200 import LLM, SamplingParams
    cfg, w, path = cases("B")
    prompts = [nc.tokens(cfg, n, 20 + n) for n in (53, 2, 19, 5, 37, 1)]
    llm = LLM(path, dtype="float32", device="cuda", max_model_len=128, max_num_seqs=3, max_num_batched_tokens=16,
              num_gpu_blocks_override=8, cudagraph_capture_sizes=[1, 2, 3], async_scheduling=async_scheduling)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    for p, o in zip(prompts, outs):
        seq = list(p) + list(o.outputs[0].token_ids)
        lg = no.forward(cfg, w, seq)
        assert [int(t) for t in lg[len(p) - 1:-1].argmax(-1)] == seq[len(p):]


def test_bf16_generation_of_random_weights_preset():
    """Through the bf16 path the engine serves: sampling with a seed repeats itself."""
    from vllm_ascend_b200 import LLM, SamplingParams
    llm = LLM("tiny-nevotar", dtype="bfloat16", device="cuda", max_model_len=128, max_num_seqs=4,
              max_num_batched_tokens=64, num_gpu_blocks_override=16, cudagraph_capture_sizes=[1, 2, 4])
    sp = SamplingParams(temperature=0.8, seed=3, max_tokens=12, ignore_eos=True)
    runs = [[list(o.outputs[0].token_ids) for o in llm.generate([[1, 2, 3], [7] * 70], sp)] for _ in range(2)]
    assert runs[0] == runs[1] and all(len(t) == 12 for t in runs[0])
    assert llm.engine.runner.total_launches() > 0


def test_runs_of_a_layer_have_states_of_their_own(cases):
    """The second run of a layer's weights must not see the first run's state: two requests that differ only in an early
    token, decoded side by side."""
    cfg, w, path = cases("E")
    a = nc.tokens(cfg, 40, 5)
    b = [(a[0] + 1) % cfg["vocab"]] + a[1:]
    rp = engine(path, "float32", page=16)
    got = nc.replay(rp, nc.interleave({"a": nc.cut(a, [17, 1, 1, 2]), "b": nc.cut(b, [3, 1])}, 2))
    nc.check_all([(got["a"], a), (got["b"], b)], cfg, w, "float32")
