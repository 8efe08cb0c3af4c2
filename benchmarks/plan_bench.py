#!/usr/bin/env python
"""Prefill and decode throughput of plan-built decoders (Vofelix, Pegopel, Dubizen, Nevotar) beside the closest existing
models at equal size, random weights, one GPU.

    python bench.py --mode layers                 # or: python benchmarks/plan_bench.py
    python benchmarks/plan_bench.py --kernels     # the single kernels with their rooflines (--variant-kernels,
                                                  # --expert-kernels, --recurrence-kernels: those of one design)

Model cases time the engine's own step on the device (CUDA events, median): a prefill step of whole prompts,
and decode-graph replays of a batch with a given context.  Weights and caches are larger than L2.  Kernel
cases rewrite a buffer larger than L2 between iterations.  Rooflines are the measured copy bandwidth and
cuBLAS bf16 rate of MEASURED_PEAKS.json.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import sys

import numpy as np
import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))

VOCAB, LAYERS = 32000, 8


def _latent(heads, window):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 12288}, "mixer": {
        "heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
        "mask": {"size": window} if window else None, "rot": {"base": 1e4, "dims": 64}}}


def _delta(ff=12288):
    return {"type": "delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": 32, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4}}


def _vofelix(layers, side=128, loop=None):
    from vllm_ascend_b200.config import ModelConfig
    d = {"architecture": "Vofelix", "vocab": VOCAB, "width": 4096, "norm": {"eps": 1e-6}, "embedding": {"scale": 64.0},
         "layers": layers}
    if side:
        d["token_side"] = {"dim": side}
    if loop:
        d["loop"] = loop
    return ModelConfig.from_hf_dict(d, name="vofelix-bench")


def _biased(window=1024, conv=4):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": 12288}, "mixer": {
        "heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "conv": conv, "scale": 128 ** -0.5, "bias_max": 512,
        "mask": {"size": window}}}


def _gated(window=1024, keep=64):
    return {"type": "attention_2", "mlp": {"kind": "dense", "ff": 12288}, "mixer": {
        "heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
        "mask": {"size": window, "keep_first": keep},
        "rot": {"base": 1e4, "dims": 128, "scaling": {"factor": 4.0, "original": 1024, "fast": 24.0, "slow": 2.0}}}}


def _pegopel(layers, streams=1, loop=None):
    from vllm_ascend_b200.config import ModelConfig
    d = {"architecture": "Pegopel", "vocab": VOCAB, "width": 4096, "norm": {"eps": 1e-6}, "max_positions": 4096,
         "streams": streams, "layers": layers}
    if loop:
        d["loop"] = loop
    return ModelConfig.from_hf_dict(d, name="pegopel-bench")


def _shared_latent(mlp, kv_from=None, heads=32):
    m = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": 1536, "scale": 192 ** -0.5,
         "rot": {"base": 1e4, "dims": 64}}
    return {"type": "latent_attention", "mlp": mlp, "mixer": m if kv_from is None else dict(m, kv_from=kv_from)}


def _normed(mlp, window=1024):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "bias_max": 512, "mask": {"size": window}}}


_PLAIN_FF = {"kind": "dense", "ff": 12288}
_EXPERTS = {"kind": "moe", "expert": {"ff": 1408}, "shared": {"ff": 2816},
            "router": {"experts": 64, "top": 8, "scale": 2.5, "groups": {"count": 8, "keep": 4}}}


def _dubizen(layers):
    from vllm_ascend_b200.config import ModelConfig
    return ModelConfig.from_hf_dict({"architecture": "Dubizen", "vocab": VOCAB, "width": 4096, "norm": {"eps": 1e-6},
                                     "residual_mult": 0.5, "layers": layers}, name="dubizen-bench")


_CLAMPED = {"kind": "moe", "expert": {"ff": 1408, "limit": 7.0}, "shared": {"ff": 2816, "limit": 7.0},
            "router": {"experts": 64, "top": 8}}


def _side(mlp, window=1024):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": window},
                 "rot": {"base": 1e4, "dims": 128}},
        "right": {"heads": 64, "vdim": 64, "state": 128, "groups": 4, "conv": 4, "norm_groups": 4},
        "left_scale": 0.7, "right_scale": 0.7}}


def _two_maps(mlp):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": 32, "kv_heads": 8, "dim": 64, "vdim": 128, "scale": 64 ** -0.5, "diff": 0.5, "q_temp": {"coef": 0.1, "every": 512}}}


def _forget(mlp):
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": 32, "dim": 128, "vdim": 128}}


def _nevotar(layers):
    from vllm_ascend_b200.config import ModelConfig
    return ModelConfig.from_hf_dict({"architecture": "Nevotar", "vocab": VOCAB, "width": 4096,
                                     "norm": {"eps": 1e-6, "groups": 4}, "layers": layers}, name="nevotar-bench")


def _gqa(window, heads=32, kv_heads=8, **kw):
    return _existing(name="gqa-dense", architecture="Qwen3ForCausalLM", num_attention_heads=heads, num_key_value_heads=kv_heads,
                     head_dim=128, qk_norm=True, sliding_window=window, rope_theta=1e4, **kw)


def _existing(**kw):
    from vllm_ascend_b200.config import ModelConfig
    kw.setdefault("hidden_act", "gelu_pytorch_tanh")
    return ModelConfig(vocab_size=VOCAB, hidden_size=4096, intermediate_size=12288, num_hidden_layers=LAYERS, **kw)


def _mla(heads, **kw):
    return _existing(name="mla-dense", architecture="DeepseekV2ForCausalLM", num_attention_heads=heads,
                     num_key_value_heads=heads, head_dim=192, use_mla=True, kv_lora_rank=512, qk_nope_head_dim=128,
                     qk_rope_head_dim=64, v_head_dim=128, rope_theta=1e4, **kw)


#: the feed-forwards of the Dubizen stacks, for existing models
_UNGATED = dict(mlp_gated=False, hidden_act="gelu")
_MOE = dict(num_experts=64, num_experts_per_tok=8, moe_intermediate_size=1408, n_shared_experts=2, scoring_func="softmax",
            n_group=8, topk_group=4, routed_scaling_factor=2.5, e_score_correction_bias=True)


_SIGMOID_MOE = dict(_MOE, scoring_func="sigmoid", n_group=1, topk_group=1, routed_scaling_factor=1.0, e_score_correction_bias=False,
                    norm_topk_prob=False)


def _gdn(**kw):
    return _existing(name="gdn-hybrid", architecture="Qwen3NextForCausalLM", num_attention_heads=32,
                     num_key_value_heads=8, head_dim=128, qk_norm=True, full_attention_interval=LAYERS,
                     linear_num_key_heads=16, linear_num_value_heads=32, linear_key_head_dim=128,
                     linear_value_head_dim=128, linear_conv_kernel_dim=4, **kw)


#: label -> configuration.  The plain Vofelix and Pegopel stacks have the mixers and feed-forward of their neighbour
MODELS = {
    "latent w=0 h32": lambda: _vofelix([_latent(32, 0)] * LAYERS, side=0),
    "existing MLA h32": lambda: _mla(32),
    "latent w=1024 h32": lambda: _vofelix([_latent(32, 1024)] * LAYERS, side=0),
    "latent w=1024 h16": lambda: _vofelix([_latent(16, 1024)] * LAYERS, side=0),
    "existing MLA h16": lambda: _mla(16),
    "delta": lambda: _vofelix([_delta()] * (LAYERS - 1) + [_latent(32, 1024)], side=0),
    "existing GDN": lambda: _gdn(),
    "whole design": lambda: _vofelix([_delta(None), _latent(32, 1024), _delta(None), _delta(None), _latent(32, 1024),
                                      _delta(None)], loop={"start": 1, "stop": 4, "times": 2}),
    "biased attention w=1024": lambda: _pegopel([_biased()] * LAYERS),
    "gated attention w=1024": lambda: _pegopel([_gated()] * LAYERS),
    "existing GQA w=1024": lambda: _gqa(1024),
    "biased attention 4 streams": lambda: _pegopel([_biased()] * LAYERS, streams=4),
    "Pegopel 2 streams loop": lambda: _pegopel([_gated(), _biased(), _biased(), _gated(), _biased(), _biased()], streams=2,
                                                 loop={"start": 1, "stop": 3, "times": 2}),
    "Dubizen latent": lambda: _dubizen([_shared_latent(_PLAIN_FF)] * LAYERS),
    "Dubizen latent, 6 of 8 shared": lambda: _dubizen([_shared_latent(_PLAIN_FF)] + [_shared_latent(_PLAIN_FF, 0)] * 3 +
                                                      [_shared_latent(_PLAIN_FF)] + [_shared_latent(_PLAIN_FF, 4)] * 3),
    "existing MLA, query latent": lambda: _mla(32, q_lora_rank=1536, **_UNGATED),
    "Dubizen attention w=1024": lambda: _dubizen([_normed(_PLAIN_FF)] * LAYERS),
    "existing GQA w=1024, plain feed-forward": lambda: _gqa(1024, **_UNGATED),
    "Dubizen latent, experts": lambda: _dubizen([_shared_latent(_EXPERTS)] * LAYERS),
    "existing MLA, experts": lambda: _mla(32, q_lora_rank=1536, **_MOE),
    "Dubizen whole": lambda: _dubizen([_shared_latent(_PLAIN_FF), _shared_latent(_EXPERTS), _normed(_PLAIN_FF),
                                       _normed(_EXPERTS), _shared_latent(_EXPERTS, 1), _shared_latent(_PLAIN_FF, 1)]),
    "Nevotar attention beside state space": lambda: _nevotar([_side(_CLAMPED)] * LAYERS),
    "existing GQA 16/4 w=1024, experts": lambda: _gqa(1024, 16, 4, **_SIGMOID_MOE),
    "Nevotar two maps": lambda: _nevotar([_two_maps(_CLAMPED)] * LAYERS),
    "existing GQA, experts": lambda: _gqa(None, **_SIGMOID_MOE),
    "Nevotar HGRN2, 7 of 8": lambda: _nevotar([_forget(_CLAMPED)] * (LAYERS - 1) + [_two_maps(_CLAMPED)]),
    "existing GDN, experts": lambda: _gdn(**_SIGMOID_MOE),
    "Nevotar whole": lambda: _nevotar([_side(_CLAMPED), _side(_CLAMPED), _two_maps(_CLAMPED), _forget(_CLAMPED)] +
                                      [dict(f(_CLAMPED), weights_of=i) for i, f in enumerate((_side, _side, _two_maps, _forget))]),
}


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        d = json.load(open(p))
        return d["hbm_gbs"], d["bf16_tflops"]
    return 6650.0, 1590.0


def _median_ms(fn, iters=12, warm=4):
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    ts = []
    for _ in range(iters):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return float(np.median(ts))


def bench_model(cfg, prefill=((4, 2048),), decode=((1, 2048), (64, 2048), (256, 2048))) -> dict:
    """Tokens/s of prefill steps (sequences, length) and of decode steps (sequences, context)."""
    from vllm_ascend_b200 import LLM, SamplingParams
    from vllm_ascend_b200.engine.request import Request
    B = max(b for b, _ in decode)
    L = max(n for _, n in decode + tuple(prefill)) + 128
    llm = LLM(cfg, device="cuda", max_model_len=L, max_num_seqs=B, max_num_batched_tokens=8192, async_scheduling=False,
              num_gpu_blocks_override=B * (L // 128 + 1) + 2, cudagraph_capture_sizes=sorted({b for b, _ in decode}))
    eng, run = llm.engine.scheduler, llm.engine.runner
    rng = np.random.default_rng(0)
    out = {}

    def requests(n, length):
        return [Request(f"b{rng.integers(1 << 60)}", rng.integers(0, VOCAB, size=length).astype(np.int32),
                        SamplingParams(max_tokens=1)) for _ in range(n)]

    def finish(reqs):
        for r in reqs:
            eng.abort_request(r.request_id)
            eng.requests.pop(r.request_id, None)
    with torch.inference_mode():
        for b, n in prefill:
            reqs = requests(b, n)
            so = eng.schedule_portions([(r, n) for r in reqs])
            run._sync_rows(so)
            meta, _, Tp, _, _ = run._prepare_inputs(so)
            ms = _median_ms(lambda: run._forward(Tp, meta))
            out[f"prefill {b}x{n}"] = {"ms": round(ms, 3), "tok_s": round(b * n / ms * 1e3)}
            finish(reqs)
        for b, n in decode:
            reqs = requests(b, n + 1)
            # context: cache contents are whatever is there, lengths and pages are real
            so = eng.schedule_portions([(r, n) for r in reqs])
            run._sync_rows(so)
            for r in reqs:
                r.num_computed_tokens = n
            so = eng.schedule_portions([(r, 1) for r in reqs])
            run._sync_rows(so)
            run._prepare_inputs(so, pad_to=b)
            ms = _median_ms(lambda: run.graph_wrapper.replay(run.graphs[(b, False)]), iters=20)
            out[f"decode {b} ctx {n}"] = {"ms": round(ms, 3), "tok_s": round(b / ms * 1e3)}
            finish(reqs)
    run.drop_graphs()
    del llm, eng, run
    gc.collect()
    torch.cuda.empty_cache()
    return out


# ---------------------------------------------------------------- single kernels
def bench_kernels() -> list[dict]:
    from kernel_bench import timeit
    from vllm_ascend_b200 import ops
    from vllm_ascend_b200.attention import mla
    from vllm_ascend_b200.ops import linear_attn as la
    from vllm_ascend_b200.ops import stream as st
    hbm, tf = peaks()
    bf, dev = torch.bfloat16, "cuda"
    res = []

    def rec(name, ms, nbytes=0, flops=0):
        t_mem, t_fl = nbytes / hbm / 1e6, flops / tf / 1e9
        res.append({"kernel": name, "ms": round(ms, 4), "GB/s": round(nbytes / ms / 1e6), "TFLOP/s": round(flops / ms / 1e9, 1),
                    "roofline_frac": round(max(t_mem, t_fl) / ms, 3)})

    def mk(*s, dtype=bf):
        return torch.randn(*s, device=dev, dtype=dtype)
    for T in (256, 8192):
        W = 4096
        r, y, w, b = mk(T, W, dtype=torch.float32), mk(T, W), mk(W), mk(W)
        ln = st.NormSpec("layer", w, b)
        rec(f"stream_norm post+next T={T}", timeit(lambda: st.stream_norm(r, y, ln, ln, 1e-6, bf)), T * W * 12)
        res_b = mk(T, W)
        rec(f"[existing] add+rms_norm T={T}", timeit(lambda: ops.rms_norm(y, w, 1e-6, res_b)), T * W * 8)
    H, Hk, D = 32, 16, 128
    for B, n in ((256, 1), (4, 2048), (1, 8192)):
        T = B * n
        C = (2 * Hk + H) * D
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        init = torch.ones(B, dtype=torch.int32, device=dev)
        x, cw, cs = mk(T, C + H * D), mk(C, 4), mk(B, 3, C)
        ba, A, dt = mk(T, 2 * H), mk(H, dtype=torch.float32), mk(H, dtype=torch.float32)
        S = torch.zeros(B, H, D, D, dtype=torch.float32, device=dev)
        tag = f"{B}x{n}"
        rec(f"conv+gates {tag}", timeit(lambda: la.causal_conv1d(x[:, :C], cw, None, cs, cu, slots, init, uniform=n == 1,
                                                                gates=(ba, A, dt))),
            T * (C * 4 + H * 12) + B * 3 * C * 4)
        m, be, g = la.causal_conv1d(x[:, :C], cw, None, cs, cu, slots, init, uniform=n == 1, gates=(ba, A, dt))
        q, k, v = (m[:, :Hk * D].view(T, Hk, D), m[:, Hk * D:2 * Hk * D].view(T, Hk, D), m[:, 2 * Hk * D:].view(T, H, D))
        rec(f"delta rule {tag}", timeit(lambda: la.gated_delta_rule(q, k, v, g, be, S, cu, slots, init, D ** -0.5,
                                                                    uniform=n == 1)),
            T * (C + H * D) * 2 + B * H * D * D * 8, 8 * T * H * D * D)
        o, nw = mk(T, H, D), mk(D)
        rec(f"gated head norm {tag}", timeit(lambda: st.gated_head_norm(o, x[:, C:], nw, 1e-6)), T * H * D * 6)
    for H in (16, 32):
        for B, n, ctx, win in ((256, 1, 2048, 0), (256, 1, 2048, 1024), (4, 2048, 2048, 0), (4, 2048, 2048, 1024)):
            if n > 1 and win == 0 and H == 32:
                continue
            bs, nb = 128, B * ctx // 128 + 1
            lat, pe = mk(nb, bs, 1, 512), mk(nb, bs, 1, 64)
            bt = (torch.arange(B * ctx // bs, dtype=torch.int32, device=dev).view(B, -1) + 1).contiguous()
            T = B * n
            cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
            sl = torch.full((B,), ctx, dtype=torch.int32, device=dev)
            ql, qp = mk(T, H, 512), mk(T, H, 64)
            sink = torch.zeros(H, device=dev) if win else None
            keys = sum(min(win or ctx, ctx - n + i + 1) for i in range(n)) * B
            reads = B * min(ctx, (win or ctx) + n)
            rec(f"latent attention H={H} {B}x{n} ctx {ctx} window {win}",
                timeit(lambda: mla.latent_attention_tc(ql, qp, lat, pe, bt, 0.07, cu=cu, seq_lens=sl, uniform=n == 1,
                                                       window=win, sink=sink, max_kv_len=ctx)),
                reads * 1152 + T * H * (576 + 512) * 2, keys * H * (576 + 512) * 2)
    res += _variant_kernels(rec_list=[], hbm=hbm, tf=tf)
    res += _expert_kernels(rec_list=[], hbm=hbm, tf=tf)
    res += _recurrence_kernels(rec_list=[], hbm=hbm, tf=tf)
    return res


def _recurrence_kernels(rec_list, hbm, tf) -> list[dict]:
    """The kernels of the Nevotar stacks that others do not have, beside their counterparts."""
    from kernel_bench import timeit
    from vllm_ascend_b200 import ops
    from vllm_ascend_b200.attention import variant as va
    from vllm_ascend_b200.attention.metadata import AttentionMetadata, build_tile_worklist
    from vllm_ascend_b200.ops import linear_attn as la
    from vllm_ascend_b200.ops import linear_recurrence as lr
    from vllm_ascend_b200.ops import moe_native
    from vllm_ascend_b200.ops import stream as st
    bf, dev = torch.bfloat16, "cuda"

    def rec(name, ms, nbytes=0, flops=0):
        t_mem, t_fl = nbytes / hbm / 1e6, flops / tf / 1e9
        rec_list.append({"kernel": name, "ms": round(ms, 4), "GB/s": round(nbytes / ms / 1e6),
                         "TFLOP/s": round(flops / ms / 1e9, 1), "roofline_frac": round(max(t_mem, t_fl) / ms, 3)})

    def mk(*s, dtype=bf):
        return torch.randn(*s, device=dev, dtype=dtype)
    W = 4096
    for T in (256, 8192):
        r, y, w, res_b, z = mk(T, W, dtype=torch.float32), mk(T, W), mk(W), mk(T, W), mk(T, W)
        rec(f"[existing] add+rms_norm T={T}", timeit(lambda: ops.rms_norm(y, w, 1e-6, res_b)), T * W * 8)
        for groups in (1, 4):
            n = st.NormSpec("rms", w, None, groups)
            rec(f"stream_norm {groups} groups T={T}", timeit(lambda: st.stream_norm(r, y, st.PLAIN, n, 1e-6, bf)), T * W * 12)
        h128 = mk(128)
        rec(f"[existing] gated head norm T={T}", timeit(lambda: st.gated_head_norm(y.view(T, 32, 128), z, h128, 1e-6)), T * W * 6)
        rec(f"group_norm 4 groups, gate T={T}", timeit(lambda: lr.group_norm(y, w, 4, 1e-6, z)), T * W * 6)
        rec(f"group_norm per head T={T}", timeit(lambda: lr.group_norm(y, h128, 32, 1e-6)), T * W * 4)
        o = mk(T, 64, 128, dtype=torch.float32)
        rec(f"map_difference T={T}", timeit(lambda: lr.map_difference(o, 0.5, 1e-6, 0.5, bf)), T * 64 * 128 * 4 + T * W * 2)
        I = 2816
        sw, x = mk(2 * I, W) * 0.02, mk(T, W)
        rec(f"[existing] gate / up product T={T}", timeit(lambda: ops.linear_swiglu(x, sw)), 2 * I * W * 2 + T * (W + I) * 2, 4 * T * I * W)
        rec(f"gate / up product, clamped T={T}", timeit(lambda: ops.linear_swiglu(x, sw, limit=7.0)),
            2 * I * W * 2 + T * (W + I) * 2, 4 * T * I * W)
        E, k, I = 64, 8, 1408
        w13 = mk(E, 2 * I, W) * 0.02
        ids = torch.stack([torch.randperm(E, device=dev)[:k] for _ in range(T)]).to(torch.int32)
        tw = torch.rand(T, k, device=dev)
        perm = moe_native.Permutation(ids, None, E)
        xs = perm.gather(x)
        used = int((perm.counts > 0).sum())
        scale = perm.row_weights(tw)
        rec(f"row weights T={T}", timeit(lambda: perm.row_weights(tw)), T * k * 12)
        cost = (used * 2 * I * W * 2 + T * k * (W + I) * 2, 4 * T * k * I * W)
        rec(f"[existing] grouped product, gate and up T={T}", timeit(lambda: moe_native.grouped_gemm(xs, w13, perm.offsets, True)), *cost)
        rec(f"grouped product, clamped, weighted rows T={T}",
            timeit(lambda: moe_native.grouped_gemm(xs, w13, perm.offsets, True, scale, 7.0)), *cost)
        del w13, xs, o
    for B, n in ((256, 1), (4, 2048), (1, 8192)):
        T, tag = B * n, f"{B}x{n}"
        cu = torch.arange(0, T + 1, n, dtype=torch.int32, device=dev)
        slots, init = torch.arange(B, dtype=torch.int32, device=dev), torch.ones(B, dtype=torch.int32, device=dev)
        H, Hk, D = 32, 16, 128
        S = torch.zeros(B, H, D, D, dtype=torch.float32, device=dev)
        q, v, g, be = mk(T, Hk, D), mk(T, H, D), -torch.rand(T, H, device=dev), torch.rand(T, H, device=dev)
        state = B * H * D * D * 8
        rec(f"[existing] delta rule {tag}", timeit(lambda: la.gated_delta_rule(q, q, v, g, be, S, cu, slots, init, D ** -0.5, uniform=n == 1)),
            T * (2 * Hk + 2 * H) * D * 2 + state, 8 * T * H * D * D)
        qfv, fb, low, nw = mk(T, 3 * H * D), mk(H * D), torch.rand(H * D, device=dev).to(bf), mk(D)
        at = H * D
        rec(f"HGRN2 recurrence with its norm {tag}", timeit(lambda: lr.forget_recurrence(
            qfv[:, :at], qfv[:, at:2 * at], qfv[:, 2 * at:], fb, low, S, cu, slots, init, nw, 1e-6, uniform=n == 1)),
            T * 4 * H * D * 2 + state, 6 * T * H * D * D)
        del S
        H, G, N, P = 64, 4, 128, 64
        C = H * P + 2 * G * N
        S = torch.zeros(B, H, N, P, dtype=torch.float32, device=dev)
        sp = lr.StateSpace(mk(H, dtype=torch.float32), mk(H, dtype=torch.float32), mk(H, dtype=torch.float32), G)
        xbc, dt = mk(T, C), mk(T, H)
        rec(f"Mamba-2 recurrence {tag}", timeit(lambda: lr.state_space(sp, xbc, dt, S, cu, slots, init, uniform=n == 1)),
            T * (C + H * P + H) * 2 + B * H * N * P * 8, 6 * T * H * N * P)
        del S
    for B, n, ctx in ((64, 1, 2048), (256, 1, 2048), (4, 2048, 2048)):
        bs, T = 128, B * n
        nb = B * ctx // bs + 1
        bt = (torch.arange(B * ctx // bs, dtype=torch.int32, device=dev).view(B, -1) + 1).contiguous()
        cu, sl = np.arange(0, T + 1, n, dtype=np.int32), np.full(B, ctx, dtype=np.int32)
        pos = torch.arange(ctx - n, ctx, device=dev).repeat(B)
        slot = (bt[torch.arange(B, device=dev).repeat_interleave(n), pos // bs].long()) * bs + pos % bs
        tag, cs, sc = f"{B}x{n} ctx {ctx}", torch.randn(4096, 128, device=dev), 128 ** -0.5

        def meta_for(group):
            m = AttentionMetadata(
                num_reqs=B, num_actual_tokens=T, max_query_len=n, max_seq_len=ctx, query_start_loc=torch.from_numpy(cu).to(dev),
                seq_lens=torch.from_numpy(sl).to(dev), block_table=bt, slot_mapping=slot, positions=pos, query_start_loc_cpu=cu,
                seq_lens_cpu=sl, num_decodes=B if n == 1 else 0, num_decode_tokens=B if n == 1 else 0)
            if n > 1:
                ts, tq = build_tile_worklist(np.full(B, n, dtype=np.int32), 128 // group, sl)
                m.tile_seq, m.tile_qoff, m.num_tiles = torch.from_numpy(ts).to(dev), torch.from_numpy(tq).to(dev), len(ts)
            else:
                m.num_splits = ops.choose_num_splits(B, G, ctx)
            return m
        for kind, H, G, parts, win in (("talk", 16, 4, 4, 1024), ("maps", 32, 8, 2, 0)):
            D = 128
            meta = meta_for(H // G)
            kc, vc = (ops.alloc_kv_cache(nb, bs, G, D, bf, dev) for _ in "kv")
            kc.normal_()
            vc.normal_()
            keys = sum(min(win or ctx, ctx - n + i + 1) for i in range(n)) * B
            nbytes, q = B * min(ctx, (win or ctx) + n) * G * D * 4 + T * H * D * 4, mk(T, H, D)
            qkv, qn = mk(T, (H + 2 * G) * D), mk(D)
            rec(f"[existing] qknorm_rope_kvwrite {H}/{G} heads {tag}", timeit(lambda: ops.qknorm_rope_kvwrite(
                qkv, pos, cs, D, qn, qn, 1e-6, kc, vc, slot, H, G, D)), T * (H + 2 * G) * D * 4)
            rec(f"[existing] paged attention {H}/{G} heads {tag} window {win}",
                timeit(lambda: ops.paged_attention(q, kc, vc, meta, sc, window=win)), nbytes, keys * H * D * 4)
            if kind == "talk":
                wide = torch.randn(nb, bs, 1, G * D, device=dev, dtype=bf)
                mix = torch.randn(H, H, device=dev)
                spec = va.PrepSpec(H, G, D, D, 1e-6, qn, qn, (H * D, G * D), rot_dims=D, cos_sin=cs, head_norm=True, v_heads=G,
                                   key_parts=G, part_run=H // G, mix=mix)
                o, flops = va.AttnOptions(sc, win, out_scale=0.7), keys * (H * D * 4 + H * H * 2)
                wq = T * H * G * D * 2
            else:
                wide = torch.randn(nb, bs, G, D, device=dev, dtype=bf)
                table = torch.rand(4096, device=dev)
                spec = va.PrepSpec(2 * H, 2 * G, D // 2, D, 1e-6, None, None, (0, 0), v_heads=G, key_parts=2, q_scale=table)
                o, flops = va.AttnOptions(sc, win, out_f32=True), keys * H * (2 * D + 4 * D)
                wq = T * H * 2 * D * 2
            rec(f"qkv_prep {kind} {tag}", timeit(lambda: va.qkv_prep(spec, qkv, meta, wide, vc)), T * (H + 2 * G) * D * 2 + T * 2 * G * D * 2 + wq)
            qw = va.qkv_prep(spec, qkv, meta, wide, vc)
            rec(f"attention {kind} {tag} window {win}", timeit(lambda: va.variant_attention(qw, wide, vc, meta, o)),
                B * min(ctx, (win or ctx) + n) * G * D * 4 + wq + T * H * D * (2 if kind == "talk" else 8), flops)
            del kc, vc, wide, qw
    return rec_list


def _expert_kernels(rec_list, hbm, tf) -> list[dict]:
    """The kernels of the Dubizen stacks that others do not have, beside their counterparts."""
    from kernel_bench import timeit
    from vllm_ascend_b200 import ops
    from vllm_ascend_b200.attention import variant as va
    from vllm_ascend_b200.attention.metadata import AttentionMetadata
    from vllm_ascend_b200.ops import fused_moe, moe_native, reference as ref
    from vllm_ascend_b200.ops import stream as st
    bf, dev = torch.bfloat16, "cuda"

    def rec(name, ms, nbytes=0, flops=0):
        t_mem, t_fl = nbytes / hbm / 1e6, flops / tf / 1e9
        rec_list.append({"kernel": name, "ms": round(ms, 4), "GB/s": round(nbytes / ms / 1e6),
                         "TFLOP/s": round(flops / ms / 1e9, 1), "roofline_frac": round(max(t_mem, t_fl) / ms, 3)})

    def mk(*s, dtype=bf):
        return torch.randn(*s, device=dev, dtype=dtype)
    W, H, dn, dr, dc, rq, G, D = 4096, 32, 128, 64, 512, 1536, 8, 128
    cs = ref.build_cos_sin_cache(dr, 8192, 1e4, None, torch.device("cuda"))
    for T in (64, 256, 8192):
        r, y, w, res_b = mk(T, W, dtype=torch.float32), mk(T, W), mk(W), mk(T, W)
        ln = st.NormSpec("layer", w)
        rec(f"[existing] add+rms_norm T={T}", timeit(lambda: ops.rms_norm(y, w, 1e-6, res_b)), T * W * 8)
        rec(f"stream_norm output norm T={T}", timeit(lambda: st.stream_norm(r, y, ln, st.PLAIN, 1e-6, bf, post_scale=0.5)),
            T * W * 12)
        q, kv, down, nw, qw = mk(T, H, dn + dr), mk(T, dc + dr), mk(T, rq + dc + dr), mk(dc), mk(rq)
        nb = (T + 127) // 128 + 1
        lat, pe = torch.zeros(nb, 128, 1, dc, device=dev, dtype=bf), torch.zeros(nb, 128, 1, dr, device=dev, dtype=bf)
        pos, slots = torch.arange(T, device=dev) % 4096, torch.arange(T, device=dev) + 128
        rec(f"[existing] mla_preprocess T={T}", timeit(lambda: ops.mla_preprocess(q, kv, nw, 1e-6, pos, cs, slots, lat, pe, dn, dr)),
            T * (H * dr + dc + dr) * 4)
        cq = mk(T, rq)
        rec(f"[existing] rms_norm of the query latent T={T}", timeit(lambda: ops.rms_norm(cq, qw, 1e-6)), T * rq * 4)
        rec(f"[existing] copy to head-major rows T={T}", timeit(lambda: q[..., :dn].transpose(0, 1).contiguous()), T * H * dn * 4)
        rec(f"latent_prep T={T}", timeit(lambda: ops.latent_prep(down, qw, nw, 1e-6, pos, cs, slots, lat, pe)),
            T * (rq + dc + dr) * 4)
        rec(f"latent_query T={T}", timeit(lambda: ops.latent_query(q, pos, cs)), T * H * (dn + dr) * 4)
        kc, vc = (ops.alloc_kv_cache(nb, 128, G, D, bf, dev) for _ in "kv")
        C = (H + 2 * G) * D
        qkv, hn, c128 = mk(T, C), mk(D), torch.randn(8192, D, device=dev)
        cu = np.array([0, T], dtype=np.int32)
        meta = AttentionMetadata(num_reqs=1, num_actual_tokens=T, max_query_len=T, max_seq_len=T,
                                 query_start_loc=torch.from_numpy(cu).to(dev), seq_lens=None, block_table=None,
                                 slot_mapping=slots, positions=pos, query_start_loc_cpu=cu, seq_lens_cpu=None)
        rec(f"[existing] qknorm_rope_kvwrite T={T}", timeit(lambda: ops.qknorm_rope_kvwrite(
            qkv, pos, c128, D, hn, hn, 1e-6, kc, vc, slots, H, G, D)), T * C * 4)
        spec = va.PrepSpec(H, G, D, D, 1e-6, hn, hn, (H * D, G * D), head_norm=True)
        rec(f"qkv_prep norm per head T={T}", timeit(lambda: va.qkv_prep(spec, qkv, meta, kc, vc)), T * C * 4)
        act = mk(T, 12288)
        rec(f"gelu T={T}", timeit(lambda: ops.activation(act, "gelu")), T * 12288 * 4)
        E, k, I = 64, 8, 1408
        rw, corr = mk(E, W), torch.randn(E, device=dev) * 0.1
        rf = rw.float()
        rec(f"[existing] router product, fp32 operands T={T}", timeit(lambda: torch.nn.functional.linear(y.float(), rf)),
            T * W * 2 + E * W * 2, 2 * T * W * E)
        rec(f"router product T={T}", timeit(lambda: ops.linear_fp32(y, rw)), T * W * 2 + E * W * 2 + T * E * 4, 2 * T * W * E)
        z = ops.linear_fp32(y, rw) * 0.01
        for name, score in (("[existing] gating, best two of a group", "top2"), ("gating, best of a group", "max")):
            rec(f"{name} T={T}", timeit(lambda: fused_moe.gating_topk(z, k, "softmax", True, 8, 4, corr, 2.5, score)),
                T * E * 4 + T * k * 8)
        tw, ids = fused_moe.gating_topk(z, k, "softmax", True, 8, 4, corr, 2.5, "max")
        w13, w2, s, sg = mk(E, 2 * I, W) * 0.02, mk(E, W, I) * 0.02, mk(T, W), mk(1, W)
        perm = moe_native.Permutation(ids, None, E)
        rec(f"permute T={T}", timeit(lambda: moe_native.Permutation(ids, None, E)), T * k * 16)
        xs = perm.gather(y)
        rec(f"gather T={T}", timeit(lambda: perm.gather(y)), T * W * 2 + T * k * W * 2)
        used = int((perm.counts > 0).sum())
        h = moe_native.grouped_gemm(xs, w13, perm.offsets, True)
        rec(f"grouped product, gate and up T={T}", timeit(lambda: moe_native.grouped_gemm(xs, w13, perm.offsets, True)),
            used * 2 * I * W * 2 + T * k * (W + I) * 2, 4 * T * k * I * W)
        o = moe_native.grouped_gemm(h, w2, perm.offsets, False)
        rec(f"grouped product, down T={T}", timeit(lambda: moe_native.grouped_gemm(h, w2, perm.offsets, False)),
            used * I * W * 2 + T * k * (W + I) * 2, 2 * T * k * I * W)

        def apart():
            return perm.combine(o, tw) + s * torch.sigmoid(torch.nn.functional.linear(y.float(), sg.float())).to(bf)
        rec(f"[existing] combine, then the gated shared expert T={T}", timeit(apart), T * W * 2 * (k + 3))
        rec(f"combine with the gated shared expert T={T}", timeit(lambda: perm.combine(o, tw, shared=s, x=y, shared_gate=sg)),
            T * W * 2 * (k + 3))
        del w13, w2, xs, h, o
    return rec_list


def _variant_kernels(rec_list, hbm, tf) -> list[dict]:
    """The kernels of paged attention with options and of parallel streams, beside their plain counterparts."""
    from kernel_bench import timeit
    from vllm_ascend_b200 import ops
    from vllm_ascend_b200.attention import variant as va
    from vllm_ascend_b200.attention.metadata import AttentionMetadata, build_tile_worklist
    from vllm_ascend_b200.ops import stream as st
    bf, dev = torch.bfloat16, "cuda"

    def rec(name, ms, nbytes=0, flops=0):
        t_mem, t_fl = nbytes / hbm / 1e6, flops / tf / 1e9
        rec_list.append({"kernel": name, "ms": round(ms, 4), "GB/s": round(nbytes / ms / 1e6),
                         "TFLOP/s": round(flops / ms / 1e9, 1), "roofline_frac": round(max(t_mem, t_fl) / ms, 3)})

    def mk(*s, dtype=bf):
        return torch.randn(*s, device=dev, dtype=dtype)
    W = 4096
    for T in (256, 8192):
        y, w, res_b = mk(T, W), mk(W), mk(T, W)
        rec(f"[existing] add+rms_norm T={T}", timeit(lambda: ops.rms_norm(y, w, 1e-6, res_b)), T * W * 8)
        for S in (1, 2, 4):
            r = mk(T, S, W, dtype=torch.float32)
            m = st.StreamMix(torch.ones(S, device=dev) / S, torch.ones(S, device=dev), torch.eye(S, device=dev))
            n = st.NormSpec("rms", w)
            rec(f"stream_mix S={S} T={T}", timeit(lambda: st.stream_mix(r, y, st.PLAIN, m, m, n, 1e-6, bf)),
                T * W * (8 * S + 4))
    Hq, G, D = 32, 8, 128
    for B, n, ctx in ((64, 1, 2048), (256, 1, 2048), (4, 2048, 2048)):
        bs, T = 128, B * n
        nb = B * ctx // bs + 1
        kc, vc = (ops.alloc_kv_cache(nb, bs, G, D, bf, dev) for _ in "kv")
        kc.normal_()
        vc.normal_()
        bt = (torch.arange(B * ctx // bs, dtype=torch.int32, device=dev).view(B, -1) + 1).contiguous()
        cu = np.arange(0, T + 1, n, dtype=np.int32)
        sl = np.full(B, ctx, dtype=np.int32)
        pos = torch.arange(ctx - n, ctx, device=dev).repeat(B)
        slot = (bt[torch.arange(B, device=dev).repeat_interleave(n), pos // bs].long()) * bs + pos % bs
        meta = AttentionMetadata(
            num_reqs=B, num_actual_tokens=T, max_query_len=n, max_seq_len=ctx, query_start_loc=torch.from_numpy(cu).to(dev),
            seq_lens=torch.from_numpy(sl).to(dev), block_table=bt, slot_mapping=slot, positions=pos, query_start_loc_cpu=cu,
            seq_lens_cpu=sl, num_decodes=B if n == 1 else 0, num_decode_tokens=B if n == 1 else 0)
        meta.state_slots = torch.arange(B, dtype=torch.int32, device=dev)
        meta.has_initial_state = torch.ones(B, dtype=torch.int32, device=dev)
        if n > 1:
            ts, tq = build_tile_worklist(np.full(B, n, dtype=np.int32), 128 // (Hq // G), sl)
            meta.tile_seq, meta.tile_qoff, meta.num_tiles = torch.from_numpy(ts).to(dev), torch.from_numpy(tq).to(dev), len(ts)
        else:
            meta.num_splits = ops.choose_num_splits(B, G, ctx)
        tag = f"{B}x{n} ctx {ctx}"
        C = (Hq + 2 * G) * D
        qkv, qn, kn = mk(T, C), mk(Hq * D), mk(G * D)
        cs = torch.randn(4096, D, device=dev)
        rec(f"[existing] qknorm_rope_kvwrite {tag}", timeit(lambda: ops.qknorm_rope_kvwrite(
            qkv, pos, cs, D, qn[:D], kn[:D], 1e-6, kc, vc, slot, Hq, G, D)), T * C * 4)
        spec = va.PrepSpec(Hq, G, D, D, 1e-6, qn, kn, (Hq * D, G * D), conv=mk(C, 4))
        state = mk(B, 3, C)
        rec(f"qkv_prep conv {tag}", timeit(lambda: va.qkv_prep(spec, qkv, meta, kc, vc, state)),
            T * C * 4 + B * C * 3 * 4)
        spec2 = va.PrepSpec(Hq, G, D, D, 1e-6, qn, kn, (Hq * D, G * D), values_from_keys=True, rot_dims=D, cos_sin=cs)
        rec(f"qkv_prep rotary, v = k {tag}", timeit(lambda: va.qkv_prep(spec2, qkv, meta, kc, vc)),
            T * ((Hq + G) * D * 2 + (Hq + 2 * G) * D * 2))
        q = mk(T, Hq, D)
        bias = torch.randn(Hq, 460, device=dev)
        zero, gate = torch.zeros(Hq, device=dev), mk(T, Hq)
        sc = D ** -0.5
        for win in (1024, 0):
            keys = sum(min(win or ctx, ctx - n + i + 1) for i in range(n)) * B
            nbytes = B * min(ctx, (win or ctx) + n) * G * D * 4 + T * Hq * D * 4
            fl = keys * Hq * D * 4
            rec(f"[existing] paged attention {tag} window {win}",
                timeit(lambda: ops.paged_attention(q, kc, vc, meta, sc, window=win)), nbytes, fl)
            for name, o, g in (("no options", va.AttnOptions(sc, win), None),
                               ("bias", va.AttnOptions(sc, win, bias=bias), None),
                               ("bias + sink", va.AttnOptions(sc, win, bias=bias, sink=zero), None),
                               ("cap + kept + gate", va.AttnOptions(sc, win, 64, 30.0, sink=zero), gate)):
                rec(f"attention {name} {tag} window {win}", timeit(lambda: va.variant_attention(q, kc, vc, meta, o, g)),
                    nbytes, fl)
    return rec_list


def run_models(names=None) -> dict:
    return {k: bench_model(MODELS[k]()) for k in MODELS if not names or k in names}


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--variant-kernels", action="store_true", help="only the kernels of attention with options")
    ap.add_argument("--expert-kernels", action="store_true", help="only the kernels of the Dubizen stacks")
    ap.add_argument("--recurrence-kernels", action="store_true", help="only the kernels of the Nevotar stacks")
    ap.add_argument("--only", default="", help="model labels with semicolons between them")
    args = ap.parse_args()
    if args.variant_kernels:
        for row in _variant_kernels([], *peaks()):
            print(json.dumps(row))
        return
    if args.expert_kernels:
        for row in _expert_kernels([], *peaks()):
            print(json.dumps(row), flush=True)
        return
    if args.recurrence_kernels:
        for row in _recurrence_kernels([], *peaks()):
            print(json.dumps(row), flush=True)
        return
    if args.kernels:
        for row in bench_kernels():
            print(json.dumps(row))
        return
    for k in MODELS:
        if not args.only or k in args.only.split(";"):
            print(json.dumps({k: bench_model(MODELS[k]())}), flush=True)


if __name__ == "__main__":
    main()
