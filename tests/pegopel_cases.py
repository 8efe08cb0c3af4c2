"""Small Pegopel configurations and random weights for the tests, and comparisons with the plain definitions."""
import json

import numpy as np
import torch

import pegopel_oracle as po
from vofelix_cases import alone, cut, error, errors, replay, save, tokens  # noqa: F401  (shared helpers)


def biased(heads, kv_heads, dim, vdim, conv, size, bias_max, scale, ff=None):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale,
                      "bias_max": bias_max, "mask": {"size": size}}}


def gated(heads, kv_heads, dim, size, keep, scale, cap, rot, base=10000.0, scaling=None, ff=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention_2", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "softcap": cap,
                      "mask": {"size": size, "keep_first": keep}, "rot": r}}


def config(vocab, width, layers, streams, loop=None, eps=1e-5, positions=400):
    d = {"architecture": "Pegopel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
         "max_positions": positions, "streams": streams}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


#: A: odd sizes, many taps; B: multiples of 8 (tensor-core kernels in bf16), windows over several pages; C: one
#: stream, one key head for more heads than a decode tile holds, kept tokens beyond a tile, heads of 128; D: every
#: count that can be 1 is 1
CONFIGS = {
    "A": lambda: config(90, 40, [biased(6, 2, 9, 14, 3, 11, 40, 0.4, ff=36), gated(4, 4, 10, 7, 2, 0.5, 6.0, 6, ff=28),
                                 biased(3, 1, 7, 5, 7, 5, 9, 0.5)], 3, loop=(0, 2, 2)),
    "B": lambda: config(264, 128, [gated(8, 2, 32, 50, 9, 0.3, 8.0, 24, 5e5, (8.0, 512, 8.0, 1.0), ff=96),
                                   biased(6, 2, 40, 24, 4, 70, 64, 0.3, ff=112), biased(4, 4, 64, 128, 2, 40, 100, 0.2),
                                   gated(10, 2, 72, 18, 5, 0.2, 30.0, 72, ff=64)], 2, loop=(1, 4, 2)),
    "C": lambda: config(200, 72, [gated(20, 1, 24, 12, 140, 0.4, 5.0, 8, 1e4, (3.0, 64, 4.0, 2.0), ff=48),
                                  biased(24, 1, 16, 40, 5, 135, 50, 0.4, ff=40), gated(16, 1, 128, 90, 33, 0.2, 4.0, 128)],
                        1, loop=(1, 2, 3)),
    "D": lambda: config(33, 24, [biased(1, 1, 8, 16, 1, 1, 20, 1.0), gated(1, 1, 2, 1, 1, 1.0, 2.0, 2),
                                 biased(1, 1, 1, 1, 2, 30, 18, 1.0, ff=1)], 5, eps=1e-3),
}


def weights(cfg, seed=0, buckets=16):
    """Random bf16 weights under the checkpoint names, strong enough that a far key, a sink or a bias shows."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

    def vec(name, n, mean, std):
        w[name] = mean + std * torch.randn(n, generator=g)
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g) * 0.7
    w["pos"] = torch.randn(cfg["max_positions"], W, generator=g) * 0.4
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H, G, d, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        mat(p + "mix.q", H * d, W)
        mat(p + "mix.k", G * d, W)
        vec(p + "mix.q.norm", H * d, 1.6, 0.3)
        vec(p + "mix.k.norm", G * d, 1.6, 0.3)
        if L["type"] == "attention":
            mat(p + "mix.v", G * vd, W)
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                mat(p + f"mix.{n}.conv", rows, m["conv"], 1.2)
            w[p + "mix.rel"] = torch.randn(buckets, H, generator=g)
            vec(p + "mix.sink", H, 1.0, 1.5)
        else:
            mat(p + "mix.g", H, W, 1.5)
        mat(p + "mix.o", W, H * vd)
        vec(p + "norm1", W, 1.0, 0.2)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            vec(p + "norm2", W, 1.0, 0.2)
            mat(p + "mlp.gate", ff, W)
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
        for q in (1, 2) if L["mlp"] else (1,):
            vec(p + f"hc{q}.in", S, 1.0 / S, 0.3)
            vec(p + f"hc{q}.out", S, 1.0, 0.4)
            w[p + f"hc{q}.mix"] = 0.8 * torch.eye(S) + 0.15 * torch.randn(S, S, generator=g)
    vec("final.norm", W, 1.0, 0.2)
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}


_KNOWN = {}


def reference(cfg, w, ids, rounded=False):
    key = (json.dumps(cfg), sum(float(t.double().sum()) for t in w.values()), tuple(ids), rounded)
    if key not in _KNOWN:
        _KNOWN[key] = po.forward(cfg, w, ids, rounded=rounded)
    return _KNOWN[key]


def check_all(pairs, cfg, w, dtype, note=None):
    """``pairs`` of (logits, token ids).  fp32: every position within 1e-4.  bf16: the errors are those of rounding,
    i.e. neither their mean over all positions nor the largest is far above what rounding the sub-layers' inputs and
    outputs causes in the definition."""
    e = torch.cat([errors(got, reference(cfg, w, ids)) for got, ids in pairs])
    if dtype == "float32":
        assert float(e.max()) < 1e-4, (note, float(e.max()))
        return
    r = torch.cat([errors(reference(cfg, w, ids, True), reference(cfg, w, ids)) for _, ids in pairs])
    assert float(e.mean()) < 2.5 * float(r.mean()) and float(e.max()) < 3 * max(float(r.max()), 0.02), \
        (note, float(e.mean()), float(r.mean()), float(e.max()), float(r.max()))


def check(got, cfg, w, ids, dtype, note=None):
    check_all([(got, ids)], cfg, w, dtype, note)


def interleave(queue, seed):
    """Steps over requests whose pieces wait in ``queue``: up to four live at a time, some left out of a step."""
    rng = np.random.default_rng(seed)
    queue = {i: list(p) for i, p in queue.items()}
    steps, live, waiting = [], [], list(queue)
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step = []
        for i in list(live):
            if rng.random() < 0.25 and len(live) > 1:
                continue
            piece = queue[i].pop(0)
            step.append((i, piece, not queue[i]))
            if not queue[i]:
                live.remove(i)
        if step:
            steps.append(step)
    return steps
