"""Small Nevotar configurations and random weights for the tests, and comparisons with the plain definitions."""
import json

import torch

import nevotar_oracle as no
from pegopel_cases import interleave  # noqa: F401  (shared helpers)
from vofelix_cases import alone, cut, error, errors, replay, save, tokens  # noqa: F401


def moe(experts, top, ff, limit, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = dict(zip(("ff", "limit"), shared))
    return out


def maps(heads, kv_heads, dim, vdim, scale, diff, temp=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if temp:
        m["q_temp"] = dict(zip(("coef", "every"), temp))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def hgrn2(heads, dim, vdim, mlp=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def parallel(left, right, scales, mlp=None):
    """left: heads, kv_heads, dim, vdim, scale, window, (base, dims); right: heads, vdim, state, groups, conv, norms."""
    H, G, d, vd, scale, size, rot = left
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": d, "vdim": vd, "scale": scale, "mask": {"size": size},
                 "rot": dict(zip(("base", "dims"), rot))},
        "right": dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), right)),
        "left_scale": scales[0], "right_scale": scales[1]}}


def again(layers, *sources):
    """The layers, then layers that use the weights of the given ones."""
    return layers + [dict(layers[j], weights_of=j) for j in sources]


def config(vocab, width, groups, layers, eps=1e-5):
    return {"architecture": "Nevotar", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps, "groups": groups}}


#: A: odd sizes; B: multiples of 8 (tensor-core kernels in bf16: keys of 160 and 192 side by side), windows over several
#: pages; C: more heads than a decode tile holds, one key head, keys too wide for the tensor-core prompt kernel, norms in
#: one part and in many, no shared expert; D: every count that can be 1 is 1; E: layers that use others' weights first
#: and last, no feed-forwards in some
CONFIGS = {
    "A": lambda: config(91, 45, 5, again([
        parallel((6, 3, 10, 7, 0.4, 11, (5e3, 6)), (6, 5, 9, 3, 4, 2), (0.8, 0.35), moe(7, 3, 13, 1.5, (11, 2.5))),
        maps(6, 2, 7, 11, 0.3, 0.45, (0.4, 9), moe(5, 2, 9, 0.7)), hgrn2(3, 9, 13, moe(4, 1, 6, 3.0, (5, 0.5)))], 1, 0)),
    "B": lambda: config(264, 128, 4, [
        parallel((10, 5, 32, 40, 0.2, 70, (2e5, 16)), (8, 24, 40, 4, 4, 8), (0.45, 0.9), moe(24, 5, 72, 2.0, (48, 3.0))),
        maps(6, 3, 96, 56, 0.11, 0.2, (0.25, 50), moe(12, 2, 40, 1.0, (136, 1.5))),
        hgrn2(6, 40, 32, moe(16, 4, 128, 0.8, (56, 1.2))), maps(8, 2, 24, 128, 0.2, 0.6)]),
    "C": lambda: config(200, 72, 1, [
        parallel((24, 1, 72, 24, 0.15, 135, (1e3, 72)), (3, 40, 72, 1, 2, 1), (1.3, 0.2), moe(4, 4, 24, 5.0)),
        maps(40, 1, 8, 16, 0.5, 0.8, (1.0, 33), moe(9, 1, 16, 0.4, (8, 0.3))),
        parallel((18, 9, 64, 8, 0.08, 300, (1e4, 0)), (4, 16, 136, 2, 1, 4), (0.5, 0.5)),
        hgrn2(2, 136, 72), hgrn2(2, 72, 264), maps(16, 2, 72, 24, 0.12, 0.1)]),
    "D": lambda: config(33, 24, 24, [
        parallel((1, 1, 1, 1, 1.0, 1, (100.0, 0)), (1, 1, 1, 1, 1, 1), (1.0, 1.0), moe(1, 1, 1, 1.0, (1, 1.0))),
        maps(1, 1, 1, 1, 1.0, 0.5, (0.1, 1), moe(2, 1, 1, 1.0)), hgrn2(1, 1, 1),
        parallel((2, 2, 8, 8, 0.5, 2, (1e4, 8)), (2, 4, 8, 2, 3, 1), (0.5, 1.0)), hgrn2(1, 8, 4)], eps=0.05),
    "E": lambda: config(120, 96, 2, again([
        hgrn2(4, 32, 24, moe(6, 2, 32, 1.1, (40, 0.9))),
        parallel((4, 2, 24, 16, 0.25, 33, (1e4, 8)), (4, 16, 16, 1, 5, 4), (0.7, 0.6)),
        maps(4, 4, 16, 32, 0.25, 0.3)], 0, 2, 1, 1) + [hgrn2(2, 16, 48)]),
}


def weights(cfg, seed=0):
    """Random bf16 weights under the checkpoint names, strong enough that a far key, a gate or an expert shows."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

    def vec(name, n, mean, std):
        w[name] = mean + std * torch.randn(n, generator=g)

    def expert(name, ff):
        mat(name + ".gate", ff, W, 1.5)
        mat(name + ".up", ff, W, 1.5)
        mat(name + ".down", W, ff)

    def biased(p, m, parts):
        for n, rows in (("q", m["heads"] * m["dim"] * parts), ("k", m["kv_heads"] * m["dim"] * parts),
                        ("v", m["kv_heads"] * m["vdim"])):
            mat(p + n, rows, W)
            vec(p + n + ".b", rows, 0.0, 0.5)
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g)
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", L["mixer"]
        vec(p + "norm1", W, 1.0, 0.2)
        if L["type"] == "attention":
            biased(p + "mix.", m, 2)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(p + "mix." + n, m["dim"], 0.1, 0.4 * m["dim"] ** -0.5)
            mat(p + "mix.o", W, m["heads"] * m["vdim"])
        elif L["type"] == "hgrn2":
            H, d, vd = m["heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * d, W)
            mat(p + "mix.f", H * d, W, 2.0)
            vec(p + "mix.f.b", H * d, 1.0, 1.5)
            w[p + "mix.lower"] = torch.rand(H * d, generator=g) * 0.9
            mat(p + "mix.v", H * vd, W)
            vec(p + "mix.norm", vd, 1.0, 0.2)
            mat(p + "mix.o", W, H * vd)
        else:
            left, r = m["left"], m["right"]
            biased(p + "mix.left.", left, 1)
            vec(p + "mix.left.q.norm", left["dim"], 1.6, 0.3)
            vec(p + "mix.left.k.norm", left["dim"], 1.6, 0.3)
            w[p + "mix.left.talk"] = torch.eye(left["heads"]) + 0.4 * torch.randn(left["heads"], left["heads"], generator=g)
            mat(p + "mix.left.o", W, left["heads"] * left["vdim"])
            inner, gn, H = r["heads"] * r["vdim"], r["groups"] * r["state"], r["heads"]
            mat(p + "mix.right.in", 2 * inner + 2 * gn + H, W)
            w[p + "mix.right.conv"] = torch.randn(inner + 2 * gn, r["conv"], generator=g) * r["conv"] ** -0.5
            vec(p + "mix.right.conv.b", inner + 2 * gn, 0.0, 0.3)
            vec(p + "mix.right.dt_bias", H, -1.0, 1.0)
            vec(p + "mix.right.A_log", H, 0.0, 1.0)
            vec(p + "mix.right.D", H, 1.0, 0.3)
            vec(p + "mix.right.norm", inner, 1.0, 0.2)
            mat(p + "mix.right.o", W, inner)
        if not L["mlp"]:
            continue
        vec(p + "norm2", W, 1.0, 0.2)
        for e in range(L["mlp"]["router"]["experts"]):
            expert(f"{p}mlp.e{e}", L["mlp"]["expert"]["ff"])
        mat(p + "mlp.router", L["mlp"]["router"]["experts"], W, 2.0)
        if L["mlp"].get("shared"):
            expert(p + "mlp.shared", L["mlp"]["shared"]["ff"])
    vec("final.norm", W, 1.0, 0.2)
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}


_KNOWN = {}


def reference(cfg, w, ids, rounded=False):
    key = (json.dumps(cfg), sum(float(t.double().sum()) for t in w.values()), tuple(ids), rounded)
    if key not in _KNOWN:
        _KNOWN[key] = no.forward(cfg, w, ids, rounded=rounded)
    return _KNOWN[key]


def check_all(pairs, cfg, w, dtype, note=None):
    """``pairs`` of (logits, token ids).  fp32: every position within 1e-4.  bf16: neither the mean error nor the
    largest is far above what rounding causes in the definition; rounding may exchange two experts that are close, and
    a state carries the difference on, so the fifth with the largest errors does not count."""
    e = torch.cat([errors(got, reference(cfg, w, ids)) for got, ids in pairs])
    if dtype == "float32":
        assert float(e.max()) < 1e-4, (note, float(e.max()))
        return
    r = torch.cat([errors(reference(cfg, w, ids, True), reference(cfg, w, ids)) for _, ids in pairs])
    e, r = (t.sort().values[:max(1, len(t) * 4 // 5)] for t in (e, r))
    assert float(e.mean()) < 2.5 * float(r.mean()) and float(e.max()) < 3 * max(float(r.max()), 0.02), \
        (note, float(e.mean()), float(r.mean()), float(e.max()), float(r.max()))


def check(got, cfg, w, ids, dtype, note=None):
    check_all([(got, ids)], cfg, w, dtype, note)
