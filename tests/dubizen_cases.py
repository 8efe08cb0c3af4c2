"""Small Dubizen configurations and random weights for the tests, and comparisons with the plain definitions."""
import json

import torch

import dubizen_oracle as do
from pegopel_cases import interleave  # noqa: F401  (shared helpers)
from vofelix_cases import alone, cut, error, errors, replay, save, tokens  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, groups=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups:
        router["groups"] = dict(zip(("count", "keep"), groups))
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mlp=None, base=10000.0, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": mixer}


def attention(heads, kv_heads, dim, vdim, size, bias_max, scale, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max,
        "mask": {"size": size}}}


def config(vocab, width, layers, mult=0.6, eps=1e-5):
    return {"architecture": "Dubizen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "residual_mult": mult}


#: A: odd sizes; B: multiples of 8 (tensor-core kernels in bf16), windows over several pages; C: more heads than a
#: decode tile holds, wide latents and rotary parts, all experts chosen, no groups, no shared expert; D: every count
#: that can be 1 is 1; E: no experts, latents shared from two layers
CONFIGS = {
    "A": lambda: config(90, 38, [latent(3, 10, 6, 14, 21, 27, 0.3, moe(9, 3, 13, 11, (3, 2), 1.7)),
                                 attention(6, 2, 9, 14, 11, 40, 0.4, dense(35)),
                                 latent(5, 7, 6, 5, 21, 12, 0.35, dense(17), kv_from=0),
                                 attention(3, 1, 7, 5, 5, 9, 0.5, moe(6, 3, 7, 5, (2, 1), 0.8))]),
    "B": lambda: config(264, 128, [attention(6, 2, 40, 24, 70, 100, 0.15, moe(24, 5, 72, 48, (6, 3), 3.0)),
                                   latent(8, 24, 16, 40, 72, 96, 0.2, dense(112), 5e5),
                                   latent(5, 48, 16, 24, 72, 48, 0.15, moe(16, 4, 128, 256, (4, 2)), 5e5, kv_from=1),
                                   attention(4, 4, 64, 128, 50, 64, 0.12)], mult=0.4),
    "C": lambda: config(200, 72, [latent(20, 16, 64, 40, 136, 56, 0.11, moe(4, 4, 24, None, None, 0.5)),
                                  attention(24, 1, 16, 40, 135, 200, 0.25, dense(40)),
                                  latent(2, 8, 72, 8, 520, 40, 0.11), latent(17, 40, 64, 16, 136, 24, 0.1, kv_from=0),
                                  attention(16, 1, 128, 96, 90, 30, 0.09, moe(8, 1, 40, 8, (8, 1)))]),
    "D": lambda: config(33, 24, [latent(1, 1, 2, 1, 1, 1, 1.0, moe(1, 1, 1, 1, (1, 1))),
                                 attention(1, 1, 1, 1, 1, 20, 1.0, dense(1)),
                                 latent(1, 8, 2, 8, 1, 8, 1.0, moe(3, 1, 8, 1), kv_from=0)], mult=1.0, eps=1e-3),
    "E": lambda: config(120, 96, [latent(6, 16, 8, 16, 40, 32, 0.25, dense(64)), attention(8, 2, 32, 32, 20, 15, 0.2),
                                  latent(4, 32, 16, 24, 104, 64, 0.15, dense(80), 1e3),
                                  latent(6, 24, 8, 8, 40, 24, 0.2, dense(48), kv_from=0),
                                  latent(8, 16, 16, 32, 104, 40, 0.2, dense(64), 1e3, kv_from=2)], mult=0.5),
}


def weights(cfg, seed=0, buckets=16):
    """Random bf16 weights under the checkpoint names, strong enough that a far key, a bias or an expert shows."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

    def vec(name, n, mean, std):
        w[name] = mean + std * torch.randn(n, generator=g)

    def expert(name, ff):
        mat(name + ".gate", ff, W)
        mat(name + ".up", ff, W)
        mat(name + ".down", W, ff)
    w["embed"] = torch.randn(cfg["vocab"], W, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H, d, vd = m["heads"], m["dim"], m["vdim"]
        vec(p + "norm1", W, 1.0, 0.2)
        if L["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * vd)):
                mat(p + "mix." + n, rows, W)
                vec(p + f"mix.{n}.b", rows, 0.0, 0.5)
            vec(p + "mix.q.norm", d, 1.6, 0.3)
            vec(p + "mix.k.norm", d, 1.6, 0.3)
            w[p + "mix.rel"] = torch.randn(buckets, H, generator=g)
            vec(p + "mix.o.b", W, 0.0, 0.3)
        else:
            r, c, rq = m["rot_dim"], m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", rq, W)
            vec(p + "mix.dq.norm", rq, 1.4, 0.2)
            mat(p + "mix.uq", H * (d + r), rq)
            if m.get("kv_from") is None:
                mat(p + "mix.dkv", c + r, W)
                vec(p + "mix.dkv.norm", c, 1.2, 0.2)
            mat(p + "mix.uk", H * d, c)
            mat(p + "mix.uv", H * vd, c)
        mat(p + "mix.o", W, H * vd)
        if not L["mlp"]:
            continue
        vec(p + "norm2", W, 1.0, 0.2)
        if L["mlp"]["kind"] == "dense":
            mat(p + "mlp.up", L["mlp"]["ff"], W, 1.5)
            mat(p + "mlp.down", W, L["mlp"]["ff"])
            continue
        E = L["mlp"]["router"]["experts"]
        for e in range(E):
            expert(f"{p}mlp.e{e}", L["mlp"]["expert"]["ff"])
        mat(p + "mlp.router", E, W, 2.0)
        vec(p + "mlp.correction", E, -0.2, 0.2)
        if L["mlp"].get("shared"):
            expert(p + "mlp.shared", L["mlp"]["shared"]["ff"])
            mat(p + "mlp.shared.sg", 1, W, 2.0)
    vec("final.norm", W, 1.0, 0.2)
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}


_KNOWN = {}


def reference(cfg, w, ids, rounded=False):
    key = (json.dumps(cfg), sum(float(t.double().sum()) for t in w.values()), tuple(ids), rounded)
    if key not in _KNOWN:
        _KNOWN[key] = do.forward(cfg, w, ids, rounded=rounded)
    return _KNOWN[key]


def check_all(pairs, cfg, w, dtype, note=None):
    """``pairs`` of (logits, token ids).  fp32: every position within 1e-4.  bf16: neither the mean error nor the
    largest is far above what rounding the sub-layers' inputs and outputs causes in the definition; where there are
    experts, rounding may exchange two that are close, so the tenth with the largest errors does not count."""
    e = torch.cat([errors(got, reference(cfg, w, ids)) for got, ids in pairs])
    if dtype == "float32":
        assert float(e.max()) < 1e-4, (note, float(e.max()))
        return
    r = torch.cat([errors(reference(cfg, w, ids, True), reference(cfg, w, ids)) for _, ids in pairs])
    if any(L["mlp"] and L["mlp"]["kind"] == "moe" for L in cfg["layers"]):
        e, r = (t.sort().values[:max(1, len(t) * 9 // 10)] for t in (e, r))
    assert float(e.mean()) < 2.5 * float(r.mean()) and float(e.max()) < 3 * max(float(r.max()), 0.02), \
        (note, float(e.mean()), float(r.mean()), float(e.max()), float(r.max()))


def check(got, cfg, w, ids, dtype, note=None):
    check_all([(got, ids)], cfg, w, dtype, note)
