"""Small Vofelix configurations and random weights for the tests, and helpers that run them through the
engine's replay path."""
import json

import numpy as np
import torch

import vofelix_oracle as vo


def latent(heads, dim, rot_dim, vdim, kv_rank, size, scale, base=10000.0, scaling=None, ff=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "mask": {"size": size}, "rot": rot}}


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(vocab, width, layers, loop=None, side=8, eps=1e-5, emb=6.0):
    d = {"architecture": "Vofelix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
         "embedding": {"scale": emb}, "token_side": {"dim": side}}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


#: odd sizes everywhere; B: multiples of 8 (tensor-core attention in bf16); C: attention only, many heads;
#: D: recurrent only, every count that can be 1 is 1
CONFIGS = {
    "A": lambda: config(90, 40, [delta(4, 2, 12, 20, 3), latent(3, 10, 6, 14, 20, 7, 1.1, ff=36),
                                 delta(3, 1, 9, 5, 6, ff=28)], loop=(0, 2, 2), side=6),
    "B": lambda: config(264, 128, [latent(8, 32, 16, 24, 72, 50, 0.5, 5e5, (8.0, 512, 8.0, 1.0), ff=96),
                                   delta(4, 4, 40, 48, 4), latent(5, 24, 8, 40, 200, 17, 0.6),
                                   delta(6, 3, 72, 32, 2), delta(2, 2, 16, 64, 4, ff=64)], loop=(1, 4, 3), side=16, emb=11.0),
    "C": lambda: config(200, 72, [latent(20, 16, 64, 40, 136, 33, 0.4, 1e4, (3.0, 64, 4.0, 2.0), ff=48),
                                  latent(2, 8, 2, 8, 8, 1, 1.0), latent(17, 40, 24, 16, 264, 130, 0.5)], side=24),
    "D": lambda: config(33, 24, [delta(1, 1, 8, 8, 1), delta(1, 1, 16, 1, 2)], loop=(0, 2, 3), side=1, eps=1e-3, emb=6.0),
}


def weights(cfg, seed=0):
    """Random bf16 weights under the checkpoint names."""
    g = torch.Generator().manual_seed(seed)
    W, V, D = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = torch.randn(out, inp, generator=g) * gain * inp ** -0.5

    def vec(name, n, mean, std):
        w[name] = mean + std * torch.randn(n, generator=g)

    def norm(name):
        vec(name, W, 1.0, 0.2)
        vec(name + ".b", W, 0.0, 0.1)
    w["embed"] = torch.randn(V, W, generator=g) * 0.3
    w["side.embed"] = torch.randn(V, len(cfg["layers"]) * D, generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if L["type"] == "delta":
            k, v = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, rows in (("q", k), ("k", k), ("v", v)):
                mat(p + f"mix.{n}", rows, W)
                mat(p + f"mix.{n}.conv", rows, m["conv"], 1.5)
            mat(p + "mix.b", m["heads"], W)
            mat(p + "mix.a", m["heads"], W)
            mat(p + "mix.g", v, W)
            mat(p + "mix.o", W, v)
            vec(p + "mix.A_log", m["heads"], -1.5, 1.0)
            vec(p + "mix.dt_bias", m["heads"], -0.5, 0.5)
            vec(p + "mix.norm", m["vdim"], 1.0, 0.2)
        else:
            H, d, r, c = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
            mat(p + "mix.q", H * (d + r), W, 1.5)
            mat(p + "mix.dkv", c + r, W)
            vec(p + "mix.dkv.norm", c, 1.0, 0.2)
            mat(p + "mix.uk", H * d, c)
            mat(p + "mix.uv", H * m["vdim"], c)
            vec(p + "mix.sink", H, 1.0, 1.5)
            mat(p + "mix.o", W, H * m["vdim"])
        if L["mlp"]:
            norm(p + "norm2")
            norm(p + "norm2b")
            ff = L["mlp"]["ff"]
            mat(p + "mlp.gate", ff, W)
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
        mat(p + "side.gate", D, W)
        mat(p + "side.proj", W, D)
        vec(p + "side.norm", W, 0.5, 0.1)
    norm("final.norm")
    mat("head", V, W)
    return {k: t.to(torch.bfloat16).contiguous() for k, t in w.items()}


def save(path, cfg, w):
    from safetensors.torch import save_file
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(path / "model.safetensors"))
    return str(path)


def tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def replay(rp, steps):
    """``steps``: lists of (request id, its next tokens, over afterwards).  Returns the logits of every token,
    per request."""
    out = {}
    for step in steps:
        entries = [{"id": i, "tokens": t, "want": list(range(len(t)))} for i, t, _ in step]
        got = rp.step(entries, [i for i, _, over in step if over])
        at = 0
        for i, t, _ in step:
            out.setdefault(i, []).append(got[at:at + len(t)])
            at += len(t)
    return {i: torch.cat(p) for i, p in out.items()}


def cut(ids, sizes):
    """Portions of the given sizes (repeated), as one list of pieces."""
    out, at, k = [], 0, 0
    while at < len(ids):
        out.append(ids[at:at + sizes[k % len(sizes)]])
        at += len(out[-1])
        k += 1
    return out


def alone(name, pieces):
    return [[(name, p, k == len(pieces) - 1)] for k, p in enumerate(pieces)]


def errors(got, want):
    """Per-position rms difference, relative to the spread of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d ** 2).mean(-1).sqrt() / want.double().std()


def error(got, want):
    return float(errors(got, want).max())


_KNOWN = {}


def reference(cfg, w, ids, rounded=False):
    key = (json.dumps(cfg), float(w["embed"].double().sum()), tuple(ids), rounded)
    if key not in _KNOWN:
        _KNOWN[key] = vo.forward(cfg, w, ids, rounded=rounded)
    return _KNOWN[key]


def check(got, cfg, w, ids, dtype, note=None):
    """fp32: every position within 1e-4.  bf16: the errors are those of rounding, i.e. neither their mean nor
    the largest is far above what rounding the sub-layers' inputs and outputs causes in the definition."""
    want = reference(cfg, w, ids)
    e = errors(got, want)
    if dtype == "float32":
        assert float(e.max()) < 1e-4, (note, float(e.max()))
        return
    r = errors(reference(cfg, w, ids, True), want)
    assert float(e.mean()) < 2.5 * float(r.mean()) and float(e.max()) < 3 * max(float(r.max()), 0.02), \
        (note, float(e.mean()), float(r.mean()), float(e.max()), float(r.max()))
