"""Plain definitions of the mechanisms of the Dubizen decoder, for tests: token by token, one function per
mechanism, torch on the CPU in the precision of the given weights (float64 by default).  Nothing here is
shared with the package; what the definitions of other designs already say is taken from there."""
import math

import torch

from pegopel_oracle import attend
from vofelix_oracle import rms_norm, silu, sub


def output_norm(y, w, eps):
    """Layer norm without a bias."""
    d = y - y.mean(-1, keepdim=True)
    return d / torch.sqrt((d ** 2).mean(-1, keepdim=True) + eps) * w


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def rotate_halves(x, pos, dims, base):
    """x [..., d] at position ``pos``: entry i of the first ``dims`` turns together with entry i + dims / 2."""
    y, half = x.clone(), dims // 2
    for i in range(half):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * math.cos(a) - v * math.sin(a)
        y[..., i + half] = v * math.cos(a) + u * math.sin(a)
    return y


def normed_attention(h, p, c, eps, shared=None):
    """Grouped-query attention with biases in the projections, q and k normalised head by head with one weight for
    all heads, a bias by distance and a window."""
    n, H, G, d, vd = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = ((h @ p[x].T + p[x + ".b"]).view(n, heads, size) for x, heads, size in (("q", H, d), ("k", G, d), ("v", G, vd)))
    q, k = rms_norm(q, p["q.norm"], eps), rms_norm(k, p["k.norm"], eps)
    o = attend(q, k, v, c["scale"], c["mask"]["size"], bias=p["rel"], largest=c["bias_max"])
    return o.reshape(n, H * vd) @ p["o"].T + p["o.b"]


def latents(h, p, c, eps):
    """(latent [n, kv_rank], rotated key part [n, rot_dim]) as a layer with a down-projection stores them."""
    down, rank, rot = h @ p["dkv"].T, c["kv_rank"], c["rot"]
    keys = torch.stack([rotate_halves(down[j, rank:], j, rot["dims"], rot["base"]) for j in range(h.shape[0])])
    return rms_norm(down[:, :rank], p["dkv.norm"], eps), keys


def latent_attention(h, p, c, eps, shared=None):
    """Latent attention over ``shared`` latents and rotated keys (None: its own); queries through a latent."""
    n, H, d, r, vd, rot = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["rot"]
    lat, key_rot = latents(h, p, c, eps) if shared is None else shared
    q = (rms_norm(h @ p["dq"].T, p["dq.norm"], eps) @ p["uq"].T).view(n, H, d + r)
    keys, vals = (lat @ p["uk"].T).view(n, H, d), (lat @ p["uv"].T).view(n, H, vd)
    out = torch.zeros(n, H, vd, dtype=h.dtype)
    for i in range(n):
        turned = rotate_halves(q[i, :, d:], i, rot["dims"], rot["base"])
        s = (torch.einsum("hd,jhd->hj", q[i, :, :d], keys[:i + 1]) + turned @ key_rot[:i + 1].T) * c["scale"]
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhv->hv", e / e.sum(-1, keepdim=True), vals[:i + 1])
    return out.reshape(n, H * vd) @ p["o"].T


MIXERS = {"attention": normed_attention, "latent_attention": latent_attention}


def dense(x, p):
    return gelu_erf(x @ p["up"].T) @ p["down"].T


def expert(x, p):
    return (silu(x @ p["gate"].T) * (x @ p["up"].T)) @ p["down"].T


def route(logits, correction, c):
    """One token's router: {expert: weight} of the chosen experts."""
    s = [float(v) for v in torch.softmax(logits, -1)]
    choice = [a + float(b) for a, b in zip(s, correction)]
    groups = c.get("groups") or {"count": 1, "keep": 1}
    size = len(s) // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(choice[g * size:(g + 1) * size]))[:groups["keep"]]
    open_ = [e for e in range(len(s)) if e // size in best]
    chosen = sorted(open_, key=lambda e: -choice[e])[:c["top"]]
    total = sum(s[e] for e in chosen) + 1e-20
    return {e: s[e] / total * c.get("scale", 1.0) for e in chosen}


def mixture(x, p, c):
    """Routed experts and the gated shared expert of x [n, width]."""
    out = []
    for row in x:
        y = torch.zeros_like(row)
        for e, w in route(row @ p["router"].T, p["correction"], c["router"]).items():
            y = y + w * expert(row, sub(p, f"e{e}."))
        if c.get("shared"):
            y = y + torch.sigmoid(row @ p["shared.sg"][0]) * expert(row, sub(p, "shared."))
        out.append(y)
    return torch.stack(out)


def feed_forward(x, p, c):
    return mixture(x, p, c) if c["kind"] == "moe" else dense(x, p)


def forward(cfg, w, ids, dtype=torch.float64, collect=None, rounded=False):
    """Logits [n, vocab] of one sequence; ``collect`` receives the stream after every layer.  ``rounded``: what
    enters and leaves a sub-layer is rounded to bf16."""
    def cast(t):
        return t.to(torch.bfloat16).to(dtype) if rounded else t
    w = {k: t.to(dtype) for k, t in w.items()}
    x = w["embed"][torch.as_tensor(ids, dtype=torch.int64)]
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    known = {}                       # layer -> its latents and rotated keys
    for i, L in enumerate(cfg["layers"]):
        p, c = sub(w, f"l{i}."), L["mixer"]
        mix = sub(p, "mix.")
        if L["type"] == "latent_attention" and c.get("kv_from") is None:
            known[i] = latents(cast(x), mix, c, eps)
        y = MIXERS[L["type"]](cast(x), mix, c, eps, known.get(i if c.get("kv_from") is None else c["kv_from"]))
        x = x + m * output_norm(cast(y), p["norm1"], eps)
        if L["mlp"] is not None:
            x = x + m * output_norm(cast(feed_forward(cast(x), sub(p, "mlp."), L["mlp"])), p["norm2"], eps)
        if collect is not None:
            collect.append(x)
    return cast(output_norm(x, w["final.norm"], eps)) @ w["embed"].T
