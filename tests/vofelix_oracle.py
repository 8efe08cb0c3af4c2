"""Plain definitions of the mechanisms of the Vofelix decoder, for tests: token by token, one function
per mechanism, torch on the CPU in whatever precision the weights are given in (float64 by default).
Nothing here is shared with the package."""
import math

import torch


def layer_norm(x, w, b, eps):
    mu = x.mean(-1, keepdim=True)
    var = ((x - mu) ** 2).mean(-1, keepdim=True)
    return (x - mu) / torch.sqrt(var + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def rotary_frequencies(dims, base, scaling):
    """(frequencies [dims / 2], factor on cos and sin) with optional YaRN interpolation."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def turning_dim(turns):
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(turning_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turning_dim(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, pos, dims, base, scaling):
    """x [..., d] at position ``pos``: pairs (2i, 2i + 1) of the first ``dims`` entries are turned."""
    freqs, m = rotary_frequencies(dims, base, scaling)
    y = x.clone()
    for i, f in enumerate(freqs):
        c, s = math.cos(pos * f) * m, math.sin(pos * f) * m
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def latent_attention(h, p, c, eps):
    """h [n, width] of one whole sequence -> [n, width].  ``p``: tensors without the layer prefix."""
    n, H, d, r, vd, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    rot = c["rot"]
    q = (h @ p["q"].T).view(n, H, d + r)
    down = h @ p["dkv"].T
    lat = rms_norm(down[:, :rank], p["dkv.norm"], eps)
    keys = (lat @ p["uk"].T).view(n, H, d)
    vals = (lat @ p["uv"].T).view(n, H, vd)
    kr = torch.stack([rotate(down[j, rank:], j, rot["dims"], rot["base"], rot.get("scaling")) for j in range(n)])
    size = (c.get("mask") or {}).get("size") or n
    out = torch.zeros(n, H, vd, dtype=h.dtype)
    for i in range(n):
        qr = rotate(q[i, :, d:], i, rot["dims"], rot["base"], rot.get("scaling"))
        a = max(0, i - size + 1)
        s = (torch.einsum("hd,jhd->hj", q[i, :, :d], keys[a:i + 1]) + qr @ kr[a:i + 1].T) * c["scale"]
        sink = p["sink"][:, None]
        top = torch.maximum(s.max(-1, keepdim=True).values, sink)
        e = torch.exp(s - top)
        w = e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))
        out[i] = torch.einsum("hj,jhv->hv", w, vals[a:i + 1])
    return out.reshape(n, H * vd) @ p["o"].T


def short_conv(x, taps):
    """x [n, channels], taps [channels, K]: the last column meets the current token."""
    n, K = x.shape[0], taps.shape[1]
    pad = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return sum(pad[j:j + n] * taps[:, j] for j in range(K))


def unit(x):
    return x / torch.sqrt((x ** 2).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, beta, g, state=None):
    """q, k [n, H, d] (unit, q scaled), v [n, H, vd], beta, g [n, H] -> (o [n, H, vd], state [H, d, vd])."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def delta_mixer(h, p, c, eps):
    n, H, Hk, d, vd = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = silu(short_conv(h @ p["q"].T, p["q.conv"])).view(n, Hk, d)
    k = silu(short_conv(h @ p["k"].T, p["k.conv"])).view(n, Hk, d)
    v = silu(short_conv(h @ p["v"].T, p["v.conv"])).view(n, H, vd)
    owner = [hh // (H // Hk) for hh in range(H)]
    q, k = unit(q)[:, owner] * d ** -0.5, unit(k)[:, owner]
    beta = torch.sigmoid(h @ p["b"].T)
    g = torch.exp(-torch.exp(p["A_log"]) * softplus(h @ p["a"].T + p["dt_bias"]))
    o, _ = delta_scan(q, k, v, beta, g)
    o = rms_norm(o, p["norm"], eps) * silu(h @ p["g"].T).view(n, H, vd)
    return o.reshape(n, H * vd) @ p["o"].T


def feed_forward(x, p):
    return (gelu_tanh(x @ p["gate"].T) * (x @ p["up"].T)) @ p["down"].T


def token_side(x, ids, i, dim, table, p, eps):
    e = table[ids][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T
    return x + rms_norm(y, p["norm"], eps)


def layer_order(cfg):
    """Layer index of every run, and the set of runs before which the embedding output is added."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n)), set()
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = list(range(a))
    again = set()
    for t in range(times):
        if t:
            again.add(len(order))
        order += list(range(a, b))
    return order + list(range(b, n)), again


def sub(w, prefix):
    return {k[len(prefix):]: t for k, t in w.items() if k.startswith(prefix)}


def forward(cfg, w, ids, dtype=torch.float64, collect=None, rounded=False):
    """Logits [n, vocab] of one sequence; ``collect`` receives the stream after every layer run.  ``rounded``:
    what enters and leaves a sub-layer is rounded to bf16 (the size of the error that rounding causes)."""
    def cast(t):
        return t.to(torch.bfloat16).to(dtype) if rounded else t
    w = {k: t.to(dtype) if t.is_floating_point() else t for k, t in w.items()}
    ids = torch.as_tensor(ids, dtype=torch.int64)
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][ids] * cfg["embedding"]["scale"]
    x = x0
    order, again = layer_order(cfg)
    for run, i in enumerate(order):
        L, p = cfg["layers"][i], sub(w, f"l{i}.")

        def norm(name, t):
            return cast(layer_norm(cast(t) if name.endswith("b") else t, p[name], p[name + ".b"], eps))
        if run in again:
            x = x + x0
        mixer = {"latent_attention": latent_attention, "delta": delta_mixer}[L["type"]]
        x = x + norm("norm1b", mixer(norm("norm1", x), sub(p, "mix."), L["mixer"], eps))
        if L["mlp"] is not None:
            x = x + norm("norm2b", feed_forward(norm("norm2", x), sub(p, "mlp.")))
        if cfg.get("token_side"):
            x = token_side(x, ids, i, cfg["token_side"]["dim"], w["side.embed"], sub(p, "side."), eps)
        if collect is not None:
            collect.append(x)
    return cast(layer_norm(x, w["final.norm"], w["final.norm.b"], eps)) @ w["head"].T
