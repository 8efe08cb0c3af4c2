"""Plain definitions of the mechanisms of the Nevotar decoder, for tests: token by token, one function per
mechanism, torch on the CPU in the precision of the given weights (float64 by default).  Nothing here is
shared with the package; what the definitions of other designs already say is taken from there."""
import math

import torch

from dubizen_oracle import rotate_halves
from vofelix_oracle import rms_norm, silu, softplus, sub


def group_norm(x, w, eps, groups):
    """RMS norm of ``groups`` equal consecutive parts, each by itself."""
    size = x.shape[-1] // groups
    parts = [x[..., g * size:(g + 1) * size] for g in range(groups)]
    return torch.cat([t / torch.sqrt((t ** 2).mean(-1, keepdim=True) + eps) for t in parts], -1) * w


def softmax_rows(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def query_temperature(pos, coef, every):
    return 1 + coef * math.log(math.floor((pos + 1) / every) + 1)


def difference_of_maps(q, k, v, scale, lam, diff, eps, temp=None):
    """q [n, H, 2, d], k [n, G, 2, d], v [n, G, vd] -> [n, H, vd]: softmax map 1 minus ``lam`` times softmax map 2,
    RMS-normed per head without a weight, times 1 - diff.  ``temp``: (coef, every) or None."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        f = query_temperature(i, *temp) if temp else 1.0
        for h in range(H):
            g = h // (H // G)
            a = [softmax_rows((k[:i + 1, g, m] @ (q[i, h, m] * f)) * scale) @ v[:i + 1, g] for m in (0, 1)]
            o = a[0] - lam * a[1]
            out[i, h] = o / torch.sqrt((o ** 2).mean() + eps) * (1 - diff)
    return out


_rounding = [False]


def cast(t):
    """What a 16-bit engine stores between two operations (``forward`` with ``rounded``)."""
    return t.to(torch.bfloat16).to(t.dtype) if _rounding[0] else t


def projection(h, p, name, heads, size):
    return cast(h @ p[name].T + p[name + ".b"]).view(h.shape[0], heads, size)


def difference_attention(h, p, c, eps):
    n, H, G, d, vd = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k = projection(h, p, "q", H, 2 * d).view(n, H, 2, d), projection(h, p, "k", G, 2 * d).view(n, G, 2, d)
    v = projection(h, p, "v", G, vd)
    lam = torch.exp((p["lq1"] * p["lk1"]).sum()) - torch.exp((p["lq2"] * p["lk2"]).sum()) + c["diff"]
    t = c.get("q_temp")
    o = difference_of_maps(q, k, v, c["scale"], lam, c["diff"], eps, (t["coef"], t["every"]) if t else None)
    return o.reshape(n, H * vd) @ p["o"].T


def talking_attention(q, k, v, scale, mix, size):
    """q [n, H, d], k [n, G, d], v [n, G, vd] -> [n, H, vd]: the scaled scores of all heads are mixed by
    ``mix`` [H, H] before the softmax; position i sees the last ``size`` tokens, itself included."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    owner = [h // (H // G) for h in range(H)]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = max(0, i - size + 1)
        s = mix @ (torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1, owner]) * scale)
        out[i] = torch.einsum("hj,jhv->hv", softmax_rows(s), v[lo:i + 1, owner])
    return out


def windowed_attention(h, p, c, eps):
    n, H, G, d, vd, rot = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"], c["rot"]
    q, k = (rms_norm(projection(h, p, x, heads, d), p[x + ".norm"], eps) for x, heads in (("q", H), ("k", G)))
    q, k = (torch.stack([rotate_halves(t[i], i, rot["dims"], rot["base"]) for i in range(n)]) for t in (q, k))
    o = talking_attention(q, k, projection(h, p, "v", G, vd), c["scale"], p["talk"], c["mask"]["size"])
    return o.reshape(n, H * vd) @ p["o"].T


def state_space(x, B, C, dt, A_log, D):
    """x [n, H, P], B, C [n, G, N], dt [n, H] (after the softplus) -> y [n, H, P], and the last state."""
    n, H, P = x.shape
    own = [h // (H // B.shape[1]) for h in range(H)]
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(n):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + (dt[t][:, None] * B[t, own])[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t, own]) + D[:, None] * x[t]
    return y, S


def mamba(h, p, c, eps):
    n, H, P, N, G = h.shape[0], c["heads"], c["vdim"], c["state"], c["groups"]
    inner, gn = H * P, G * N
    u = cast(h @ p["in"].T)
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * gn], u[:, 2 * inner + 2 * gn:]
    xbc = cast(conv_silu(xbc, p["conv"], p["conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + gn], xbc[:, inner + gn:]
    y, _ = state_space(x.reshape(n, H, P), B.reshape(n, G, N), C.reshape(n, G, N), softplus(dt + p["dt_bias"]), p["A_log"],
                       p["D"])
    return group_norm(y.reshape(n, inner) * silu(z), p["norm"], eps, c["norm_groups"]) @ p["o"].T


def conv_silu(x, w, b):
    """Causal convolution per channel (last column: the current token's weight) with a bias, then SiLU."""
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            if t - (taps - 1) + j >= 0:
                out[t] += w[:, j] * x[t - (taps - 1) + j]
    return silu(out + b)


def side_by_side(h, p, c, eps):
    return (c["left_scale"] * windowed_attention(h, sub(p, "left."), c["left"], eps) +
            c["right_scale"] * mamba(h, sub(p, "right."), c["right"], eps))


def forget_recurrence(q, f, v):
    """q, f [n, H, d], v [n, H, vd]: what the gate lets go of is what the value replaces."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(n):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def hgrn2(h, p, c, eps):
    n, H, d, vd = h.shape[0], c["heads"], c["dim"], c["vdim"]
    low = p["lower"]
    f = low + (1 - low) / (1 + torch.exp(-(cast(h @ p["f"].T) + p["f.b"])))
    q, v = cast(h @ p["q"].T), cast(h @ p["v"].T)
    o, _ = forget_recurrence(silu(q).view(n, H, d), f.view(n, H, d), v.view(n, H, vd))
    return rms_norm(o, p["norm"], eps).reshape(n, H * vd) @ p["o"].T


MIXERS = {"attention": difference_attention, "parallel": side_by_side, "hgrn2": hgrn2}


def clamped_expert(x, p, limit):
    g = torch.clamp(x @ p["gate"].T, max=limit)
    u = torch.clamp(x @ p["up"].T, -limit, limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ p["down"].T


def route(z, top):
    """One token's router: {expert: weight}, the largest sigmoid scores as they are."""
    s = [1 / (1 + math.exp(-float(v))) for v in z]
    return {e: s[e] for e in sorted(range(len(s)), key=lambda e: -s[e])[:top]}


def mixture(x, p, c):
    """The chosen experts work on the weighted input; the shared expert on the input."""
    out = []
    for row in x:
        y = torch.zeros_like(row)
        for e, w in route(row @ p["router"].T, c["router"]["top"]).items():
            y = y + clamped_expert(w * row, sub(p, f"e{e}."), c["expert"]["limit"])
        if c.get("shared"):
            y = y + clamped_expert(row, sub(p, "shared."), c["shared"]["limit"])
        out.append(y)
    return torch.stack(out)


def forward(cfg, w, ids, dtype=torch.float64, collect=None, rounded=False):
    """Logits [n, vocab] of one sequence; ``collect`` receives the stream after every layer.  ``rounded``: what
    enters and leaves a sub-layer, and the projections inside, are rounded to bf16."""
    _rounding[0] = rounded
    try:
        w = {k: t.to(dtype) for k, t in w.items()}
        x = w["embed"][torch.as_tensor(ids, dtype=torch.int64)]
        eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
        for i, L in enumerate(cfg["layers"]):
            p = sub(w, f"l{L.get('weights_of', i)}.")
            x = x + cast(MIXERS[L["type"]](cast(group_norm(x, p["norm1"], eps, groups)), sub(p, "mix."), L["mixer"], eps))
            if L["mlp"] is not None:
                x = x + cast(mixture(cast(group_norm(x, p["norm2"], eps, groups)), sub(p, "mlp."), L["mlp"]))
            if collect is not None:
                collect.append(x)
        return cast(group_norm(x, w["final.norm"], eps, groups)) @ w["embed"].T
    finally:
        _rounding[0] = False
