"""Plain definitions of the mechanisms of the Pegopel decoder, for tests: token by token, one function per
mechanism, torch on the CPU in the precision of the given weights (float64 by default).  Nothing here is
shared with the package; what the Vofelix definitions already say is taken from there."""
import math

import torch

from vofelix_oracle import feed_forward, rms_norm, rotate, short_conv, sub


def distance_bucket(n, rows, largest):
    """Bucket of the distance ``n`` >= 0 in a table of ``rows`` rows: one each for the near half, then
    logarithmic up to ``largest``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(largest / half) * (rows - half)))


def visible(i, j, size=None, keep_first=0):
    """Whether position ``i`` sees position ``j``."""
    return j <= i and (size is None or i - j < size or j < keep_first)


def softmax_with_sink(s, sink):
    """s [heads, keys]; exp(sink[h]) is one more term of head h's denominator."""
    top = torch.maximum(s.max(-1).values, sink)[:, None]
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None] - top))


def attend(q, k, v, scale, size=None, keep_first=0, softcap=None, bias=None, largest=None, sink=None, rows=None):
    """q [n, H, d], k [n, G, d], v [n, G, vd] of one whole sequence -> [n, H, vd].  ``bias`` [buckets, H];
    ``rows``: positions to compute (all)."""
    n, H, _ = q.shape
    owner = [h // (H // k.shape[1]) for h in range(H)]          # key / value head of a query head
    k, v = k[:, owner], v[:, owner]
    row = None if bias is None else torch.tensor([distance_bucket(m, bias.shape[0], largest) for m in range(n)])
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n) if rows is None else rows:
        js = torch.tensor([j for j in range(n) if visible(i, j, size, keep_first)])
        s = torch.einsum("hd,jhd->hj", q[i], k[js]) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        if bias is not None:
            s = s + bias[row[i - js]].T
        w = torch.softmax(s, -1) if sink is None else softmax_with_sink(s, sink)
        out[i] = torch.einsum("hj,jhv->hv", w, v[js])
    return out


def biased_attention(h, p, c, eps):
    """Mixer with short convolutions on q, k and v, a distance bias and a learned sink."""
    n, H, G, d, vd = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_conv(h @ p[x].T, p[x + ".conv"]) for x in "qkv")
    q, k = rms_norm(q, p["q.norm"], eps), rms_norm(k, p["k.norm"], eps)
    o = attend(q.view(n, H, d), k.view(n, G, d), v.view(n, G, vd), c["scale"], c["mask"]["size"], bias=p["rel"],
               largest=c["bias_max"], sink=p["sink"])
    return o.reshape(n, H * vd) @ p["o"].T


def gated_attention(h, p, c, eps):
    """Mixer with rotary positions whose values are the raw keys, capped scores, kept first tokens, one added
    to the denominator and an output gate per head."""
    n, H, G, d = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    rot = c["rot"]
    raw = h @ p["k"].T
    q, k = rms_norm(h @ p["q"].T, p["q.norm"], eps).view(n, H, d), rms_norm(raw, p["k.norm"], eps).view(n, G, d)
    q, k = (torch.stack([rotate(t[i], i, rot["dims"], rot["base"], rot.get("scaling")) for i in range(n)]) for t in (q, k))
    o = attend(q, k, raw.view(n, G, d), c["scale"], c["mask"]["size"], c["mask"]["keep_first"], c["softcap"],
               sink=torch.zeros(H, dtype=h.dtype))
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(n, H * d) @ p["o"].T


MIXERS = {"attention": biased_attention, "attention_2": gated_attention}


def mix_streams(x, y, p):
    """x [s, n, w] streams, y [n, w] a sub-layer's output -> the new streams."""
    return torch.einsum("snw,st->tnw", x, p["mix"]) + p["out"][:, None, None] * y


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, w, ids, dtype=torch.float64, collect=None, rounded=False):
    """Logits [n, vocab] of one sequence; ``collect`` receives the sum of the streams after every layer run.
    ``rounded``: what enters and leaves a sub-layer is rounded to bf16."""
    def cast(t):
        return t.to(torch.bfloat16).to(dtype) if rounded else t
    w = {k: t.to(dtype) for k, t in w.items()}
    ids = torch.as_tensor(ids, dtype=torch.int64)
    eps = cfg["norm"]["eps"]
    x = (w["embed"][ids] + w["pos"][:len(ids)])[None].repeat(cfg["streams"], 1, 1)
    for i in layer_order(cfg):
        L, p = cfg["layers"][i], sub(w, f"l{i}.")

        def sublayer(x, which, f):
            hc = sub(p, f"hc{which}.")
            u = torch.einsum("s,snw->nw", hc["in"], x)
            return mix_streams(x, cast(f(cast(rms_norm(u, p[f"norm{which}"], eps)))), hc)
        x = sublayer(x, 1, lambda h: MIXERS[L["type"]](h, sub(p, "mix."), L["mixer"], eps))
        if L["mlp"] is not None:
            x = sublayer(x, 2, lambda h: feed_forward(h, sub(p, "mlp.")))
        if collect is not None:
            collect.append(x.sum(0))
    return cast(rms_norm(x.sum(0), w["final.norm"], eps)) @ w["embed"].T
