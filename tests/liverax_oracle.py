"""Plain, slow Liverax: one function per mechanism, whole sequences only, float64 throughout, no cache. The tests compare
the framework with it; it shares no code with the product path.

`cfg` is the parsed config.json, `wt` a dict name -> tensor (any float type)."""
import math

import torch

F64 = torch.float64


def W(wt, name):
    return wt[name].to(F64)


def linear(h, wt, name):
    y = h @ W(wt, name).T
    return y + W(wt, name + ".b") if name + ".b" in wt else y


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# -- positions -------------------------------------------------------------------------------------
def frequencies(rot):
    """One angle step per pair; a linear scaling divides them all."""
    n = int(rot["dims"]) // 2
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    return [float(rot["base"]) ** (-2.0 * i / int(rot["dims"])) / factor for i in range(n)]


def rotate(x, freqs):
    """x [T, heads, d] at positions 0..T-1: entry i turns with entry i + len(freqs); what lies behind passes."""
    n = len(freqs)
    if n == 0:
        return x
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def bucket(n, rows, dmax):
    """Row of the distance table: the first half one row per distance, the rest logarithmic up to dmax."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(dmax / half) * (rows - half)))


def distance_bias(rel, t, dmax):
    """rel [rows, H] -> [H, T, T] (0 above the diagonal, which no query sees)."""
    per_distance = torch.stack([rel[bucket(n, rel.shape[0], dmax)] for n in range(t)])
    d = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return torch.where(d >= 0, per_distance[d.clamp(min=0)].permute(2, 0, 1), 0.0)


def temperature(t, q_temp):
    return torch.tensor([1.0 + float(q_temp["coef"]) * math.log(math.floor((p + 1) / q_temp["every"]) + 1)
                         for p in range(t)], dtype=F64)


def visible(t, window=None):
    d = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < int(window))


# -- attention -------------------------------------------------------------------------------------
def softmax_heads(q, k, v, scale, seen, bias=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], seen [T, T] bool, bias [H, T, T], sink [H] -> [T, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s + bias[h]
        s = s.masked_fill(~seen, float("-inf"))
        top = s.max(-1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[h]))
        e = torch.exp(s - top)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (e / den) @ v[:, g]
    return out


def mixed_values(v, lam, first):
    """`first` is a one-entry store that the first mixing layer fills with its own values."""
    if "v" not in first:
        first["v"] = v
        return v
    return (1.0 - lam) * v + lam * first["v"]


def heads_of(h, m, wt, pre):
    t = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    return (linear(h, wt, pre + "q").reshape(t, H, d), linear(h, wt, pre + "k").reshape(t, G, d),
            linear(h, wt, pre + "v").reshape(t, G, dv))


def rotary_window_attention(h, m, wt, pre, eps, first):
    q, k, v = heads_of(h, m, wt, pre)
    f = frequencies(m["rot"])
    if m.get("v_mix"):
        v = mixed_values(v, W(wt, pre + "vmix"), first)
    o = softmax_heads(rotate(q, f), rotate(k, f), v, float(m["scale"]), visible(h.shape[0], m["mask"]["size"]))
    return linear(o.reshape(h.shape[0], -1), wt, pre + "o")


def distance_attention(h, m, wt, pre, eps, first):
    t = h.shape[0]
    q, k, v = heads_of(h, m, wt, pre)
    q = (rms(q.reshape(t, -1), eps) * W(wt, pre + "q.norm")).reshape(q.shape)
    k = (rms(k.reshape(t, -1), eps) * W(wt, pre + "k.norm")).reshape(k.shape)
    if m.get("q_temp"):
        q = q * temperature(t, m["q_temp"])[:, None, None]
    if m.get("v_mix"):
        v = mixed_values(v, W(wt, pre + "vmix"), first)
    o = softmax_heads(q, k, v, float(m["scale"]), visible(t), distance_bias(W(wt, pre + "rel"), t, m["bias_max"]))
    return linear(o.reshape(t, -1) * sigmoid(linear(h, wt, pre + "g")), wt, pre + "o")


def latent_attention(h, m, wt, pre, eps, first=None):
    t = h.shape[0]
    H, d, rd, dv, r = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    cq = rms(linear(h, wt, pre + "dq"), eps) * W(wt, pre + "dq.norm")
    q = linear(cq, wt, pre + "uq").reshape(t, H, d + rd)
    kv = linear(h, wt, pre + "dkv")
    c = rms(kv[:, :r], eps) * W(wt, pre + "dkv.norm")
    f = frequencies(m["rot"])
    kr = rotate(kv[:, None, r:], f)
    q = torch.cat([q[..., :d], rotate(q[..., d:], f)], -1)
    k = torch.cat([linear(c, wt, pre + "uk").reshape(t, H, d), kr.expand(t, H, rd)], -1)
    v = linear(c, wt, pre + "uv").reshape(t, H, dv)
    o = softmax_heads(q, k, v, float(m["scale"]), visible(t, m["mask"]["size"]), sink=W(wt, pre + "sink"))
    return linear(o.reshape(t, -1) * sigmoid(linear(h, wt, pre + "g")), wt, pre + "o")


MIXERS = {"attention": rotary_window_attention, "attention_2": distance_attention, "latent_attention": latent_attention}


# -- the rest --------------------------------------------------------------------------------------
def feed_forward(h, wt, pre):
    return linear(gelu_tanh(linear(h, wt, pre + "gate")) * linear(h, wt, pre + "up"), wt, pre + "down")


def capped(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg, wt, tokens, trace=None):
    """-> logits [T, vocab] float64; `trace` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x, first = W(wt, "embed")[list(tokens)], {}
    for i, L in enumerate(cfg["layers"]):
        pre = "l%d." % i
        x = x + MIXERS[L["type"]](layer_norm(x, W(wt, pre + "norm1"), eps), L["mixer"], wt, pre + "mix.", eps, first)
        if L.get("mlp") is not None:
            x = x + feed_forward(layer_norm(x, W(wt, pre + "norm2"), eps), wt, pre + "mlp.")
        if trace is not None:
            trace.append(x.clone())
    return capped(layer_norm(x, W(wt, "final.norm"), eps) @ W(wt, "head").T, float(cfg.get("logit_softcap") or 0.0))
