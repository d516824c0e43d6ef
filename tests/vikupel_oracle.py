"""Plain, slow Vikupel: one function per mechanism, whole sequences only, float64 throughout, no cache. The tests
compare the framework with it; it shares no code with the product path.

`cfg` is the parsed config.json, `wt` a dict name -> tensor (any float type)."""
import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def W(wt, name):
    return wt[name].to(F64)


def linear(h, wt, name):
    return h @ W(wt, name).T


# -- Mamba-2 ---------------------------------------------------------------------------------------
def causal_conv(u, w, b):
    """u [T, C], w [C, taps] with the current token's tap last, b [C]."""
    t, taps = u.shape[0], w.shape[1]
    out = b.expand(t, -1).clone()
    for i in range(t):
        for j in range(taps):
            src = i - (taps - 1) + j
            if src >= 0:
                out[i] += w[:, j] * u[src]
    return out


def ssd_scan(x, B, C, dt, a_log, dskip):
    """x [T, H, V], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, V], one token at a time."""
    t, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    S = torch.zeros(H, N, V, dtype=F64)
    y = torch.zeros(t, H, V, dtype=F64)
    for i in range(t):
        for h in range(H):
            g = h // (H // G)
            S[h] = math.exp(-math.exp(float(a_log[h])) * float(dt[i, h])) * S[h] \
                + float(dt[i, h]) * torch.outer(B[i, g], x[i, h])
            y[i, h] = S[h].T @ C[i, g] + dskip[h] * x[i, h]
    return y


def gated_norm(y, z, w, groups, eps):
    v = y * silu(z)
    t, n = v.shape
    return rms(v.reshape(t, groups, n // groups), eps).reshape(t, n) * w


def mamba2(h, m, wt, pre, eps):
    t = h.shape[0]
    H, V, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner = H * V
    p = linear(h, wt, pre + "in")
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, W(wt, pre + "conv"), W(wt, pre + "conv.b")))
    x = xbc[:, :inner].reshape(t, H, V)
    B = xbc[:, inner:inner + G * N].reshape(t, G, N)
    C = xbc[:, inner + G * N:].reshape(t, G, N)
    dt = torch.log1p(torch.exp(dt + W(wt, pre + "dt_bias")))
    y = ssd_scan(x, B, C, dt, W(wt, pre + "A_log"), W(wt, pre + "D")).reshape(t, inner)
    return linear(gated_norm(y, z, W(wt, pre + "norm"), int(m["norm_groups"]), eps), wt, pre + "o")


# -- softmax attention -----------------------------------------------------------------------------
def softmax_heads(q, k, v, scale, visible, bias=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; visible [T, T] bool; bias(h) -> [T, T] taken off the scores."""
    t, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(t, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if bias is not None:
            s = s - bias(h)
        s = s.masked_fill(~visible, float("-inf"))
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, g]
    return out


def distances(t):
    i = torch.arange(t)
    return i[:, None] - i[None, :]


def distance_attention(h, m, wt, pre, eps=None):
    """Sliding window, logarithmic distance bias per head, sigmoid output gate, no rotation."""
    t = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = linear(h, wt, pre + "q").reshape(t, H, d)
    k = linear(h, wt, pre + "k").reshape(t, G, d)
    v = linear(h, wt, pre + "v").reshape(t, G, dv)
    dist = distances(t)
    visible = (dist >= 0) & (dist < int(m["mask"]["size"]))
    r1, r2 = W(wt, pre + "r1"), W(wt, pre + "r2")
    far = dist.clamp(min=0).to(F64)
    o = softmax_heads(q, k, v, float(m["scale"]), visible, lambda a: r1[a] * torch.log(1.0 + r2[a] * far))
    o = o.reshape(t, H * dv) / (1.0 + torch.exp(-linear(h, wt, pre + "g")))
    return linear(o, wt, pre + "o")


def frequencies(dims, base, scaling=None):
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            fac, lo, hi, orig = (float(scaling[n]) for n in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave < orig / hi:
                pass
            elif wave > orig / lo:
                f = f / fac
            else:
                s = (orig / wave - lo) / (hi - lo)
                f = (1.0 - s) * f / fac + s * f
        out.append(f)
    return out


def rotate(x, freqs, sign=1.0):
    """x [T, heads, d]: entry i turns with entry i + len(freqs) by position * freqs[i]; the rest passes."""
    t, n = x.shape[0], len(freqs)
    if n == 0:
        return x
    ang = torch.arange(t, dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :] * sign
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def rotated_value_attention(h, m, wt, pre, eps):
    """Causal attention; q and k rotated, then unit root mean square per head; values rotated by their position,
    the result turned back by the query's."""
    t = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    rot = m["rot"]
    f = frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
    q = rms(rotate(linear(h, wt, pre + "q").reshape(t, H, d), f), eps)
    k = rms(rotate(linear(h, wt, pre + "k").reshape(t, G, d), f), eps)
    fv = frequencies(dv, float(rot["base"]))
    v = rotate(linear(h, wt, pre + "v").reshape(t, G, dv), fv)
    o = softmax_heads(q, k, v, float(m["scale"]), distances(t) >= 0)
    return linear(rotate(o, fv, -1.0).reshape(t, H * dv), wt, pre + "o")


MIXERS = {"mamba2": mamba2, "attention": distance_attention, "attention_2": rotated_value_attention}


# -- the rest --------------------------------------------------------------------------------------
def feed_forward(h, wt, pre):
    return linear(silu(linear(h, wt, pre + "gate")) * linear(h, wt, pre + "up"), wt, pre + "down")


def token_side(x, tokens, i, dim, wt, pre, eps):
    """The layer's own embedding of the token, gated by the stream; the normed result is added to the stream."""
    e = W(wt, "side.embed")[list(tokens)][:, i * dim:(i + 1) * dim]
    g = gelu_tanh(linear(x, wt, pre + "gate")) * e
    return rms(linear(g, wt, pre + "proj"), eps) * W(wt, pre + "norm")


def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def forward(cfg, wt, tokens, trace=None):
    """-> logits [T, vocab] float64; `trace` (a list) receives the stream after every layer run."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    side = cfg.get("token_side")
    x = W(wt, "embed")[list(tokens)]
    for i in layer_order(cfg):
        L, pre = cfg["layers"][i], f"l{i}."
        h = rms(x, eps) * W(wt, pre + "norm1")
        y = MIXERS[L["type"]](h, L["mixer"], wt, pre + "mix.", eps)
        if L.get("mlp") is not None:
            y = y + feed_forward(h, wt, pre + "mlp.")
        x = x + mult * y
        if side:
            x = x + mult * token_side(x, tokens, i, int(side["dim"]), wt, pre + "side.", eps)
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * W(wt, "final.norm")) @ W(wt, "head").T
