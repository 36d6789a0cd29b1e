"""A slow, plain implementation of the Lisunex design, one function per mechanism, for the tests to compare the
framework with.  It works on a dictionary of tensors and the configuration dictionary, on whole sequences, without a
cache, in the dtype of the tensors it is given (tests use float64).  It shares no code with the package."""
import math

import torch


def rms(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z / (1.0 + torch.exp(-z))


def embed(tokens, table, scale):
    return torch.stack([table[t] for t in tokens]) * scale


# ------------------------------------------------------------------ recurrence
def short_conv(x, taps):
    """``x[n, channels]``, ``taps[channels, K]``: the last tap meets the current token, zeros before the start."""
    n, K = x.shape[0], taps.shape[1]
    out = torch.zeros_like(x)
    for i in range(n):
        for j in range(K):
            t = i - (K - 1) + j
            if t >= 0:
                out[i] = out[i] + x[t] * taps[:, j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """One head, token by token: ``q, k[n, d]``, ``v[n, dv]``, ``beta, g[n]`` -> outputs ``[n, dv]`` and the last state."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = []
    for i in range(v.shape[0]):
        S = g[i] * S
        u = beta[i] * (v[i] - S.t() @ k[i])
        S = S + torch.outer(k[i], u)
        out.append(S.t() @ q[i])
    return torch.stack(out), S


def decay(z, a_log, dt_bias):
    s = z + dt_bias
    softplus = torch.where(s > 30, s, torch.log1p(torch.exp(torch.clamp(s, max=30))))
    return torch.exp(-torch.exp(a_log) * softplus)


def delta_mixer(h, w, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(short_conv(h @ w["q"].t(), w["q.conv"])).view(n, G, d)) / math.sqrt(d)
    k = unit(silu(short_conv(h @ w["k"].t(), w["k.conv"])).view(n, G, d))
    v = silu(short_conv(h @ w["v"].t(), w["v.conv"])).view(n, H, dv)
    beta = 1.0 / (1.0 + torch.exp(-(h @ w["b"].t())))
    g = decay(h @ w["a"].t(), w["A_log"], w["dt_bias"])
    heads = []
    for a in range(H):
        j = a // (H // G)
        o, _ = delta_rule(q[:, j], k[:, j], v[:, a], beta[:, a], g[:, a])
        heads.append(rms(o, w["norm"], eps))
    o = torch.cat(heads, -1) * silu(h @ w["g"].t())
    return o @ w["o"].t()


# ------------------------------------------------------------------ attention
def frequencies(rot):
    """Angle per position of every rotated pair, and the factor on cosine and sine."""
    D, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    out, mult = [], 1.0
    if sc:
        where = lambda turns: D * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), D - 1)
        mult = 0.1 * math.log(sc["factor"]) + 1.0
    for i in range(D // 2):
        f = base ** (-2.0 * i / D)
        if sc:
            r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / sc["factor"] * r + f * (1.0 - r)
        out.append(f)
    return out, mult


def rotate(x, rot, first=0):
    """``x[n, heads, dim]`` at positions ``first ..``; pairs are (i, i + dims / 2)."""
    freq, mult = frequencies(rot)
    half = rot["dims"] // 2
    y = x.clone()
    for p in range(x.shape[0]):
        for i, f in enumerate(freq):
            c, s = mult * math.cos((first + p) * f), mult * math.sin((first + p) * f)
            u, v = x[p, :, i], x[p, :, i + half]
            y[p, :, i] = u * c - v * s
            y[p, :, i + half] = v * c + u * s
    return y


def visible(i, j, size):
    return j <= i and (not size or i // size == j // size)


def attend(q, k, v, scale, softcap, size, first=0):
    """``q[n, H, d]`` at positions ``first ..`` against ``k[t, G, d]``, ``v[t, G, dv]`` at positions 0 ..: softmax over the
    visible keys of ``softcap * tanh(score / softcap)``."""
    n, H = q.shape[:2]
    G = k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=v.dtype)
    for i in range(n):
        see = [j for j in range(k.shape[0]) if visible(first + i, j, size)]
        lo, hi = see[0], see[-1] + 1                   # the visible keys are neighbours
        assert len(see) == hi - lo
        for a in range(H):
            s = (k[lo:hi, a // (H // G)] @ q[i, a]) * scale
            if softcap:
                s = softcap * torch.tanh(s / softcap)
            p = torch.exp(s - s.max())
            out[i, a] = (p / p.sum()) @ v[lo:hi, a // (H // G)]
    return out


def attention_mixer(h, w, m, eps):
    n, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].t() + w["q.b"]).view(n, H, d)
    k = (h @ w["k"].t() + w["k.b"]).view(n, G, d)
    v = (h @ w["v"].t() + w["v.b"]).view(n, G, dv)
    q, k = rms(rotate(q, m["rot"]), None, eps), rms(rotate(k, m["rot"]), None, eps)
    o = attend(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    o = o / (1.0 + torch.exp(-(h @ w["g"].t())))[..., None]
    return o.reshape(n, H * dv) @ w["o"].t()


# ------------------------------------------------------------------ the model
def dense_ff(h, w):
    return (silu(h @ w["gate"].t()) * (h @ w["up"].t())) @ w["down"].t()


def runs(cfg):
    """(layer, pass of the loop that begins right before it or None), in the order of execution."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"delta": delta_mixer, "attention": attention_mixer}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [tokens, vocab]; ``layers_out`` collects the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, weights["embed"], cfg["embedding"]["scale"])
    for i, t in runs(cfg):
        layer, w = cfg["layers"][i], sub(weights, f"l{i}.")
        if t is not None:
            x = x + weights["loop.step"][t]
        x = x + MIXERS[layer["type"]](rms(x, w["norm1"], eps), sub(w, "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + dense_ff(rms(x, w["norm2"], eps), sub(w, "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, weights["final.norm"], eps) @ weights["head"].t()
