"""A slow, plain implementation of the Vunitar design, one function per mechanism, for the tests to compare the
framework with.  It works on a dictionary of tensors and the configuration dictionary, on whole sequences, without a
cache, in the dtype of the tensors it is given (tests use float64).  It shares no code with the package."""
import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def embed(tokens, table, bigram=None, consts=None):
    """Token rows plus, for every token, the row of the (previous, current) pair; row ``buckets`` starts a sequence."""
    rows = []
    for i, t in enumerate(tokens):
        x = table[t]
        if bigram is not None:
            n = consts["buckets"]
            r = n if i == 0 else (tokens[i - 1] * consts["mul_prev"] + t * consts["mul_cur"]) % n
            x = x + bigram[r]
        rows.append(x)
    return torch.stack(rows)


def latent(h, w, eps):
    return rms(h @ w["dkv"].t(), w["dkv.norm"], eps)


def latent_attention(h, w, m, eps):
    """Causal softmax attention whose keys and values are per-head linear maps of one normalised latent per token."""
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c = latent(h, w, eps)
    q = (h @ w["q"].t()).view(n, H, d)
    k = (c @ w["uk"].t()).view(n, H, d)
    v = (c @ w["uv"].t()).view(n, H, dv)
    out = []
    for i in range(n):
        heads = []
        for a in range(H):
            s = (k[: i + 1, a] @ q[i, a]) * m["scale"]
            p = torch.exp(s - s.max())
            heads.append((p / p.sum()) @ v[: i + 1, a])
        out.append(torch.cat(heads))
    return torch.stack(out) @ w["o"].t()


def dense_ff(h, w):
    return relu_squared(h @ w["up"].t()) @ w["down"].t()


def expert_ff(h, up, down):
    return gelu_erf(h @ up.t()) @ down.t()


def route(h, w_router, r, margins=None):
    """Chosen experts and weights per token: [(expert, weight), ...].  ``margins`` collects, per token, by how much (in
    logits) the closest decision was taken."""
    picks = []
    for z in h @ w_router.t():
        s = torch.softmax(z, 0)
        E = s.numel()
        allowed = set(range(E))
        g = r.get("groups")
        if g:
            size = E // g["count"]
            ranked = sorted(range(g["count"]), key=lambda i: -float(s[i * size:(i + 1) * size].max()))
            best = ranked[: g["keep"]]
            allowed = {e for i in best for e in range(i * size, (i + 1) * size)}
        ordered = sorted(allowed, key=lambda e: -float(s[e]))
        order = ordered[: r["top"]]
        if margins is not None:
            gap = float(z[order[-1]] - z[ordered[len(order)]]) if len(ordered) > len(order) else math.inf
            if g and g["keep"] < g["count"]:
                top = lambda i: float(z[i * size:(i + 1) * size].max())
                gap = min(gap, top(best[-1]) - top(ranked[g["keep"]]))
            margins.append(gap)
        picks.append([(e, s[e] * r["scale"]) for e in order])
    return picks


def moe_ff(h, w, mlp, margins=None):
    rows = []
    for x, pick in zip(h, route(h, w["router"], mlp["router"], margins)):
        y = torch.zeros_like(x)
        for e, g in pick:
            y = y + g * expert_ff(x[None], w[f"e{e}.up"], w[f"e{e}.down"])[0]
        if mlp.get("shared"):
            y = y + torch.sigmoid(w["shared.sg"] @ x) * expert_ff(x[None], w["shared.up"], w["shared.down"])[0]
        rows.append(y)
    return torch.stack(rows)


def softcap(logits, cap):
    return logits if not cap else cap * torch.tanh(logits / cap)


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None, margins_out=None):
    """Logits [tokens, vocab]; ``layers_out`` collects the residual stream after every layer, ``margins_out`` the routers'
    margins per expert layer."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, weights["embed"], weights.get("bigram"), (cfg.get("embedding") or {}).get("bigram"))
    for i, layer in enumerate(cfg["layers"]):
        w = sub(weights, f"l{i}.")
        x = x + rms(latent_attention(x, sub(w, "mix."), layer["mixer"], eps), w["norm1"], eps) * w["ls1"]
        mlp = layer["mlp"]
        if mlp is not None:
            margins = []
            y = dense_ff(x, sub(w, "mlp.")) if mlp["kind"] == "dense" else moe_ff(x, sub(w, "mlp."), mlp, margins)
            if margins and margins_out is not None:
                margins_out.append(margins)
            x = x + rms(y, w["norm2"], eps) * w["ls2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return softcap(rms(x, weights["final.norm"], eps) @ weights["head"].t(), cfg.get("logit_softcap"))
