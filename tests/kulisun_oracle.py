"""Plain, slow statement of the Kulisun design in float64: one function per mechanism, whole sequences at once, no caches, no
kernels, nothing shared with the serving path.  Weights come as a dict of checkpoint tensors (``l<i>.mix.*`` etc.), configurations
as the ``config.json`` dict."""
import math

import torch

F64 = torch.float64


def lin(w, name, x):
    y = x @ w[name].to(F64).T
    return y + w[name + ".b"].to(F64) if name + ".b" in w else y


def layer_norm(w, name, x, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w[name].to(F64) + w[name + ".b"].to(F64)


def rms(x, g, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * g.to(F64)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rotation(rot):
    """(frequencies, amplitude): turns per coordinate pair, with the long-context interpolation where the configuration has one."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freqs, 1.0
    # the (fractional) pair index whose wave makes `turns` full turns over the original context length
    index = lambda turns: dims * math.log(sc["original"] / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))
    first = max(math.floor(index(sc["fast"])), 0)
    last = min(math.ceil(index(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        slowed = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(slowed * f / sc["factor"] + (1.0 - slowed) * f)
    return out, 1.0 + 0.1 * math.log(sc["factor"])


def rotate_halves(x, rot):
    """x [S, heads, D]: coordinates (i, i + dims/2) of every head turned by position * frequency; the rest untouched."""
    freqs, amp = rotation(rot)
    half = rot["dims"] // 2
    y = x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)
    for i, f in enumerate(freqs):
        c, s = (amp * torch.cos(pos * f))[:, None], (amp * torch.sin(pos * f))[:, None]
        y[:, :, i] = x[:, :, i] * c - x[:, :, i + half] * s
        y[:, :, i + half] = x[:, :, i + half] * c + x[:, :, i] * s
    return y


def latent_rows(m, w, p, h, eps):
    """What a layer keeps per token: the normed latents [S, C] and the rotated key part all heads share [S, R]."""
    C = m["kv_rank"]
    kv = lin(w, p + "dkv", h)
    return rms(kv[:, :C], w[p + "dkv.norm"], eps), rotate_halves(kv[:, None, C:], m["rot"])[:, 0]


def sink_softmax(scores, sink):
    """Weights of one query's visible keys: the denominator also holds exp(sink)."""
    top = max(scores.max().item(), sink)
    e = torch.exp(scores - top)
    return e / (e.sum() + math.exp(sink - top))


def latent_attention(m, w, p, h, eps):
    S = h.shape[0]
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = lin(w, p + "q", h).view(S, H, D + R)
    qu, qr = q[..., :D], rotate_halves(q[..., D:], m["rot"])
    c, kr = latent_rows(m, w, p, h, eps)
    ku, v = (c @ w[p + "uk"].to(F64).T).view(S, H, D), (c @ w[p + "uv"].to(F64).T).view(S, H, V)
    out = torch.zeros(S, H, V, dtype=F64)
    for hd in range(H):
        for i in range(S):
            sc = (ku[: i + 1, hd] @ qu[i, hd] + kr[: i + 1] @ qr[i, hd]) * m["scale"]
            out[i, hd] = sink_softmax(sc, float(w[p + "sink"][hd])) @ v[: i + 1, hd]
    return lin(w, p + "o", out.reshape(S, H * V) * sigmoid(lin(w, p + "g", h)))


def gated_ffn(w, p, h):
    return lin(w, p + "down", silu(lin(w, p + "gate", h)) * lin(w, p + "up", h))


def choose(r, scores):
    """One token's chosen experts (best first): group scores first, then the best of the kept groups."""
    E, allowed = r["experts"], set(range(r["experts"]))
    g = r.get("groups")
    if g:
        n = E // g["count"]
        worth = [sum(sorted((float(scores[e]) for e in range(k * n, (k + 1) * n)), reverse=True)[:2]) for k in range(g["count"])]
        kept = sorted(range(g["count"]), key=lambda k: -worth[k])[: g["keep"]]
        allowed = {e for k in kept for e in range(k * n, (k + 1) * n)}
    return sorted(allowed, key=lambda e: -float(scores[e]))[: r["top"]]


def routed_ffn(f, w, p, h):
    scores = sigmoid(lin(w, p + "router", h))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        picked = choose(f["router"], scores[t])
        total = scores[t, picked].sum() + 1e-20
        for e in picked:
            out[t] += scores[t, e] / total * gated_ffn(w, p + f"e{e}.", h[t])
    if f.get("shared"):
        out = out + sigmoid(lin(w, p + "shared.sg", h)) * gated_ffn(w, p + "shared.", h)
    return out


def forward(cfg, w, tokens, taps=None):
    """Logits [S, vocab] (float64) of one sequence; ``taps`` collects the stream after every layer."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"].to(F64)[tokens] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = latent_attention(L["mixer"], w, p + "mix.", layer_norm(w, p + "norm1", x, eps), eps)
        x = x + m * (y * w[p + "ls1"].to(F64))
        f = L.get("mlp")
        if f:
            h = layer_norm(w, p + "norm2", x, eps)
            y = routed_ffn(f, w, p + "mlp.", h) if f["kind"] == "moe" else gated_ffn(w, p + "mlp.", h)
            x = x + m * (y * w[p + "ls2"].to(F64))
        if taps is not None:
            taps.append(x.clone())
    return layer_norm(w, "final.norm", x, eps) @ w["head"].to(F64).T
