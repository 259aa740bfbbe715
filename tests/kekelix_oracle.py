"""Plain, slow statement of the Kekelix design in float64: one function per mechanism, whole sequences at once, no caches, no kernels,
nothing shared with the serving path.  Weights come as a dict of checkpoint tensors (``l<i>.mix.*`` etc.), configurations as the
``config.json`` dict."""
import math

import torch

F64 = torch.float64


def lin(w, name, x):
    y = x @ w[name].to(F64).T
    return y + w[name + ".b"].to(F64) if name + ".b" in w else y


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(w, name, x, eps):
    """RMS norm whose stored weight is the gain's distance from one."""
    return unit(x, eps) * (1.0 + w[name].to(F64))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rotation(rot):
    """(frequencies, amplitude) of the coordinate pairs, interpolated by pair index where the configuration asks for a longer context."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freqs, 1.0
    pair_of = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    first, last = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        part = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * part + f * (1.0 - part))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_halves(x, rot):
    """x [S, heads, D]: coordinates (i, i + dims/2) of every head turned by position * frequency; the rest untouched."""
    freqs, amp = rotation(rot)
    half, y = rot["dims"] // 2, x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)
    for i, f in enumerate(freqs):
        c, s = (amp * torch.cos(pos * f))[:, None], (amp * torch.sin(pos * f))[:, None]
        y[:, :, i] = x[:, :, i] * c - x[:, :, i + half] * s
        y[:, :, i + half] = x[:, :, i + half] * c + x[:, :, i] * s
    return y


def visible_from(i, chunk):
    """First position that position i sees: 0, or the start of its own chunk."""
    return (i // chunk) * chunk if chunk else 0


def weights_of(scores, extra):
    """Weights of one query's visible keys; ``extra`` joins the denominator (1: a score of zero without a value)."""
    top = max(scores.max().item(), 0.0)
    e = torch.exp(scores - top)
    return e / (e.sum() + extra * math.exp(-top))


def attend(q, k, v, scale, chunk=0, extra=0.0):
    """q [S,H,D], k [S,G,D], v [S,G,V] → [S,H,V]: every query head against the keys of its group that it sees."""
    S, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.zeros(S, H, v.shape[2], dtype=F64)
    for h in range(H):
        for i in range(S):
            j = visible_from(i, chunk)
            out[i, h] = weights_of(k[j:i + 1, h // per] @ q[i, h] * scale, extra) @ v[j:i + 1, h // per]
    return out


def mixing_number(m, w, p):
    """How much of the second map is taken off."""
    dot = lambda a, b: (w[p + a].to(F64) * w[p + b].to(F64)).sum().item()
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + m["diff"]


def differential_attention(m, w, p, h, eps):
    S, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = lin(w, p + "q", h).view(S, H, 2, D), lin(w, p + "k", h).view(S, G, 2, D)
    v = lin(w, p + "v", h).view(S, G, V)
    first, second = (attend(q[:, :, a], k[:, :, a], v, m["scale"]) for a in (0, 1))
    o = unit(first - mixing_number(m, w, p) * second, eps) * (1.0 - m["diff"])
    return lin(w, p + "o", o.reshape(S, H * V))


def rotary_sink_attention(m, w, p, h, eps):
    S, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = rotate_halves(lin(w, p + "q", h).view(S, H, D), m["rot"]), rotate_halves(lin(w, p + "k", h).view(S, G, D), m["rot"])
    return lin(w, p + "o", attend(q, k, lin(w, p + "v", h).view(S, G, V), m["scale"], extra=1.0).reshape(S, H * V))


def chunked_shared_attention(m, w, p, h, eps):
    """The key projection is the value too; queries and keys are rotated and then brought to unit root mean square."""
    S, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    v = lin(w, p + "k", h).view(S, G, D)
    q, k = unit(rotate_halves(lin(w, p + "q", h).view(S, H, D), m["rot"]), eps), unit(rotate_halves(v, m["rot"]), eps)
    return lin(w, p + "o", attend(q, k, v, m["scale"], chunk=m["mask"]["size"]).reshape(S, H * D))


MIXERS = {"attention": differential_attention, "attention_2": rotary_sink_attention, "attention_3": chunked_shared_attention}


def expert(f, w, p, h):
    lim = f["expert"]["limit"]
    g, u = lin(w, p + "gate", h).clamp(max=lim), lin(w, p + "up", h).clamp(-lim, lim)
    return lin(w, p + "down", g * sigmoid(1.702 * g) * (u + 1.0))


def routed_ffn(f, w, p, h):
    """The chosen experts' scores multiply what the experts READ."""
    scores = sigmoid(lin(w, p + "router", h))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(f["router"]["experts"]), key=lambda e: -float(scores[t, e]))
        for e in order[: f["router"]["top"]]:
            out[t] += expert(f, w, p + f"e{e}.", scores[t, e] * h[t])
    return out


def layer(L, w, p, x, eps):
    """Both sublayers read the same stream, each through its own norm."""
    y = MIXERS[L["type"]](L["mixer"], w, p + "mix.", offset_norm(w, p + "norm1", x, eps), eps)
    if L.get("mlp"):
        y = y + routed_ffn(L["mlp"], w, p + "mlp.", offset_norm(w, p + "norm2", x, eps))
    return x + y


def runs(cfg):
    """[(layer, pass or None before whose first layer the stream is refreshed)] in the order of execution."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return out + [(i, None) for i in range(lp["stop"], n)]


def forward(cfg, w, tokens, taps=None):
    """Logits [S, vocab] (float64) of one sequence; ``taps`` collects the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    table = w["embed"].to(F64)
    first = x = table[tokens]
    for i, t in runs(cfg):
        if t is not None:
            x = x + (first if t > 0 else 0.0) + w["loop.step"][t].to(F64)
        x = layer(cfg["layers"][i], w, f"l{i}.", x, eps)
        if taps is not None:
            taps.append(x.clone())
    return offset_norm(w, "final.norm", x, eps) @ table.T
