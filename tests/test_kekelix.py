"""Kekelix serving path against the plain oracle (tests/kekelix_oracle.py): every mechanism alone, whole prompts, prompt + token by token
decoding, unequal batches, reused slots, one loud far key at tile and chunk borders, the sink, both score maps, the repeated stretch of
layers, the first tokens, long decoding, other sizes, the cache limit, greedy generation through the serving entry points, the registry /
checkpoint reader, the trace runner and the generation command line.  Configurations and weights are made here (random, seeded)."""
import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kekelix_oracle as oracle  # noqa: E402

from neuronx_distributed_b200.inference.hf_adapter import HuggingFaceGenerationAdapter  # noqa: E402
from neuronx_distributed_b200.inference.trace_replay import TraceReplayer  # noqa: E402
from neuronx_distributed_b200.models import registry  # noqa: E402
from neuronx_distributed_b200.models.kekelix import GLU_SLOPE, KekelixConfig, KekelixForInference, load_kekelix_weights  # noqa: E402
from neuronx_distributed_b200.modules.moe.routed_ffn import RoutedFFN  # noqa: E402
from neuronx_distributed_b200.ops import seqmix  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
TOL32 = 2e-4
F64 = torch.float64
FULL = 1 << 30
YARN = {"factor": 4.0, "original": 40, "fast": 3.0, "slow": 0.5}


# ------------------------------------------------------------------------------------------------------------------ model making
def moe(ff=24, experts=6, top=2, limit=1.1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def diff(heads=4, kv_heads=2, dim=10, vdim=12, scale=None, diff=0.45, mlp="moe"):
    return {"type": "attention", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale or 1.3 / math.sqrt(dim)}}


def sink(heads=4, kv_heads=2, dim=14, vdim=9, rot=8, base=700.0, scaling=YARN, scale=None, mlp="moe"):
    r = {"base": base, "dims": rot, **({"scaling": scaling} if scaling else {})}
    return {"type": "attention_2", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": r, "scale": scale or 1.1 / math.sqrt(dim)}}


def chunked(heads=6, kv_heads=2, dim=12, chunk=7, rot=6, base=90.0, scaling=None, scale=None, mlp="moe"):
    r = {"base": base, "dims": rot, **({"scaling": scaling} if scaling else {})}
    return {"type": "attention_3", "mlp": moe() if mlp == "moe" else mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "rot": r, "scale": scale or 0.9 / math.sqrt(dim)}}


def make_cfg(layers, loop=None, vocab=50, width=48, eps=1e-5):
    return {"architecture": "Kekelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            **({"loop": dict(zip(("start", "stop", "times"), loop))} if loop else {})}


def random_checkpoint(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    bf = lambda t: t.to(torch.bfloat16).float()
    lin = lambda o, i, s=1.0: bf(torch.randn(o, i, generator=g) * s / math.sqrt(i))
    vec = lambda n, s=1.0, m=0.0: bf(torch.randn(n, generator=g) * s + m)
    W = cfg["width"]
    w = {"embed": bf(torch.randn(cfg["vocab"], W, generator=g)), "final.norm": vec(W, 0.2)}
    if cfg.get("loop"):
        w["loop.step"] = bf(torch.randn(cfg["loop"]["times"], W, generator=g) * 0.7)
    for i, L in enumerate(cfg["layers"]):
        p, m, q, f = f"l{i}.", L["mixer"], f"l{i}.mix.", L.get("mlp")
        H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        maps = 2 if L["type"] == "attention" else 1
        for k in "12" if f else "1":
            w[p + f"norm{k}"] = vec(W, 0.3)
        w.update({q + "q": lin(H * maps * D, W, 2.0), q + "k": lin(G * maps * D, W, 2.0), q + "o": lin(W, H * V, 1.5)})
        if L["type"] != "attention_3":
            w[q + "v"] = lin(G * V, W, 1.5)
        if L["type"] == "attention_2":
            w.update({q + "q.b": vec(H * D, 0.5), q + "k.b": vec(G * D, 0.5), q + "v.b": vec(G * V, 0.5)})
        if maps == 2:
            w.update({q + n: vec(D, 0.25) for n in ("lq1", "lk1", "lq2", "lk2")})
        if f:
            w[p + "mlp.router"] = lin(f["router"]["experts"], W, 2.0)
            for e in range(f["router"]["experts"]):
                y, F = p + f"mlp.e{e}.", f["expert"]["ff"]
                w.update({y + "gate": lin(F, W, 2.0), y + "up": lin(F, W, 2.0), y + "down": lin(W, F, 1.5)})
    return w


def build(cfg, weights, device, dtype=torch.float32, max_seq_len=400, batch_size=1):
    m = KekelixForInference(KekelixConfig.from_dict(cfg, dtype=dtype, device=torch.device(device)), batch_size=batch_size, max_seq_len=max_seq_len,
                            on_device_sampling=False)
    load_kekelix_weights(m.lm, weights)
    return m.eval()


def tokens_for(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_cut(model, toks, prompt):
    """Prompt of ``prompt`` tokens in one step, the rest one by one → logits at every position [S, vocab] (float, cpu)."""
    mgr = model.states
    slot = mgr.alloc()
    dev = next(model.parameters()).device
    x = model.forward_step(torch.tensor([toks[:prompt]], device=dev), [prompt], [slot], [0], True)
    mgr.advance([slot], [prompt])
    out = [model.logits(x[0])]
    for p in range(prompt, len(toks)):
        x = model.forward_step(torch.tensor([[toks[p]]], device=dev), [1], [slot], [p], False)
        mgr.advance([slot], [1])
        out.append(model.logits(x[0]))
    mgr.free(slot)
    return torch.cat(out).cpu()


def rel_err(got, want):
    """Mean-free difference relative to the spread of the expected values, per position."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    ref = (want - want.mean(-1, keepdim=True)).double().pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / ref


def close(got, want, tol):
    err = rel_err(got, want).max().item()
    assert err < tol, f"relative error {err:.3e} >= {tol}"


def i32(v, device):
    return torch.tensor(v, dtype=torch.int32, device=device)


class _Ctx:
    def __init__(self, lens, slots, pos0, fresh, device):
        self.lens, self.slots, self.pos0, self.fresh, self.scratch = i32(lens, device), i32(slots, device), i32(pos0, device), fresh, {}


# ------------------------------------------------------------------------------------------------------------ single mechanisms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,C", [(7, 48), (3, 37), (300, 64), (2, 1024), (5, 1030), (1200, 2048), (3, 5000), (2, 4608), (9, 520)])
@pytest.mark.parametrize("parts", ["all", "experts", "result", "refresh", "vector"])
def test_joint_of_parallel_layers(device, rows, C, parts):
    """The stream gets the mixer's result and the experts' rows (no weights), an embedding row and a vector; two norms of the new rows."""
    g = torch.Generator().manual_seed(rows + C)
    rnd = lambda *s: torch.randn(*s, generator=g)
    top, eps = 3, 1e-5
    x, w1, w2, vec, table = rnd(rows, C) + 2.0, rnd(C), rnd(C), rnd(C), rnd(11, C)
    y, base, tok = rnd(rows * top, C), rnd(rows, C), torch.randint(0, 11, (rows,), generator=g)
    src = torch.randperm(rows * top, generator=g).view(rows, top)
    experts, refresh = parts in ("all", "experts"), parts in ("all", "refresh")
    for dt in [torch.float32] + ([torch.bfloat16] if device == "cuda" else []):
        yd, bd, td, xd = y.to(device, dt), base.to(device, dt), table.to(device, dt), x.clone().to(device)
        ex = (src.to(device), None, bd, None) if experts else None
        inj = (tok.to(device), td, vec.to(device)) if refresh else ((None, None, vec.to(device)) if parts == "vector" else None)
        h1, h2 = seqmix.residual_norm_(xd, yd if experts else bd if parts == "result" else None, None, w1.to(device), None, eps, False, ex,
                                       w2.to(device), inj, dt)
        s = x.double()
        if experts:
            s = s + yd.cpu().double()[src].sum(1) + bd.cpu().double()
        elif parts == "result":
            s = s + bd.cpu().double()
        if refresh:
            s = s + td.cpu().double()[tok]
        if refresh or parts == "vector":
            s = s + vec.double()
        assert (xd.cpu().double() - s).abs().max() < 2e-5 * s.abs().max()
        for h, w in ((h1, w1), (h2, w2)):
            n = oracle.unit(s, eps) * w.double()
            assert h.dtype == dt and (h.cpu().double() - n).abs().max() < (2e-5 if dt == torch.float32 else 8e-3) * n.abs().max()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,rot,scaling", [(4, 2, 12, 6, None), (3, 1, 8, 8, YARN), (2, 2, 7, 4, YARN), (8, 1, 64, 20, YARN), (5, 5, 33, 2, None), (1, 1, 130, 128, None)])
def test_queries_and_keys_brought_to_unit_size_after_the_rotation(device, H, G, D, rot, scaling):
    """Inside a stacked projection, in place for the queries, beside the projected keys that stay and go to the cache as values."""
    g = torch.Generator().manual_seed(H * D)
    B, S, ring, eps = 2, 9, 4, 1e-2                                  # an eps that shows where it stands
    lens, slots = [9, 3], [2, 0]
    r = {"dims": rot, "base": 300.0, **({"scaling": scaling} if scaling else {})}
    p0 = torch.randn(B, S, H * D + G * D + 5, generator=g) * 0.3
    pd = p0.clone().to(device)
    q, k = pd[..., :H * D].unflatten(-1, (H, D)), pd[..., H * D:(H + G) * D].unflatten(-1, (G, D))
    kout = torch.full((B, S, G, D), 5.0, device=device)
    kc, vc = torch.full((3, ring, G, D), 7.0, device=device), torch.full((3, ring, G, D), 7.0, device=device)
    seqmix.window_qk_prepare(q, k, k, None, None, eps, i32([0, 0], device), i32(lens, device), i32(slots, device), kc, vc,
                             inv_freq=seqmix.rotary_inv_freq(rot, 300.0, device, scaling), rot_dims=rot, amp=seqmix.rotary_amplitude(scaling), unit=True, kout=kout)
    assert torch.equal(pd[..., H * D:].cpu(), p0[..., H * D:])
    for b, n in enumerate(lens):
        raw_q, raw_k = p0[b, :n, :H * D].double().view(n, H, D), p0[b, :n, H * D:(H + G) * D].double().view(n, G, D)
        wq, wk = oracle.unit(oracle.rotate_halves(raw_q, r), eps), oracle.unit(oracle.rotate_halves(raw_k, r), eps)
        assert (q[b, :n].cpu().double() - wq).abs().max() < 2e-5 and (kout[b, :n].cpu().double() - wk).abs().max() < 2e-5
        for t in range(max(0, n - ring), n):
            assert (kc[slots[b], t % ring].cpu().double() - wk[t]).abs().max() < 2e-5
            assert torch.equal(vc[slots[b], t % ring].cpu().double(), raw_k[t])
    assert (kc[1] == 7.0).all() and (kc[0, 3:] == 7.0).all()


MIXER_CASES = {
    "diff": (diff(), 21), "diff_one_group": (diff(4, 1, 6, 5), 17), "diff_no_groups": (diff(3, 3, 7, 16, diff=0.2), 40), "diff_one_head": (diff(1, 1, 5, 4), 9),
    "diff_wide": (diff(2, 1, 24, 70, diff=0.8), 70), "diff_many_heads": (diff(20, 1, 4, 6), 34),
    "sink": (sink(), 21), "sink_all_rotated": (sink(2, 2, 8, 8, rot=8), 18), "sink_one_group": (sink(5, 1, 6, 20, rot=2, scaling=None), 40), "sink_wide": (sink(1, 1, 40, 66, rot=12), 70),
    "chunk": (chunked(), 30), "chunk_one": (chunked(2, 1, 8, chunk=1, rot=4), 9), "chunk_longer_than_prompt": (chunked(2, 2, 10, chunk=64, rot=10), 50),
    "chunk_scaled": (chunked(3, 3, 9, chunk=5, rot=4, scaling=YARN), 23), "chunk_odd": (chunked(4, 1, 40, chunk=33, rot=8), 80),
}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", sorted(MIXER_CASES))
def test_mixer_prompt_and_single_tokens(device, name):
    """The module alone: a prompt, and the same tokens one by one (and after a prompt of half of them) against a dirty cache."""
    spec, S = MIXER_CASES[name]
    cfg = make_cfg([dict(spec, mlp=None)], width=31)
    w = random_checkpoint(cfg, len(name))
    h = torch.randn(S, 31, generator=torch.Generator().manual_seed(S))
    want = oracle.MIXERS[spec["type"]](spec["mixer"], w, "l0.mix.", h.double(), 1e-5)
    mix = build(cfg, w, device, max_seq_len=S + 3).lm.layers[0].mixer
    assert mix.ring == (min(spec["mixer"]["mask"]["size"], S + 3) if spec["type"] == "attention_3" else S + 3)
    tol = 2e-4 * max(1.0, want.abs().max().item())
    for cut in (S, 1, (S + 1) // 2):
        st = {n: torch.full((3,) + shape, 9.0, device=device) for n, (shape, _) in mix.state_spec().items()}
        out = [mix(h[:cut].to(device)[None], _Ctx([cut], [2], [0], True, device), st)[0]]
        out += [mix(h[t:t + 1].to(device)[None], _Ctx([1], [2], [t], False, device), st)[0] for t in range(cut, S)]
        assert (torch.cat(out).cpu().double() - want).abs().max() < tol, cut


def test_attention_mistakes_would_show():
    """The mixer cases tell the design from its near misses (planted in the oracle's arithmetic)."""
    spec, S = MIXER_CASES["diff"]
    w, h = random_checkpoint(make_cfg([dict(spec, mlp=None)]), 1), torch.randn(12, 48, generator=torch.Generator().manual_seed(1)).double()
    want = oracle.differential_attention(spec["mixer"], w, "l0.mix.", h, 1e-5)
    lam = oracle.mixing_number(spec["mixer"], w, "l0.mix.")
    for changed in ({"lq1": "lq2"}, {"lk2": "lk1"}):
        other = dict(w, **{"l0.mix." + a: w["l0.mix." + b] for a, b in changed.items()})
        assert abs(oracle.mixing_number(spec["mixer"], other, "l0.mix.") - lam) > 1e-2
        assert (oracle.differential_attention(spec["mixer"], other, "l0.mix.", h, 1e-5) - want).abs().max() > 1e-2
    H, D = spec["mixer"]["heads"], spec["mixer"]["dim"]
    swapped = dict(w, **{"l0.mix.q": w["l0.mix.q"].view(H, 2, D, -1).transpose(0, 1).reshape(H * 2 * D, -1)})   # maps before heads
    assert (oracle.differential_attention(spec["mixer"], swapped, "l0.mix.", h, 1e-5) - want).abs().max() > 1e-1
    q, k, v = torch.randn(12, 2, 6).double(), torch.randn(12, 1, 6).double(), torch.randn(12, 1, 5).double()
    a = oracle.attend(q, k, v, 0.3, extra=1.0)
    assert (a - oracle.attend(q, k, v, 0.3)).abs().max() > 1e-1 and (oracle.attend(q, k, v, 0.3, chunk=5) - oracle.attend(q, k, v, 0.3, chunk=6)).abs().max() > 1e-1


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,G,D,V,maps,chunk", [(4, 2, 16, 16, 1, 0), (3, 1, 8, 16, 2, 0), (6, 3, 24, 32, 1, 10), (2, 2, 5, 7, 2, 6)])
def test_single_tokens_take_part_in_no_row_they_do_not_see(device, H, G, D, V, maps, chunk):
    """Cache rows that hold no visible position are NaN here: they may not reach any result."""
    g = torch.Generator().manual_seed(H * D)
    ring, p = chunk or 90, 74
    lo = oracle.visible_from(p, chunk)
    k, v, q = torch.randn(p + 1, G * maps, D, generator=g), torch.randn(p + 1, G, V, generator=g), torch.randn(1, 1, H * maps, D, generator=g)
    s0 = torch.randn(H * maps, generator=g)
    dts = [torch.float32] + ([torch.bfloat16] if device == "cuda" else [])
    for dt in dts:
        kc, vc = torch.full((2, ring, G * maps, D), float("nan")), torch.full((2, ring, G, V), float("nan"))
        for j in range(lo, p + 1):
            kc[1, j % ring], vc[1, j % ring] = k[j], v[j]
        out = torch.empty(1, H * V, device=device, dtype=dt)
        lam = torch.tensor([0.6], device=device)
        seqmix.window_attention_token(q.to(device, dt), kc.to(device, dt), vc.to(device, dt), None, i32([1], device), i32([p], device), i32([1], device), FULL, 0.3,
                                      0.0, out, 1.0, sink=s0.to(device), chunk=chunk, diff=(lam, 1e-5, 0.7) if maps == 2 else None)
        kd, vd, qd = (t.to(dt).double() for t in (k, v, q[0, 0]))
        heads = []
        for h in range(H):
            a = []
            for m in range(maps):
                sc = kd[lo:, h // (H // G) * maps + m] @ qd[h * maps + m] * 0.3
                a.append(oracle.weights_of(sc, math.exp(s0[h * maps + m])) @ vd[lo:, h // (H // G)])
            heads.append(a[0] if maps == 1 else oracle.unit(a[0] - 0.6 * a[1], 1e-5) * 0.7)
        assert (out.cpu().double().view(H, V) - torch.stack(heads)).abs().max() < (1e-5 if dt == torch.float32 else 4e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,F", [(1, 8), (5, 7), (33, 96), (3, 33)])
def test_clamped_gate_with_a_number_per_row(device, rows, F):
    g = torch.Generator().manual_seed(F)
    gu, s = torch.randn(rows, 2 * F, generator=g) * 4, torch.rand(rows, generator=g) * 2
    a, b = (gu.double() * s.double()[:, None]).split(F, 1)
    want = a.clamp(max=1.5) * oracle.sigmoid(GLU_SLOPE * a.clamp(max=1.5)) * (b.clamp(-1.5, 1.5) + 1)
    got = seqmix.clamped_glu(gu.to(device), 1.5, GLU_SLOPE, s.to(device)).cpu().double()
    assert (got - want).abs().max() < 1e-5
    assert (a < -1.5).any() and (a > 1.5).any() and (b < -1.5).any() and (b > 1.5).any() or rows < 3


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("E,F,I,M", [(3, 8, 16, 5), (5, 7, 13, 4), (2, 24, 260, 9)])
def test_streamed_matrices_with_weighted_input_and_clamped_gate(device, E, F, I, M):
    g = torch.Generator().manual_seed(F)
    w, x, s = torch.randn(E, 2 * F, I, generator=g), torch.randn(M, I, generator=g), torch.rand(M, generator=g) + 0.2
    sel = torch.randint(-1, E + 1, (M,), generator=g)
    got = seqmix.indexed_gemv(w.to(device), sel.to(device), x.to(device), "clamped_glu", s.to(device), 2.0, GLU_SLOPE).cpu().double()
    for m in range(M):
        if not 0 <= sel[m] < E:
            assert (got[m] == 0).all()
            continue
        a, b = (w[sel[m]].double() @ (s[m].double() * x[m].double())).split(F)
        want = a.clamp(max=2.0) * oracle.sigmoid(GLU_SLOPE * a.clamp(max=2.0)) * (b.clamp(-2.0, 2.0) + 1)
        assert (got[m] - want).abs().max() < 1e-4


def _routed(f, P, width, device, dtype=torch.float32):
    r, e = f["router"], f["expert"]
    m = RoutedFFN(width, e["ff"], r["experts"], r["top"], gated=True, glu=(e["limit"], GLU_SLOPE), weigh_input=True, dtype=dtype, device=device)
    m.up.copy_(torch.stack([torch.cat([P[f"e{i}.gate"], P[f"e{i}.up"]]) for i in range(r["experts"])]))
    m.down.copy_(torch.stack([P[f"e{i}.down"] for i in range(r["experts"])]))
    m.router.linear_router.weight.copy_(P["router"])
    return m


def _ffn_weights(f, width, seed):
    w = random_checkpoint(make_cfg([diff(mlp=f)], width=width), seed)
    return {k[len("l0.mlp."):]: v for k, v in w.items() if k.startswith("l0.mlp.")}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows", [1, 5, 90])
@pytest.mark.parametrize("f", [moe(), moe(17, 5, 1, 0.4), moe(24, 4, 4, 3.0), moe(9, 40, 3, 0.9)])
def test_routed_feed_forward(device, rows, f):
    P = _ffn_weights(f, 32, rows)
    h = torch.randn(rows, 32, generator=torch.Generator().manual_seed(rows))
    got = _routed(f, P, 32, device)(h.to(device)).cpu().double()
    want = oracle.routed_ffn(f, P, "", h.double())
    assert (got - want).abs().max() < 2e-4 * max(1.0, want.abs().max().item())
    scores = oracle.sigmoid(oracle.lin(P, "router", h.double()))
    after = torch.zeros_like(want)                                   # the weight on the output instead would be another function
    for t in range(rows):
        for e in scores[t].topk(f["router"]["top"]).indices.tolist():
            after[t] += scores[t, e] * oracle.expert(f, P, f"e{e}.", h[t].double())
    assert (after - want).abs().max() > 1e-2


@pytest.mark.gpu
@pytest.mark.parametrize("rows,width,ff,top", [(6, 48, 24, 2), (90, 48, 24, 1), (300, 128, 64, 3)])
def test_bfloat16_routed_feed_forward_rows_with_a_clear_choice(rows, width, ff, top):
    """Few rows (streamed experts), many rows of odd sizes (an expert at a time), many rows in whole 64s (the grouped GEMM when the main
    extension is built), on the rows whose choice of experts is no close call."""
    f = moe(ff=ff, experts=6, top=top)
    P = _ffn_weights(f, width, 4)
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(3)).bfloat16()
    s = oracle.sigmoid(h.double() @ P["router"].double().T).sort(-1, descending=True).values
    clear = (s[:, top - 1] - s[:, top] > 0.02).nonzero()[:, 0]
    got = _routed(f, P, width, "cuda", torch.bfloat16)(h.cuda()).cpu().double()
    want = oracle.routed_ffn(f, P, "", h.double())
    assert len(clear) >= rows // 3
    assert (got - want)[clear].abs().max() < 3e-2 * want.abs().max()


# ------------------------------------------------------------------------------------------------------------------ whole models
SINGLE = {
    "diff": ([diff()], None), "sink": ([sink()], None), "chunked": ([chunked()], None), "bare": ([sink(mlp=None)], None),
    "one_expert": ([diff(mlp=moe(experts=1, top=1))], None), "every_expert": ([chunked(mlp=moe(experts=3, top=3))], None),
    "alone_again": ([chunked()], (0, 1, 4)), "once": ([diff(), sink()], (0, 2, 1)), "last_again": ([sink(), diff()], (1, 2, 2)),
    "bare_again": ([diff(mlp=None), chunked(mlp=None)], (0, 2, 2)), "odd_sizes": ([diff(3, 1, 7, 5), chunked(3, 1, 9, 4, rot=2)], (0, 1, 3)),
}
MIXED = [sink(mlp=moe(16, 5, 1)), diff(2, 1, 16, 8, mlp=None), chunked(4, 2, 10, 9, rot=4), diff(), sink(3, 3, 8, 8, rot=8, scaling=None, mlp=None)]
LOOP = (1, 4, 3)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_small_models(device, name):
    layers, loop = SINGLE[name]
    cfg = make_cfg(layers, loop, width=47 if name == "odd_sizes" else 48)
    w = random_checkpoint(cfg, seed=len(name))
    toks = tokens_for(cfg, 30, 5)
    want = oracle.forward(cfg, w, toks)
    close(run_cut(build(cfg, w, device), toks, 30), want, TOL32)
    close(run_cut(build(cfg, w, device), toks, 11), want, TOL32)


@pytest.fixture(scope="module")
def mixed():
    cfg = make_cfg(MIXED, LOOP)
    w = random_checkpoint(cfg, seed=11)
    toks = tokens_for(cfg, 48, 7)
    stream = []
    want = oracle.forward(cfg, w, toks, taps=stream)
    return cfg, w, toks, want, stream


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("prompt", [48, 1, 2, 6, 31])
def test_prompt_then_decode_matches_oracle(device, mixed, prompt):
    cfg, w, toks, want, _ = mixed
    close(run_cut(build(cfg, w, device), toks, prompt), want, TOL32)


@pytest.mark.parametrize("device", DEVICES)
def test_residual_stream_after_every_layer_run(device, mixed):
    cfg, w, toks, _, stream = mixed
    model = build(cfg, w, device)
    assert len(stream) == 1 + 3 * 3 + 1 == len(model.lm.runs) == len(model.lm.state_specs())
    seen = {}
    model.forward_step(torch.tensor([toks], device=device), [len(toks)], [model.states.alloc()], [0], True, tap=lambda i, x: seen.__setitem__(i, x[0].cpu().clone()))
    for i in range(len(stream)):
        close(seen[i], stream[i], TOL32)


def test_the_repeated_stretch_is_told_from_its_near_misses(mixed):
    cfg, w, toks, want, _ = mixed
    toks, want = toks[:12], want[:12]
    for change in ({"loop": dict(cfg["loop"], times=2)}, {"loop": dict(cfg["loop"], start=2)}, {"loop": dict(cfg["loop"], stop=3)}):
        assert rel_err(oracle.forward(dict(cfg, **change), w, toks), want).max() > 1e-2
    for t in range(3):
        step = w["loop.step"].clone()
        step[t] = 0
        assert rel_err(oracle.forward(cfg, dict(w, **{"loop.step": step}), toks), want).max() > 1e-3
    caches = build(cfg, w, "cpu").states
    assert all(caches.layer(a)["k"] is not caches.layer(b)["k"] for a in range(11) for b in range(a))


@pytest.mark.parametrize("device", DEVICES)
def test_unequal_batch_against_each_alone_and_reused_slots(device, mixed):
    cfg, w, toks, _, _ = mixed
    model = build(cfg, w, device)
    reqs = [tokens_for(cfg, n, 20 + n) for n in (1 + 6, 7 + 6, 23 + 6, 2 + 6)]
    prompts, steps = [1, 7, 23, 2], [0, 6, 3, 6]                      # row 0 ends with its prompt, row 2 leaves early
    mgr = model.states
    warm = [mgr.alloc() for _ in range(3)]                            # dirty a few slots first, then give them back
    model.forward_step(torch.randint(0, 50, (3, 40), device=device), [40, 40, 40], warm, [0, 0, 0], True)
    for s in warm:
        mgr.free(s)
    slots = [mgr.alloc() for _ in reqs]
    assert set(warm) <= set(slots)
    S = max(prompts)
    ids = torch.zeros(len(reqs), S, dtype=torch.long)
    for b, (r, p) in enumerate(zip(reqs, prompts)):
        ids[b, :p] = torch.tensor(r[:p])
    x = model.forward_step(ids.to(device), prompts, slots, [0] * len(reqs), True)
    got = [[model.logits(x[b, :p]).cpu()] for b, p in enumerate(prompts)]
    live = [b for b in range(len(reqs)) if steps[b] > 0]
    mgr.free(slots[0])
    for k in range(max(steps)):
        live = [b for b in live if k < steps[b]]
        step_ids = torch.tensor([[reqs[b][prompts[b] + k]] for b in live], device=device)
        x = model.forward_step(step_ids, [1] * len(live), [slots[b] for b in live], [prompts[b] + k for b in live], False)
        lg = model.logits(x[:, 0]).cpu()
        for j, b in enumerate(live):
            got[b].append(lg[j:j + 1])
    for b, r in enumerate(reqs):
        n = prompts[b] + steps[b]
        close(torch.cat(got[b]), oracle.forward(cfg, w, r[:n]), TOL32)
    fresh = build(cfg, w, device)
    close(torch.cat(got[2]), run_cut(fresh, reqs[2][:26], 23), 1e-5)        # the batch changes nothing beyond rounding


# ------------------------------------------------------------------------------- far keys, chunk borders, first tokens, long decoding
def _needle_model(kind, seed=3, map_=0, **kw):
    """One layer whose head 0 looks for token 0 wherever it is: coordinate 0 of every embedding is a constant that the head's query (a
    coordinate that is not rotated) reads, and the key there is large for token 0 alone."""
    make = {"attention": diff, "attention_2": sink, "attention_3": chunked}[kind]
    cfg = make_cfg([make(mlp=None, **kw)], vocab=20)
    w, m = random_checkpoint(cfg, seed), cfg["layers"][0]["mixer"]
    w["embed"][:, 0] = 2.0
    h = oracle.offset_norm(w, "l0.norm1", w["embed"].double(), 1e-5)
    u = (h[0] - h[1:].mean(0)).float()
    u[0] = 0.0
    D = m["dim"]
    row = map_ * D + D - 1                                           # the head's last coordinate in the chosen map
    w["l0.mix.q"][row] = 0.0
    w["l0.mix.q"][row, 0] = 16.0
    w["l0.mix.k"][row] = (u / u.norm() * 4).bfloat16().float()
    return cfg, w


def _needle_case(cfg, w, at, n):
    toks = [1 + (5 * t) % 19 for t in range(n)]
    plain = list(toks)
    toks[at] = 0
    want = oracle.forward(cfg, w, toks)
    return toks, want, rel_err(want, oracle.forward(cfg, w, plain))


NEEDLES = [(0, 200), (0, 1), (3, 150), (31, 40), (32, 33), (63, 130), (64, 65), (127, 128), (128, 129), (100, 200)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("kind,map_", [("attention", 0), ("attention", 1), ("attention_2", 0)])
@pytest.mark.parametrize("at,prompt", NEEDLES)
def test_one_loud_far_key(device, kind, map_, at, prompt):
    """The needle moves every later position's logits, however far away it lies — in the prompt and over decoded tokens, at and next
    to the borders of the kernels' tiles; a lost cache row, a window or an off-by-one in the causal edge would show."""
    cfg, w = _needle_model(kind, map_=map_, heads=2, kv_heads=1)
    toks, want, moved = _needle_case(cfg, w, at, 200)
    assert (moved[at:] > 1e-2).all() and (moved[:at] < 1e-12).all()
    close(run_cut(build(cfg, w, device), toks, prompt), want, TOL32)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("chunk", [1, 5, 32, 33, 64, 100])
@pytest.mark.parametrize("prompt", [130, 1, 63])
def test_loud_keys_at_chunk_borders(device, chunk, prompt):
    """A needle just before and just behind a chunk's edge moves its own chunk and nothing else, in prompts, over decoded tokens and with
    the edge between the two."""
    cfg, w = _needle_model("attention_3", heads=2, kv_heads=1, chunk=chunk, rot=4, scale=2.0)
    model = build(cfg, w, device)
    edge = chunk * max(1, 64 // chunk)
    for at in sorted({edge - 1, edge, min(edge + chunk - 1, 129), 0}):
        toks, want, moved = _needle_case(cfg, w, at, 130)
        inside = torch.tensor([t >= at and t // chunk == at // chunk for t in range(130)])
        assert (moved[inside] > 1e-2).all() and (moved[~inside] < 1e-12).all()
        close(run_cut(model, toks, prompt), want, TOL32)


@pytest.mark.gpu
@pytest.mark.parametrize("kind,kw", [("attention", dict(dim=16, vdim=32)), ("attention", dict(dim=64, vdim=144, heads=8, kv_heads=2)),
                                     ("attention_2", dict(dim=32, vdim=48)), ("attention_3", dict(dim=32, chunk=100, scale=1.0)),
                                     ("attention_3", dict(dim=48, chunk=64, heads=5, kv_heads=1, scale=1.0))])
@pytest.mark.parametrize("at,prompt", [(0, 300), (0, 1), (31, 32), (63, 70), (64, 65), (99, 100), (100, 101), (127, 290), (250, 255)])
def test_one_loud_key_in_bfloat16(kind, kw, at, prompt):
    """The tensor-core kernels (sizes in whole 16s) against the same needles."""
    cfg, w = _needle_model(kind, **kw)
    toks, want, moved = _needle_case(cfg, w, at, 300)
    assert moved[at] > 0.05
    close(run_cut(build(cfg, w, "cuda", dtype=torch.bfloat16), toks, prompt), want, 6e-2)


@pytest.mark.parametrize("device", DEVICES)
def test_the_sink_is_one_and_unscaled(device):
    """Scores near zero and far below it: leaving the sink out, scaling it or counting it twice is far outside the tolerance."""
    cfg = make_cfg([sink(mlp=None, scale=0.2), sink(2, 1, mlp=None, scale=0.9)])
    w = random_checkpoint(cfg, seed=6)
    for n in ("q", "q.b"):
        w["l1.mix." + n] = -w["l1.mix." + n] * 3
    toks = tokens_for(cfg, 25, 8)
    want = oracle.forward(cfg, w, toks)
    for prompt in (25, 1, 9):
        close(run_cut(build(cfg, w, device), toks, prompt), want, TOL32)
    plain = oracle.weights_of
    try:
        for extra in (0.0, 2.0):
            oracle.weights_of = lambda s, e: plain(s, extra if e else 0.0)
            assert rel_err(oracle.forward(cfg, w, toks), want).max() > 50 * TOL32
    finally:
        oracle.weights_of = plain


@pytest.mark.parametrize("device", DEVICES)
def test_first_tokens_on_one_slot_again_and_again(device, mixed):
    cfg, w, _, _, _ = mixed
    model = build(cfg, w, device)
    for seed, n, prompt in [(1, 1, 1), (2, 2, 1), (3, 2, 2), (4, 9, 1), (5, 3, 2)]:
        toks = tokens_for(cfg, n, seed)
        close(run_cut(model, toks, prompt), oracle.forward(cfg, w, toks), TOL32)
        assert model.states.num_slots == 1


@pytest.mark.parametrize("device", DEVICES)
def test_long_decoding_from_one_token(device):
    cfg = make_cfg([diff(2, 1), chunked(2, 1, 8, 19), sink(2, 2)], (0, 2, 2))
    w = random_checkpoint(cfg, seed=21)
    toks = tokens_for(cfg, 130, 9)
    close(run_cut(build(cfg, w, device), toks, 1), oracle.forward(cfg, w, toks), TOL32)


def test_positions_beyond_the_cache_are_refused(mixed):
    cfg, w, toks, want, _ = mixed
    model = build(cfg, w, "cpu", max_seq_len=20)
    assert model.states.layer(0)["k"].shape[1] == 20 and model.states.layer(2)["k"].shape[1] == 9
    close(run_cut(model, toks[:20], 15), want[:20], TOL32)             # the last row of the cache is used
    slot = model.states.alloc()
    with pytest.raises(ValueError):
        model.forward_step(torch.tensor([toks[:21]]), [21], [slot], [0], True)
    with pytest.raises(ValueError):
        model.forward_step(torch.tensor([[1]]), [1], [slot], [20], False)
    with pytest.raises(ValueError):
        model.generate(torch.tensor([toks[:16]]), 6)
    model.on_device_sampling = True
    assert model.generate(torch.tensor([toks[:16]]), 5).shape == (1, 5)
    only_chunks = make_cfg([chunked(2, 1, 8, 6)])
    v = random_checkpoint(only_chunks, 2)
    toks = tokens_for(only_chunks, 60, 1)
    m = build(only_chunks, v, "cpu", max_seq_len=20)                   # chunks shorter than the limit: a sequence may grow on
    assert m.lm.position_limit is None
    close(run_cut(m, toks, 30), oracle.forward(only_chunks, v, toks), TOL32)


def test_unknown_parts_and_unfitting_checkpoints_are_refused(mixed):
    cfg, w, _, _, _ = mixed
    for layers in ([dict(diff(), type="something")], [diff(mlp={"kind": "other"})]):
        with pytest.raises(ValueError):
            build(make_cfg(layers), {}, "cpu")
    with pytest.raises((KeyError, ValueError)):
        build(make_cfg([diff(heads=6)]), random_checkpoint(make_cfg([diff()])), "cpu")
    with pytest.raises(KeyError):
        build(cfg, {k: v for k, v in w.items() if k != "l0.mix.v.b"}, "cpu")
    for loop in ((1, 1, 2), (0, 6, 2), (0, 2, 0)):
        with pytest.raises(ValueError):
            KekelixConfig.from_dict(make_cfg(MIXED, loop))


def test_continuing_step_carries_one_token(mixed):
    cfg, w, toks, _, _ = mixed
    model = build(cfg, w, "cpu")
    s = model.states.alloc()
    model.forward_step(torch.tensor([toks[:4]]), [4], [s], [0], True)
    with pytest.raises(ValueError):
        model.forward_step(torch.tensor([toks[4:7]]), [3], [s], [4], False)


# ---------------------------------------------------------------------------------------------- generation, registry, command lines
def _oracle_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_through_the_serving_entry_points(device, mixed):
    cfg, w, _, _, _ = mixed
    prompts = [tokens_for(cfg, 9, 31), tokens_for(cfg, 4, 32)]
    want = [_oracle_greedy(cfg, w, p, 5) for p in prompts]
    model = build(cfg, w, device, batch_size=2)
    model.on_device_sampling = True
    ids = torch.zeros(2, 9, dtype=torch.long)
    mask = torch.zeros(2, 9, dtype=torch.long)
    for b, p in enumerate(prompts):
        ids[b, :len(p)], mask[b, :len(p)] = torch.tensor(p), 1
    out = model.generate(ids.to(device), 5, prompt_lens=mask.sum(1).to(device))
    assert out.cpu().tolist() == want
    out = HuggingFaceGenerationAdapter(model, pad_token_id=0).generate(ids.to(device), attention_mask=mask.to(device), max_new_tokens=5)
    assert out[:, 9:].cpu().tolist() == want


@pytest.mark.gpu
def test_token_generation_replayed_from_a_cuda_graph(mixed):
    """A captured token-generation step reads positions on the device: replays at growing positions match the eager steps."""
    cfg, w, _, _, _ = mixed
    model = build(cfg, w, "cuda", dtype=torch.bfloat16, batch_size=2)
    ids = torch.tensor([tokens_for(cfg, 40, 61), tokens_for(cfg, 40, 62)], device="cuda")
    tok, pos = torch.zeros(2, 1, dtype=torch.long, device="cuda"), torch.zeros(2, dtype=torch.long, device="cuda")
    step = lambda: model.token_generation(tok, pos)

    def run(fn):
        model.context_encoding(ids[:, :20])
        out = []
        for p in range(20, 40):
            tok.copy_(ids[:, p:p + 1]), pos.fill_(p)
            out.append(fn().clone())
        return torch.stack(out)

    eager = run(step)
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for _ in range(2):
            step()
    torch.cuda.current_stream().wait_stream(side)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        held = step()

    def replay():
        graph.replay()
        return held

    assert torch.equal(run(replay), eager)


def _save_model_dir(path, cfg, w):
    from neuronx_distributed_b200.utils.safetensors_utils import save_state_dict_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_state_dict_safetensors({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))


def _trace(cfg):
    a, b, c = tokens_for(cfg, 14, 41), tokens_for(cfg, 5, 42), tokens_for(cfg, 9, 43)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:10], "want": [0, 9]}, {"id": "b", "tokens": b[:3], "want": [2]}], "end": []}]
    for k in range(4):
        ent = [{"id": "a", "tokens": [a[10 + k]], "want": [0]}]
        if k < 2:
            ent.append({"id": "b", "tokens": [b[3 + k]], "want": [] if k == 0 else [0]})
        steps.append({"step": k + 1, "entries": ent, "end": (["b"] if k == 1 else []) + (["a"] if k == 3 else [])})
    steps.append({"step": 5, "entries": [{"id": "c", "tokens": c, "want": [8]}], "end": ["c"]})
    rows = {0: [("a", 0), ("a", 9), ("b", 2)], 1: [("a", 10)], 2: [("a", 11), ("b", 4)], 3: [("a", 12)], 4: [("a", 13)], 5: [("c", 8)]}
    return {"a": a, "b": b, "c": c}, steps, rows


@pytest.mark.parametrize("device", DEVICES)
def test_registry_checkpoint_reader_and_trace_replay(device, mixed, tmp_path):
    import numpy as np

    cfg, w, _, _, _ = mixed
    _save_model_dir(str(tmp_path / "m"), cfg, w)
    model = registry.load_for_serving(str(tmp_path / "m"), dtype=torch.float32, device=torch.device(device), max_seq_len=64, on_device_sampling=False)
    assert isinstance(model, KekelixForInference)
    reqs, steps, rows = _trace(cfg)
    out = tmp_path / "o"
    os.makedirs(out)
    log = io.StringIO()
    TraceReplayer(model, str(out)).run([json.dumps(s) for s in steps], log)
    assert log.getvalue().split() == [x for s in steps for x in ("done", str(s["step"]))]
    assert model.states.in_use == 0
    for n, want_rows in rows.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(len(want_rows), cfg["vocab"]).copy())
        for j, (rid, pos) in enumerate(want_rows):
            close(got[j:j + 1], oracle.forward(cfg, w, reqs[rid][:pos + 1])[-1:], TOL32)


def test_trace_runner_command_line(mixed, tmp_path):
    import numpy as np

    cfg, w, _, _, _ = mixed
    _save_model_dir(str(tmp_path / "m"), cfg, w)
    reqs, steps, rows = _trace(cfg)
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(tmp_path / "o"),
                        "--max-tokens", "40"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    got = np.fromfile(tmp_path / "o" / "5.f32", dtype="<f4")
    close(torch.from_numpy(got.copy())[None], oracle.forward(cfg, w, reqs["c"])[8:9], TOL32)


def test_generate_command_line(mixed, tmp_path):
    cfg, w, _, _, _ = mixed
    _save_model_dir(str(tmp_path / "m"), cfg, w)
    prompts = [tokens_for(cfg, 6, 51), tokens_for(cfg, 3, 52)]
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    args = [os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--max-new-tokens", "4"]
    for p in prompts:
        args += ["--prompt-ids", ",".join(map(str, p))]
    r = subprocess.run(args, capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = [[int(t) for t in line.split(",")] for line in r.stdout.strip().splitlines()[-2:]]
    assert got == [_oracle_greedy(cfg, w, p, 4) for p in prompts]


# ---------------------------------------------------------------------------------------------------------------- bfloat16 (GPU)
@pytest.mark.gpu
def test_bfloat16_serving_close_to_the_oracle():
    """No feed-forwards: a routed layer may take another expert on a close call in bfloat16 (covered row by row above)."""
    cfg = make_cfg([diff(4, 2, 16, 32, mlp=None), chunked(4, 1, 32, 20, rot=16, mlp=None), sink(4, 4, 16, 48, rot=16, mlp=None), diff(2, 1, 24, 16, mlp=None)],
                   (0, 2, 2), width=64)
    w = random_checkpoint(cfg, seed=13)
    toks = tokens_for(cfg, 80, 3)
    want = oracle.forward(cfg, w, toks)
    model = build(cfg, w, "cuda", dtype=torch.bfloat16)
    for prompt in (50, 80, 1):
        err = rel_err(run_cut(model, toks, prompt), want)
        assert err.mean() < 4e-2 and err.max() < 0.2, (err.mean().item(), err.max().item())


def _heads64(q, k, v, ok, s0, lam, scale):
    """q [I,H*maps,D], k [J,G*maps,D], v [J,G,V] float64, ok [I,J] → ([I,H,V], [I,H]): the results, and how much the final norm enlarges what
    was rounded before it (two maps that nearly cancel leave little to be enlarged)."""
    maps = 1 if lam is None else 2
    H, G = q.shape[1] // maps, v.shape[1]
    a = []
    for m in range(maps):
        sc = torch.einsum("ihd,jhd->hij", q[:, m::maps], k[:, m::maps].repeat_interleave(H // G, 1)) * scale
        sc = sc.masked_fill(~ok, float("-inf"))
        extra = s0[m::maps, None, None] if s0 is not None else torch.full((H, 1, 1), float("-inf"), dtype=F64)
        top = torch.maximum(sc.amax(-1, keepdim=True), extra)
        e = torch.exp(sc - top)
        a.append(torch.einsum("hij,jhv->ihv", e / (e.sum(-1, keepdim=True) + torch.exp(extra - top)), v.repeat_interleave(H // G, 1)))
    if maps == 1:
        return a[0], torch.ones(a[0].shape[:2], dtype=F64)
    rms = lambda x: x.pow(2).mean(-1).sqrt()
    return oracle.unit(a[0] - lam * a[1], 1e-5) * 0.7, ((rms(a[0]) + lam * rms(a[1])) / rms(a[0] - lam * a[1])).clamp(min=1.0)


def _close_heads(got, want, gain, what):
    err, room = (got - want).abs().amax(-1), 1.5e-2 * gain * max(1.0, want.abs().max().item())
    assert (err < room).all(), (what, (err / room).max().item())


SIZES = [(4, 2, 16, 16, 2), (3, 1, 64, 128, 2), (2, 2, 128, 256, 2), (2, 1, 48, 80, 2), (4, 4, 96, 112, 2), (20, 1, 32, 48, 2), (4, 1, 64, 64, 1), (6, 2, 128, 128, 1),
         (2, 1, 256, 256, 1), (5, 1, 80, 48, 1), (2, 2, 24, 40, 1), (1, 1, 136, 144, 2)]


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,V,maps", SIZES)
@pytest.mark.parametrize("window,chunk", [(FULL, 0), (70, 0), (FULL, 64), (FULL, 100), (50, 96), (FULL, 1)])
def test_bfloat16_prompt_attention_in_one_kernel(H, G, D, V, maps, window, chunk):
    """Unequal rows around the tile borders, sinks, windows and chunks, one and two maps, against float64 on the same bfloat16 inputs (sizes
    the tensor-core kernel takes and sizes it leaves to the scalar one)."""
    g = torch.Generator().manual_seed(H * D + V)
    lens, S = [333, 128, 129, 1], 333
    B = len(lens)
    nq, nk, nv = H * maps * D, G * maps * D, G * V
    p = torch.randn(B, S, -(-(nq + nk + nv) // 8) * 8, generator=g).bfloat16()
    s0, lam, scale = torch.randn(H * maps, generator=g) * 2, 0.6, 1.0 / math.sqrt(D)
    pd = p.cuda()
    cut = lambda t: (t[..., :nq].unflatten(-1, (H * maps, D)), t[..., nq:nq + nk].unflatten(-1, (G * maps, D)), t[..., nq + nk:nq + nk + nv].unflatten(-1, (G, V)))
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    ok = (j <= i) & (j > i - window) & ((i // chunk == j // chunk) if chunk else True)
    for with_sink in (True, False):
        out = torch.full((B * S, H * V + 8), 3.0, device="cuda", dtype=torch.bfloat16)
        seqmix.window_attention_prompt(*cut(pd), None, i32(lens, "cuda"), window, scale, 0.0, out, 1.0, sink=s0.cuda() if with_sink else None, chunk=chunk,
                                       diff=(torch.tensor([lam], device="cuda"), 1e-5, 0.7) if maps == 2 else None)
        assert (out[:, H * V:] == 3.0).all()
        got = out[:, :H * V].view(B, S, H, V).cpu().double()
        for b, n in enumerate(lens):
            q, k, v = (t[b, :n].double() for t in cut(p))
            _close_heads(got[b, :n], *_heads64(q, k, v, ok[:n, :n], s0.double() if with_sink else None, lam if maps == 2 else None, scale), (b, with_sink))
            assert (got[b, n:] == 0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,D,V,maps", SIZES)
@pytest.mark.parametrize("window,chunk", [(FULL, 0), (50, 0), (FULL, 96), (40, 96), (FULL, 64)])
def test_bfloat16_single_token_attention_at_many_lengths(H, G, D, V, maps, window, chunk):
    """Rows of a batch at very different positions — stretch, tile and chunk borders, a single visible row, a ring that has wrapped — a padded
    row, sinks, rows never written (NaN)."""
    g = torch.Generator().manual_seed(D + H)
    ring = chunk or (700 if window > 700 else 64)
    pos = [0, 1, 30, 49, 50, 63, 64, 65, 95, 96, 127, 128, 300, 639, 699, 5]
    B = len(pos)
    lens = [1] * B
    lens[14] = 0
    k, v = torch.randn(B, 700, G * maps, D, generator=g).bfloat16(), torch.randn(B, 700, G, V, generator=g).bfloat16()
    kc, vc = torch.full((B + 1, ring, G * maps, D), float("nan")), torch.full((B + 1, ring, G, V), float("nan"))
    slots = torch.randperm(B + 1, generator=g)[:B].tolist()
    lo = [max(0, p - window + 1, (p // chunk) * chunk if chunk else 0) for p in pos]
    for b, p in enumerate(pos):
        for t in range(lo[b], p + 1):
            kc[slots[b], t % ring], vc[slots[b], t % ring] = k[b, t].float(), v[b, t].float()
    q = torch.randn(B, 1, H * maps, D, generator=g).bfloat16()
    s0, lam, scale = torch.randn(H * maps, generator=g) * 2, 0.6, 1.0 / math.sqrt(D)
    out = torch.empty(B, H * V, device="cuda", dtype=torch.bfloat16)
    seqmix.window_attention_token(q.cuda(), kc.bfloat16().cuda(), vc.bfloat16().cuda(), None, i32(slots, "cuda"), i32(pos, "cuda"), i32(lens, "cuda"), window, scale, 0.0,
                                  out, 1.0, sink=s0.cuda(), chunk=chunk, diff=(torch.tensor([lam], device="cuda"), 1e-5, 0.7) if maps == 2 else None)
    got = out.view(B, H, V).cpu().double()
    for b, p in enumerate(pos):
        if lens[b] == 0:
            assert (got[b] == 0).all()
            continue
        seen = slice(lo[b], p + 1)
        _close_heads(got[b][None], *_heads64(q[b].double(), k[b, seen].double(), v[b, seen].double(), torch.ones(1, p + 1 - lo[b], dtype=torch.bool),
                                             s0.double(), lam if maps == 2 else None, scale), (b, p))
