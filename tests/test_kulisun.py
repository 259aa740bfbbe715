"""Kulisun serving path against the plain oracle (tests/kulisun_oracle.py): every mechanism alone, whole prompts, prompt + token by
token decoding, unequal batches, reused slots, one loud far key at tile borders, sinks, the first tokens, long decoding, other sizes,
the cache limit, greedy generation through the serving entry points, the registry / checkpoint reader, the trace runner and the
generation command line.  Configurations and weights are made here (random, seeded)."""
import io
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kulisun_oracle as oracle  # noqa: E402

from neuronx_distributed_b200.inference.hf_adapter import HuggingFaceGenerationAdapter  # noqa: E402
from neuronx_distributed_b200.inference.trace_replay import TraceReplayer  # noqa: E402
from neuronx_distributed_b200.models import registry  # noqa: E402
from neuronx_distributed_b200.models.kulisun import KulisunConfig, KulisunForInference, load_kulisun_weights  # noqa: E402
from neuronx_distributed_b200.modules.gated_ffn import GatedFFN  # noqa: E402
from neuronx_distributed_b200.modules.moe.routed_ffn import RoutedFFN  # noqa: E402
from neuronx_distributed_b200.modules.rms_norm import AffineLayerNorm  # noqa: E402
from neuronx_distributed_b200.ops import seqmix  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
TOL32 = 2e-4
F64 = torch.float64
YARN = {"factor": 4.0, "original": 40, "fast": 3.0, "slow": 0.5}


# ------------------------------------------------------------------------------------------------------------------ model making
def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=6, top=3, groups=(3, 2), shared=20):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        f["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def att(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, base=700.0, scaling=YARN, scale=None, mlp="dense"):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "latent_attention", "mlp": dense() if mlp == "dense" else mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": rot,
                      "scale": scale if scale is not None else 1.3 / math.sqrt(dim + rot_dim)}}


def make_cfg(layers, vocab=50, width=48, eps=1e-5, mult=0.7, scale=3.0):
    return {"architecture": "Kulisun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "embedding": {"scale": scale},
            "layers": layers}


def random_checkpoint(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    bf = lambda t: t.to(torch.bfloat16).float()
    lin = lambda o, i, s=1.0: bf(torch.randn(o, i, generator=g) * s / math.sqrt(i))
    vec = lambda n, s=1.0, m=0.0: bf(torch.randn(n, generator=g) * s + m)
    W, w = cfg["width"], {}
    w["embed"], w["head"] = bf(torch.randn(cfg["vocab"], W, generator=g) * 0.5), lin(cfg["vocab"], W, 2.0)
    w["final.norm"], w["final.norm.b"] = vec(W, 0.2, 1.0), vec(W, 0.2)
    for i, L in enumerate(cfg["layers"]):
        p, m, q, f = f"l{i}.", L["mixer"], f"l{i}.mix.", L.get("mlp")
        H, D, R, V, C = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        for k in "12" if f else "1":
            w[p + f"norm{k}"], w[p + f"norm{k}.b"], w[p + f"ls{k}"] = vec(W, 0.2, 1.0), vec(W, 0.3), vec(W, 0.5, 1.0)
        w.update({q + "q": lin(H * (D + R), W, 2.0), q + "dkv": lin(C + R, W, 2.0), q + "dkv.norm": vec(C, 0.3, 1.0), q + "uk": lin(H * D, C, 1.5),
                  q + "uv": lin(H * V, C), q + "sink": vec(H, 1.0, 0.5), q + "g": lin(H * V, W, 2.0), q + "o": lin(W, H * V, 2.0)})
        if not f:
            continue
        y = p + "mlp."
        if f["kind"] == "dense":
            F = f["ff"]
            w.update({y + "gate": lin(F, W, 2.0), y + "gate.b": vec(F, 0.5), y + "up": lin(F, W, 2.0), y + "up.b": vec(F, 0.5), y + "down": lin(W, F),
                      y + "down.b": vec(W, 0.5)})
            continue
        w[y + "router"] = lin(f["router"]["experts"], W, 3.0)
        pieces = [(f"e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])]
        if f.get("shared"):
            w[y + "shared.sg"] = lin(1, W, 2.0)
            pieces.append(("shared.", f["shared"]["ff"]))
        for n, F in pieces:
            w.update({y + n + "gate": lin(F, W, 2.0), y + n + "up": lin(F, W, 2.0), y + n + "down": lin(W, F, 2.0)})
    return w


def build(cfg, weights, device, dtype=torch.float32, max_seq_len=400, batch_size=1):
    m = KulisunForInference(KulisunConfig.from_dict(cfg, dtype=dtype, device=torch.device(device)), batch_size=batch_size, max_seq_len=max_seq_len,
                            on_device_sampling=False)
    load_kulisun_weights(m.lm, weights)
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


# ------------------------------------------------------------------------------------------------------------ single mechanisms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,C,experts,center,normed", [(7, 48, False, True, True), (3, 37, True, True, True), (300, 64, True, True, True),
                                                          (2, 1024, False, False, True), (5, 1030, True, True, True), (1200, 2048, True, True, True),
                                                          (3, 5000, False, True, True), (2, 4608, True, True, True), (9, 520, True, True, False)])
def test_residual_sum_joined_with_the_next_norm(device, rows, C, experts, center, normed):
    g = torch.Generator().manual_seed(rows + C)
    rnd = lambda *s: torch.randn(*s, generator=g)
    top, eps = 3, 1e-5
    x, scale, w, b = rnd(rows, C) + 2.0, rnd(C), rnd(C), rnd(C)
    y = rnd(rows * top if experts else rows, C)
    src = torch.randperm(rows * top, generator=g).view(rows, top)
    weight, base, bw = rnd(rows, top), rnd(rows, C), rnd(rows)

    def want(y, base):
        v = y.double()
        if experts:
            v = (v[src] * weight.double()[..., None]).sum(1) + base.double() * bw.double()[:, None]
        s = x.double() + scale.double() * v
        d = s - s.mean(-1, keepdim=True) if center else s
        return s, d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w.double() + b.double()

    for dt in [torch.float32] + ([torch.bfloat16] if device == "cuda" else []):
        yd, bd, xd = y.to(device, dt), base.to(device, dt), x.clone().to(device)
        ex = (src.to(device), weight.to(device), bd, bw.to(device)) if experts else None
        h = seqmix.residual_norm_(xd, yd, scale.to(device), w.to(device) if normed else None, b.to(device) if normed else None, eps, center, ex)
        s, n = want(yd.cpu(), bd.cpu())
        assert (xd.cpu().double() - s).abs().max() < 2e-5 * s.abs().max()
        if normed:
            assert h.dtype == dt and (h.cpu().double() - n).abs().max() < (2e-5 if dt == torch.float32 else 8e-3) * n.abs().max()
        else:
            assert h is None


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,C", [(4, 48), (3, 37), (1500, 96), (2, 3000)])
def test_layer_norm_with_gain_and_bias(device, rows, C):
    g = torch.Generator().manual_seed(C)
    x, w, b = torch.randn(rows, C, generator=g) * 3 + 5, torch.randn(C, generator=g), torch.randn(C, generator=g)
    n = AffineLayerNorm(C, 1e-4, device)
    n.weight.copy_(w), n.bias.copy_(b)
    want = oracle.layer_norm({"n": w, "n.b": b}, "n", x.double(), 1e-4)
    assert (n(x.to(device)).cpu().double() - want).abs().max() < 2e-5 * want.abs().max()


def test_interpolated_rotation_frequencies_and_their_amplitude():
    cases = [(16, 700.0, {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}), (32, 10000.0, {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}),
             (8, 50.0, {"factor": 3.0, "original": 6, "fast": 2.0, "slow": 1.9}), (6, 10000.0, {"factor": 1.0, "original": 64, "fast": 4.0, "slow": 2.0}),
             (4, 10.0, {"factor": 2.0, "original": 100000, "fast": 2.0, "slow": 1.0}), (8, 300.0, None)]
    kinds = set()
    for dims, base, sc in cases:
        rot = {"dims": dims, "base": base, **({"scaling": sc} if sc else {})}
        freqs, amp = oracle.rotation(rot)
        want = torch.tensor(freqs, dtype=F64)
        got = seqmix.rotary_inv_freq(dims, base, None, sc).double()
        assert ((got - want).abs() / want).max() < 1e-6 and abs(seqmix.rotary_amplitude(sc) - amp) < 1e-12
        if sc and sc["factor"] > 1:
            ratio = want / torch.tensor(oracle.rotation({"dims": dims, "base": base})[0], dtype=F64)
            for r in ratio.tolist():
                kinds.add("kept" if r == 1 else "slowed" if abs(r - 1 / sc["factor"]) < 1e-12 else "between")
            assert abs(amp - (1 + 0.1 * math.log(sc["factor"]))) < 1e-12
    assert kinds == {"kept", "slowed", "between"}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,D,R,C", [(3, 16, 8, 40), (2, 12, 6, 21), (5, 8, 24, 64), (1, 24, 64, 32), (40, 16, 32, 16)])
def test_latent_rows_and_queries_prepared_in_one_call(device, H, D, R, C):
    """The latent's norm, the rotation (with its amplitude) of the shared key part AND of the query heads in place inside a stacked
    projection, and the cache rows: a prompt whose rows have different lengths, then single tokens at their own positions."""
    g = torch.Generator().manual_seed(H + R)
    B, S, base, eps = 2, 9, 300.0, 1e-5
    lens = [9, 4]
    nq = H * (D + R)
    off = -(-nq // 8) * 8
    p0 = torch.randn(B, S + 1, off + C + R + 3, generator=g)
    nw = torch.rand(C, generator=g) + 0.5
    rot = {"dims": R, "base": base, "scaling": YARN}
    inv, amp = seqmix.rotary_inv_freq(R, base, device, YARN), seqmix.rotary_amplitude(YARN)

    def want(b, n):
        q = oracle.rotate_halves(p0[b, :n, :nq].double().view(n, H, D + R)[..., D:], rot)
        kv = p0[b, :n, off:off + C + R].double()
        return q, torch.cat([oracle.rms(kv[:, :C], nw, eps), oracle.rotate_halves(kv[:, None, C:], rot)[:, 0]], -1)

    cache = torch.full((3, 16, C + R), 7.0, device=device)
    slots = i32([2, 0], device)

    def call(p, pos, n, rows):
        q = p[..., :nq].view(p.shape[0], p.shape[1], H, D + R)
        r = seqmix.latent_kv_store(p[..., off:off + C + R], nw.to(device), eps, inv, R, i32(pos, device), i32(n, device), slots, cache, rows, q=q, q_off=D, amp=amp)
        return q.cpu().double(), r

    q, rows = call(p0[:, :S].clone().to(device), [0, 0], lens, True)
    for b, n in enumerate(lens):
        wq, wr = want(b, n)
        assert (q[b, :n, :, D:] - wq).abs().max() < 1e-4 and torch.equal(q[b, :n, :, :D].float(), p0[b, :n, :nq].view(n, H, D + R)[..., :D])
        assert (rows[b, :n].cpu().double() - wr).abs().max() < 1e-4
        assert (cache[[2, 0][b], :n].cpu().double() - wr).abs().max() < 1e-4
        assert (cache[[2, 0][b], n:] == 7.0).all()
    one = torch.stack([p0[b, n] for b, n in enumerate(lens)])[:, None].clone().to(device)
    q, rows = call(one, lens, [1, 1], False)
    assert rows is None
    for b, n in enumerate(lens):
        wq, wr = want(b, n + 1)
        assert (q[b, 0, :, D:] - wq[n]).abs().max() < 1e-4 and (cache[[2, 0][b], n].cpu().double() - wr[n]).abs().max() < 1e-4


def _attention_case(H, D, R, V, C, S, seed, scaling=YARN, width=32):
    spec = att(H, D, R, V, C, scaling=scaling, mlp=None)
    cfg = make_cfg([spec], width=width)
    w = random_checkpoint(cfg, seed)
    h = torch.randn(S, width, generator=torch.Generator().manual_seed(seed + 1))
    return cfg, w, h, oracle.latent_attention(spec["mixer"], w, "l0.mix.", h.double(), 1e-5)


class _Ctx:
    def __init__(self, lens, slots, pos0, fresh, device):
        self.lens, self.slots, self.pos0, self.fresh, self.scratch = i32(lens, device), i32(slots, device), i32(pos0, device), fresh, {}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,D,R,V,C,S", [(3, 16, 8, 24, 40, 21), (1, 8, 2, 8, 8, 5), (5, 10, 6, 9, 21, 17), (2, 32, 32, 48, 96, 150), (17, 8, 4, 8, 12, 40)])
@pytest.mark.parametrize("order", ["expanded", "absorbed"])
def test_attention_prompt_and_cache(device, H, D, R, V, C, S, order):
    """The module alone: both evaluation orders of a prompt, then the same tokens one by one against the cache."""
    cfg, w, h, want = _attention_case(H, D, R, V, C, S, H * 100 + D, YARN if R >= 4 else None)
    model = build(cfg, w, device, max_seq_len=S + 3)
    mix = model.lm.layers[0].mixer
    mix.block_products = order == "expanded"
    st = {"kv": torch.full((3, S + 3, C + R), 9.0, device=device)}
    tol = 2e-4 * max(1.0, want.abs().max().item())
    out = mix(h.to(device)[None], _Ctx([S], [2], [0], True, device), st)
    assert (out[0].cpu().double() - want).abs().max() < tol
    st["kv"].fill_(9.0)
    for t in range(min(S, 25)):
        out = mix(h[t:t + 1].to(device)[None], _Ctx([1], [1], [t], False, device), st)
        assert (out[0, 0].cpu().double() - want[t]).abs().max() < tol, t


@pytest.mark.parametrize("device", DEVICES)
def test_rows_wider_than_the_single_token_kernels_take(device):
    """Latents beyond the decode kernels' row limit go through matrix products over the cache."""
    H, D, R, V, C, S = 2, 8, 8, 8, seqmix.LATENT_ROW_MAX, 14
    cfg, w, h, want = _attention_case(H, D, R, V, C, S, 77)
    mix = build(cfg, w, device, max_seq_len=S + 2).lm.layers[0].mixer
    st = {"kv": torch.full((2, S + 2, C + R), 9.0, device=device)}
    tol = 2e-4 * max(1.0, want.abs().max().item())
    for cut in (5, S):
        out = [mix(h[:cut].to(device)[None], _Ctx([cut], [1], [0], True, device), st)[0]]
        out += [mix(h[t:t + 1].to(device)[None], _Ctx([1], [1], [t], False, device), st)[0] for t in range(cut, S)]
        assert (torch.cat(out).cpu().double() - want).abs().max() < tol


@pytest.mark.parametrize("device", DEVICES)
def test_absorbed_attention_takes_part_in_no_row_it_does_not_see(device):
    """Cache rows never written hold NaN here: they may not reach any result."""
    H, C, R, ring = 3, 20, 6, 50
    g = torch.Generator().manual_seed(2)
    keys = torch.full((2, ring, C + R), float("nan"))
    keys[1, :9] = torch.randn(9, C + R, generator=g)
    qa, q, sink = torch.randn(H, 1, C, generator=g), torch.randn(1, 1, H, R, generator=g), torch.tensor([0.5, -30.0, 6.0])
    sc = (torch.einsum("hc,jc->hj", qa[:, 0].double(), keys[1, :9, :C].double()) + torch.einsum("hr,jr->hj", q[0, 0].double(), keys[1, :9, C:].double())) * 0.4
    want = torch.stack([oracle.sink_softmax(sc[h], float(sink[h])) @ keys[1, :9, :C].double() for h in range(H)])
    got = seqmix.latent_window_attention(qa.to(device), q.to(device), 0, keys.to(device), i32([1], device), i32([8], device), i32([1], device), 1 << 30, 0.4,
                                         sink.to(device))
    assert (got[:, 0].cpu().double() - want).abs().max() < 1e-5


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("N,E,top,groups,gate", [(9, 6, 3, (3, 2), True), (40, 12, 3, (4, 1), False), (5, 8, 8, (2, 2), True), (7, 10, 2, (10, 3), True),
                                                 (70, 64, 6, (8, 4), True), (3, 200, 5, (20, 2), False), (20, 256, 40, (8, 4), True), (4, 5, 1, None, True),
                                                 (6, 320, 6, (16, 3), True), (8, 33, 3, (1, 1), False)])
def test_router_groups_renormalised_weights_and_the_gate_column(device, N, E, top, groups, gate):
    logits = torch.randn(N, E + int(gate), generator=torch.Generator().manual_seed(N + E)) * 2
    w, idx, share = seqmix.route_topk(logits.to(device), None, top, E, "sigmoid", 1.0, groups, True, gate)
    r = {"experts": E, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    for t in range(N):
        s = torch.sigmoid(logits[t, :E].double())
        chosen = oracle.choose(r, s)
        assert idx[t].cpu().tolist() == chosen
        assert (w[t].cpu().double() - s[chosen] / s[chosen].sum()).abs().max() < 1e-6
    if gate:
        assert (share.cpu().double() - torch.sigmoid(logits[:, E].double())).abs().max() < 1e-6
    assert abs(w.sum(1).cpu() - 1).max() < 1e-5


def test_router_refuses_groups_that_do_not_leave_enough():
    for groups, top in [((3, 1), 3), ((4, 2), 2), ((3, 4), 1)]:
        with pytest.raises(ValueError):
            seqmix.route_topk(torch.zeros(2, 6), None, top, 6, "sigmoid", 1.0, groups, True)


def test_a_group_is_worth_its_two_best_and_not_its_best():
    """The largest score of all sits in a group whose second best is poor; the group is dropped, and with it that expert."""
    z = torch.tensor([[4.0, -4.0, 1.5, 1.5, 1.0, 1.0]])
    _, idx, _ = seqmix.route_topk(z, None, 2, 6, "sigmoid", 1.0, (3, 2), True)
    assert sorted(idx[0].tolist()) == [2, 3]
    assert oracle.choose({"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}}, torch.sigmoid(z[0])) == idx[0].tolist()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("H,N,V", [(3, 5, 8), (1, 1, 3), (7, 40, 20), (2, 3, 130)])
def test_heads_packed_with_a_gate_per_coordinate(device, H, N, V):
    g = torch.Generator().manual_seed(V)
    ov, gate = torch.randn(H, N, V, generator=g), torch.randn(N, H * V + 5, generator=g)
    got = seqmix.sigmoid_gate_heads(ov.to(device), gate.to(device)[:, :H * V]).cpu().double()
    want = ov.double().permute(1, 0, 2).reshape(N, H * V) * oracle.sigmoid(gate[:, :H * V].double())
    assert (got - want).abs().max() < 1e-6


def _ffn_weights(f, width, seed):
    w = random_checkpoint(make_cfg([att(mlp=f)], width=width), seed)
    return {k[len("l0.mlp."):]: v for k, v in w.items() if k.startswith("l0.mlp.")}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows", [1, 90])
def test_dense_gated_feed_forward_with_biases(device, rows):
    P = _ffn_weights(dense(37), 24, 1)
    m = GatedFFN(24, 37, True, torch.float32, device)
    m.up.copy_(torch.cat([P["gate"], P["up"]])), m.down.copy_(P["down"]), m.up_bias.copy_(torch.cat([P["gate.b"], P["up.b"]])), m.down_bias.copy_(P["down.b"])
    h = torch.randn(rows, 24, generator=torch.Generator().manual_seed(3))
    want = oracle.gated_ffn(P, "", h.double())
    assert (m(h.to(device)).cpu().double() - want).abs().max() < 1e-4


def _routed(f, P, width, device, dtype=torch.float32):
    r, g = f["router"], f["router"].get("groups")
    E, sh = r["experts"], f.get("shared")
    m = RoutedFFN(width, f["expert"]["ff"], E, r["top"], shared_ff=sh["ff"] if sh else 0, gated=True, groups=(g["count"], g["keep"]) if g else None,
                  renormalise=True, shared_gated=True, shared_gate=bool(sh), dtype=dtype, device=device)
    m.up.copy_(torch.stack([torch.cat([P[f"e{e}.gate"], P[f"e{e}.up"]]) for e in range(E)]))
    m.down.copy_(torch.stack([P[f"e{e}.down"] for e in range(E)]))
    m.router.linear_router.weight.copy_(torch.cat([P["router"]] + ([P["shared.sg"]] if sh else [])))
    if sh:
        m.shared_up.copy_(torch.cat([P["shared.gate"], P["shared.up"]])), m.shared_down.copy_(P["shared.down"])
    return m


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows", [1, 5, 90])
@pytest.mark.parametrize("f", [moe(), moe(ff=17, experts=5, top=1, groups=None, shared=0), moe(ff=24, experts=8, top=4, groups=(2, 1), shared=33),
                               moe(experts=4, top=4, groups=(4, 4), shared=24)])
def test_routed_feed_forward(device, rows, f):
    P = _ffn_weights(f, 32, rows)
    h = torch.randn(rows, 32, generator=torch.Generator().manual_seed(rows))
    got = _routed(f, P, 32, device)(h.to(device)).cpu().double()
    want = oracle.routed_ffn(f, P, "", h.double())
    assert (got - want).abs().max() < 2e-4 * max(1.0, want.abs().max().item())


@pytest.mark.gpu
@pytest.mark.parametrize("rows,width,ff,shared", [(6, 48, 24, 40), (90, 48, 24, 40), (300, 128, 64, 192)])
def test_bfloat16_routed_feed_forward_rows_with_a_clear_choice(rows, width, ff, shared):
    """Few rows (streamed experts), many rows of odd sizes (an expert at a time), many rows in whole 64s (the grouped GEMM when the main
    extension is built), on the rows whose choice of groups and experts is no close call."""
    f = moe(ff=ff, experts=6, top=2, groups=(3, 2), shared=shared)
    P = _ffn_weights(f, width, 4)
    h = torch.randn(rows, width, generator=torch.Generator().manual_seed(3)).bfloat16()
    s = torch.sigmoid(h.double() @ P["router"].double().T)
    clear = [t for t in range(rows) if len({tuple(oracle.choose(f["router"], s[t] + e)) for e in 0.01 * torch.randn(20, 6, generator=torch.Generator().manual_seed(t))}) == 1]
    got = _routed(f, P, width, "cuda", torch.bfloat16)(h.cuda()).cpu().double()
    want = oracle.routed_ffn(f, P, "", h.double())
    assert len(clear) >= rows // 3
    assert (got - want)[clear].abs().max() < 3e-2 * want.abs().max()


# ------------------------------------------------------------------------------------------------------------------ whole models
SINGLE = {
    "dense": [att()],
    "bare": [att(mlp=None, scaling=None)],
    "routed": [att(heads=2, mlp=moe())],
    "routed_no_groups_no_shared": [att(mlp=moe(groups=None, shared=0, experts=5, top=2))],
    "one_head_small": [att(heads=1, dim=4, rot_dim=2, vdim=6, kv_rank=8, mlp=moe(top=1, groups=(6, 1)))],
    "wide_value": [att(heads=4, dim=8, rot_dim=16, vdim=40, kv_rank=96, base=50.0, mlp=dense(64))],
    "odd_sizes": [att(heads=3, dim=7, rot_dim=6, vdim=5, kv_rank=13, mlp=dense(19))],
}
MIXED = [att(mlp=moe(ff=16, experts=8, top=3, groups=(4, 2), shared=12)), att(heads=2, dim=24, rot_dim=12, vdim=16, kv_rank=24, base=90.0), att(mlp=None),
         att(heads=4, dim=8, rot_dim=8, vdim=8, kv_rank=48, scaling=None, scale=0.5, mlp=moe(experts=4, top=1, groups=(2, 1))),
         att(heads=5, dim=12, rot_dim=4, vdim=20, kv_rank=32, scaling={"factor": 2.0, "original": 64, "fast": 6.0, "slow": 1.0}, mlp=moe(groups=None, top=2))]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_single_layer_models(device, name):
    cfg = make_cfg(SINGLE[name], mult=1.0 if name == "dense" else 0.7, scale=1.0 if name == "bare" else 3.0, width=47 if name == "odd_sizes" else 48)
    w = random_checkpoint(cfg, seed=len(name))
    toks = tokens_for(cfg, 30, 5)
    want = oracle.forward(cfg, w, toks)
    close(run_cut(build(cfg, w, device), toks, 30), want, TOL32)
    close(run_cut(build(cfg, w, device), toks, 11), want, TOL32)


@pytest.fixture(scope="module")
def mixed():
    cfg = make_cfg(MIXED)
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
def test_residual_stream_after_every_layer(device, mixed):
    cfg, w, toks, _, stream = mixed
    model = build(cfg, w, device)
    seen = {}
    model.forward_step(torch.tensor([toks], device=device), [len(toks)], [model.states.alloc()], [0], True, tap=lambda i, x: seen.__setitem__(i, x[0].cpu().clone()))
    for i in range(len(MIXED)):
        close(seen[i], stream[i], TOL32)


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


# ---------------------------------------------------------------------------------------- far keys, sinks, first tokens, long decoding
def _needle_model(seed=3, **kw):
    """One layer whose head 0 looks for token 0 wherever it is: coordinate 0 of the normed input is a constant (gain 0, bias 4) that the
    head's first query number reads, and latent coordinate 0 (the head's first key number) is large for token 0 alone."""
    cfg = make_cfg([att(heads=2, mlp=None, **kw)], vocab=20)
    w = random_checkpoint(cfg, seed)
    m, W = cfg["layers"][0]["mixer"], cfg["width"]
    w["l0.norm1"][0], w["l0.norm1.b"][0] = 0.0, 4.0
    w["l0.mix.q"][0] = 0.0
    w["l0.mix.q"][0, 0] = 4.0
    h = oracle.layer_norm(w, "l0.norm1", w["embed"].double() * cfg["embedding"]["scale"], 1e-5)[:, 1:]
    u = (h[0] - h[1:].mean(0)).float()
    w["l0.mix.dkv"][0] = 0.0
    w["l0.mix.dkv"][0, 1:] = (u / u.norm() * 2).bfloat16().float()
    w["l0.mix.uk"][0] = 0.0
    w["l0.mix.uk"][0, 0] = 4.0
    return cfg, w


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("at,prompt", [(0, 200), (0, 1), (3, 150), (31, 40), (32, 33), (63, 130), (64, 65), (127, 128), (128, 129), (100, 200)])
def test_one_loud_far_key(device, at, prompt):
    """The needle moves every later position's logits, however far away it lies — in the prompt and over decoded tokens, at and next
    to the borders of the kernels' tiles; a lost cache row, a window or an off-by-one in the causal edge would show."""
    cfg, w = _needle_model()
    toks = [1 + (5 * t) % 19 for t in range(200)]
    plain = list(toks)
    toks[at] = 0
    want, base = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, plain)
    moved = rel_err(want, base)
    assert (moved[at:] > 2e-2).all() and (moved[:at] < 1e-12).all()
    close(run_cut(build(cfg, w, device), toks, prompt), want, TOL32)


@pytest.mark.gpu
@pytest.mark.parametrize("at,prompt", [(0, 300), (0, 1), (31, 32), (32, 40), (63, 70), (64, 64 + 1), (127, 290), (250, 255)])
def test_one_loud_far_key_in_bfloat16(at, prompt):
    """The tensor-core kernels (sizes in whole 16s) against the same needle."""
    cfg, w = _needle_model(dim=16, rot_dim=16, vdim=32, kv_rank=48)
    toks = [1 + (5 * t) % 19 for t in range(300)]
    plain = list(toks)
    toks[at] = 0
    want, base = oracle.forward(cfg, w, toks), oracle.forward(cfg, w, plain)
    assert (rel_err(want, base)[at:] > 0.1).all()
    close(run_cut(build(cfg, w, "cuda", dtype=torch.bfloat16), toks, prompt), want, 4e-2)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("level", [-40.0, 0.0, 6.0, 60.0])
def test_the_sink_counts_once_and_unscaled(device, level):
    """Sinks from negligible to overwhelming; at the middle levels leaving one out, scaling it or counting it twice is far outside the
    tolerance."""
    cfg = make_cfg([att(mlp=None, scale=0.2), att(heads=2, mlp=None, scale=0.9)])
    w = random_checkpoint(cfg, seed=6)
    for i, H in ((0, 3), (1, 2)):
        w[f"l{i}.mix.sink"] = torch.full((H,), level) + torch.arange(H) * 0.5
    toks = tokens_for(cfg, 25, 8)
    want = oracle.forward(cfg, w, toks)
    for prompt in (25, 1, 9):
        close(run_cut(build(cfg, w, device), toks, prompt), want, TOL32)
    if level in (0.0, 6.0):
        for change in (lambda s: s - 1e4, lambda s: s * 0.2 + (s == 0) * 1.0, lambda s: s + math.log(2.0)):
            other = {k: (change(v) if k.endswith(".sink") else v) for k, v in w.items()}
            assert rel_err(oracle.forward(cfg, other, toks), want).max() > 50 * TOL32


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
    cfg = make_cfg([att(), att(heads=2, dim=8, rot_dim=16, vdim=8, kv_rank=16, mlp=moe())])
    w = random_checkpoint(cfg, seed=21)
    toks = tokens_for(cfg, 130, 9)
    close(run_cut(build(cfg, w, device), toks, 1), oracle.forward(cfg, w, toks), TOL32)


def test_positions_beyond_the_cache_are_refused(mixed):
    cfg, w, toks, want, _ = mixed
    model = build(cfg, w, "cpu", max_seq_len=20)
    assert model.states.layer(0)["kv"].shape[1] == 20
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


def test_unknown_parts_and_unfitting_checkpoints_are_refused(mixed):
    cfg, w, _, _, _ = mixed
    with pytest.raises(ValueError):
        build(make_cfg([dict(att(), type="something")]), w, "cpu")
    with pytest.raises(ValueError):
        build(make_cfg([att(mlp={"kind": "other"})]), w, "cpu")
    with pytest.raises((KeyError, ValueError)):
        build(make_cfg([att(heads=4)]), random_checkpoint(make_cfg([att()])), "cpu")
    with pytest.raises(KeyError):
        build(cfg, {k: v for k, v in w.items() if k != "l1.mlp.up.b"}, "cpu")


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
    assert isinstance(model, KulisunForInference)
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
    """Dense feed-forwards only: a routed layer may take another expert on a close call in bfloat16 (covered row by row above)."""
    cfg = make_cfg([att(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64), att(heads=2, dim=16, rot_dim=16, vdim=48, kv_rank=32, mlp=None),
                    att(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40)], width=64)
    w = random_checkpoint(cfg, seed=13)
    toks = tokens_for(cfg, 80, 3)
    want = oracle.forward(cfg, w, toks)
    model = build(cfg, w, "cuda", dtype=torch.bfloat16)
    for prompt in (50, 80, 1):                       # rounding noise of a small model with large weights: a few percent, no outliers
        err = rel_err(run_cut(model, toks, prompt), want)
        assert err.mean() < 4e-2 and err.max() < 0.2, (err.mean().item(), err.max().item())


def _softmax64(sc, ok, sink):
    sc = sc.masked_fill(~ok, float("-inf"))
    top = torch.maximum(sc.amax(-1, keepdim=True), sink)
    e = torch.exp(sc - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


@pytest.mark.gpu
@pytest.mark.parametrize("H,D,R,V", [(3, 24, 8, 32), (2, 64, 32, 64), (1, 128, 64, 128), (5, 112, 16, 48), (2, 96, 64, 128), (2, 8, 8, 16), (2, 192, 64, 256)])
@pytest.mark.parametrize("window", [1, 70, 1 << 30])
def test_bfloat16_prompt_attention_in_one_kernel(H, D, R, V, window):
    """Sinks, output gates read in place from a wider product, full and windowed visibility, unequal rows around the tile borders, against
    float64 on the same bfloat16 inputs."""
    g = torch.Generator().manual_seed(H * D + R)
    lens, S, CR = [333, 128, 129, 1], 333, 24 + R
    B = len(lens)
    rnd = lambda *s: torch.randn(*s, generator=g).bfloat16()
    p, kx, rows, v = rnd(B, S, H * (D + R) + H * V + 8), rnd(B, S, H * D), rnd(B, S, CR), rnd(B, S, H * V)
    sink = torch.randn(H, generator=g) * 3
    scale = 1.0 / math.sqrt(D + R)
    q = p[..., :H * (D + R)].double().view(B, S, H, D + R)
    k = torch.cat([kx.double().view(B, S, H, D), rows[..., CR - R:].double()[:, :, None].expand(B, S, H, R)], -1)
    sc = torch.einsum("bihd,bjhd->bhij", q, k) * scale
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    w = _softmax64(sc, ((j <= i) & (j > i - window))[None, None], sink.double().view(1, H, 1, 1))
    want = torch.einsum("bhij,bjhv->bihv", w, v.double().view(B, S, H, V)).reshape(B, S, H * V)
    gate = p[..., H * (D + R):H * (D + R) + H * V]
    pd = p.cuda()
    qd = pd[..., :H * (D + R)].view(B, S, H, D + R)
    assert seqmix.latent_prompt_fused_ok(qd, D, R, CR, V)
    for gated in (True, False):
        gd = pd[..., H * (D + R):H * (D + R) + H * V].flatten(0, 1) if gated else None
        got = seqmix.latent_prompt_attention(qd, kx.cuda(), rows.cuda(), v.cuda(), i32(lens, "cuda"), D, R, V, window, scale, sink.cuda(), gd)
        got = got.view(B, S, H * V).cpu().double()
        ref = want * torch.sigmoid(gate.double()) if gated else want
        for b, n in enumerate(lens):
            assert (got[b, :n] - ref[b, :n]).abs().max() < 2e-2 * max(1.0, ref[b, :n].abs().max().item()), (b, gated)
            assert (got[b, n:] == 0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("H,C,R", [(16, 512, 64), (5, 96, 16), (1, 16, 16), (17, 144, 32), (40, 256, 32), (8, 576, 64), (3, 40, 8)])
@pytest.mark.parametrize("window", [50, 1 << 30])
def test_bfloat16_single_token_attention_at_many_lengths(H, C, R, window):
    """The tensor-core decode kernel (and the scalar one, for the sizes it does not take): rows of a batch at very different positions —
    stretch and tile borders, a single visible row, a ring that has wrapped — a padded row, sinks, rows never written (NaN)."""
    g = torch.Generator().manual_seed(C + H)
    ring = 700 if window > 700 else 64
    pos = [0, 1, 30, 31, 32, 33, 63, 64, 65, 127, 128, 300, 639, 699, 5, 95] if window > 700 else [0, 1, 30, 49, 50, 63, 64, 65, 127, 128, 300, 639, 699, 5, 95, 77]
    B = len(pos)
    lens = [1] * B
    lens[14] = 0
    keys = torch.full((B + 1, ring, C + R), float("nan"))
    full = torch.randn(B, max(pos) + 1, C + R, generator=g).bfloat16()
    index = torch.randperm(B + 1, generator=g)[:B].tolist()
    for b, p in enumerate(pos):
        for t in range(max(0, p - ring + 1), p + 1):
            keys[index[b], t % ring] = full[b, t].float()
    qa, q = torch.randn(H, B, C, generator=g).bfloat16(), torch.randn(B, 1, H, 8 + R, generator=g).bfloat16()
    sink, scale = torch.randn(H, generator=g) * 2, 0.8 / math.sqrt(C + R)
    got = seqmix.latent_window_attention(qa.cuda(), q.cuda(), 8, keys.bfloat16().cuda(), i32(index, "cuda"), i32(pos, "cuda"), i32(lens, "cuda"), window, scale,
                                         sink.cuda()).cpu().double()
    for b, p in enumerate(pos):
        if lens[b] == 0:
            assert (got[:, b] == 0).all()
            continue
        seen = full[b, max(0, p - window + 1):p + 1].double()
        sc = torch.cat([qa[:, b].double(), q[b, 0, :, 8:].double()], -1) @ seen.T * scale
        want = _softmax64(sc, torch.ones_like(sc, dtype=torch.bool), sink.double()[:, None]) @ seen[:, :C]
        assert (got[:, b] - want).abs().max() < 2e-2 * max(1.0, want.abs().max().item()), (b, p)
