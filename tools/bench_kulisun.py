"""``bench.py --mode kulisun``: serving throughput of the Kulisun design at layer sizes that resemble a real model (random weights),
beside the framework's closest existing models at equal width and depth — Naguzen (latent attention over a window, routed feed-forward
with a shared expert) and Pulenex (latent attention with direct queries, layer norms) — plus every kernel the design added or extended,
timed alone against the measured copy bandwidth / GEMM throughput, beside the like kernel of those paths.  One GPU, bfloat16.  Device
time (CUDA events), >= 3 warm-up iterations; the weights of every model exceed L2, and the kernel timings flush L2 (a 512 MiB write)
between iterations; every kernel row is replayed from a CUDA graph.

Layers (width 2048, 16 heads of 128 + 64 rotated, value 128, latent 512, every key visible): one dense gated feed-forward of 5504, then
three routed ones of 32 gated experts of 704 in 4 groups of which 2 are kept, 4 chosen, and a shared gated expert of 1408."""
from __future__ import annotations

import json
import math
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tools"))

import bench_naguzen as base  # noqa: E402
import bench_pulenex as pul  # noqa: E402

WIDTH, VOCAB = base.WIDTH, base.VOCAB
YARN = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def kulisun_layers():
    mixer = {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 1.0 / math.sqrt(192),
             "rot": {"base": 10000.0, "dims": 64, "scaling": YARN}}
    moe = {"kind": "moe", "expert": {"ff": 704}, "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}}, "shared": {"ff": 1408}}
    lay = lambda mlp: {"type": "latent_attention", "mixer": mixer, "mlp": mlp}
    return [lay({"kind": "dense", "ff": 5504}), lay(moe), lay(moe), lay(moe)]


def build_kulisun(dev, batch, max_len):
    import torch

    from neuronx_distributed_b200.models.kulisun import KulisunConfig, KulisunForInference

    cfg = KulisunConfig(vocab=VOCAB, width=WIDTH, layers=kulisun_layers(), norm_eps=1e-6, residual_mult=0.5, embedding_scale=1.0,
                        dtype=torch.bfloat16, device=dev)
    m = KulisunForInference(cfg, batch_size=batch, max_seq_len=max_len).eval()
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for name, p in m.named_parameters():
            if p.dim() > 1:
                p.normal_(0.0, 0.02, generator=g)
                if "router" in name:                       # as a checkpoint stored in bfloat16 would hold it
                    p.copy_(p.to(torch.bfloat16).float())
        m.lm.embed.normal_(0.0, 1.0, generator=g)
    return m


def step_profile(model, dev, B, S):
    """Kernel tables (total microseconds, launches) of one context-encoding call and one token-generation step."""
    import torch

    ids = torch.randint(0, VOCAB, (B, S), device=dev)
    last = torch.full((B,), S - 1, dtype=torch.long, device=dev)
    tok, pos = torch.randint(0, VOCAB, (B, 1), device=dev), torch.full((B,), S, dtype=torch.long, device=dev)
    out = {}
    for name, fn in (("prompt", lambda: model.context_encoding(ids, last)), ("token", lambda: model.token_generation(tok, pos))):
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        with torch.profiler.profile(activities=[torch.profiler.ProfilerActivity.CUDA]) as prof:
            fn()
            torch.cuda.synchronize()
        rows = [(e.self_device_time_total, e.count, e.key) for e in prof.key_averages() if e.self_device_time_total > 0]
        out[name] = [[round(t, 1), n, k[:110]] for t, n, k in sorted(rows, reverse=True)]
    return out


def kernel_table(dev, steps, warmup):
    """Each kernel the design added or extended, alone at the sizes of the model above (4 x 2048 prompt tokens; 8 decoding rows) → time,
    achieved GB/s or TFLOP/s, fraction of the measured peak; the like kernel of the Naguzen / Pulenex path in the row after it."""
    import torch

    from neuronx_distributed_b200.ops import seqmix

    hbm, tfl, src = base._peaks()
    flush = torch.empty(128 << 20, dtype=torch.float32, device=dev)
    bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
    B, S, W, FULL = 4, 2048, WIDTH, 1 << 30
    N = B * S
    rnd = lambda *s, dtype=bf: torch.randn(*s, device=dev, dtype=f32).to(dtype)
    ints = lambda v, n: torch.full((n,), v, dtype=i32, device=dev)
    lens, slots, pos0 = ints(S, B), torch.arange(B, dtype=i32, device=dev), ints(0, B)
    Bd = 8
    l1, s8, p8 = ints(1, Bd), torch.arange(Bd, dtype=i32, device=dev), ints(2047, Bd)
    rows = []

    def replayed(fn):
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            for _ in range(2):
                fn()
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g):
            fn()
        return g.replay

    def add(name, fn, bytes_=0, flops=0, like=None):
        ms = base._timed(replayed(fn), steps, warmup, flush)
        r = {"kernel": name, "ms": round(ms, 4)}
        if bytes_:
            r["gbs"], r["frac_hbm"] = round(bytes_ / ms / 1e6, 1), round(bytes_ / ms / 1e6 / hbm, 3)
        if flops:
            r["tflops"], r["frac_bf16_gemm"] = round(flops / ms / 1e9, 2), round(flops / ms / 1e9 / tfl, 4)
        if like:
            r["like_of"] = like
        rows.append(r)

    # residual sum + norm
    x32, y16, vec = rnd(N, W, dtype=f32), rnd(N, W), torch.ones(W, device=dev)
    add("residual_norm_ (f32 stream += scale * bf16, layer norm with bias -> bf16)",
        lambda: seqmix.residual_norm_(x32, y16, vec, vec, vec, 1e-6, True), N * W * (4 + 2 + 4 + 2))
    add("naguzen / pulenex add_rms_norm_ (f32 stream += norm(bf16))", lambda: seqmix.add_rms_norm_(x32, y16, vec, 1e-6, True), N * W * 10,
        like="residual_norm_")
    top, E, FF = 4, 32, 704
    er, src_i, wt, gw = rnd(N * top, W), torch.randperm(N * top, device=dev).to(i32).view(N, top), rnd(N, top, dtype=f32), rnd(N, dtype=f32)
    ex = (src_i, wt, y16, gw)
    add("residual_norm_ that sums 4 expert rows and the gated shared one",
        lambda: seqmix.residual_norm_(x32, er, vec, vec, vec, 1e-6, True, ex), N * W * (top * 2 + 2 + 4 + 4 + 2))
    add("naguzen moe_combine (4 expert rows + shared)", lambda: seqmix.moe_combine(er, src_i, wt, y16), N * W * (top * 2 + 2 + 2), like="residual_norm_ (experts)")
    # preparation of queries and latent rows
    H, D, R, C, V = 16, 128, 64, 512, 128
    nq = H * (D + R)
    p = rnd(B, S, nq + C + R + H * V)
    nw, inv, amp = torch.ones(C, device=dev), seqmix.rotary_inv_freq(R, 10000.0, dev, YARN), seqmix.rotary_amplitude(YARN)
    q, kv, gate = p[..., :nq].view(B, S, H, D + R), p[..., nq:nq + C + R], p[..., nq + C + R:].flatten(0, 1)
    cache = torch.zeros(B, S, C + R, dtype=bf, device=dev)
    add("latent_kv_store + query rotation in one launch (strided stacked projection; every row cached)",
        lambda: seqmix.latent_kv_store(kv, nw, 1e-6, inv, R, pos0, lens, slots, cache, True, q=q, q_off=D, amp=amp), N * ((C + R) * 6 + H * R * 4))
    qc, kvc, c1k = q.contiguous(), kv.contiguous(), torch.zeros(B, 1024, C + R, dtype=bf, device=dev)
    add("naguzen latent_kv_store, then rope_q_ (two launches, ring 1024)",
        lambda: (seqmix.latent_kv_store(kvc, nw, 1e-6, inv, R, pos0, lens, slots, c1k, True), seqmix.rope_q_(qc, D, R, inv, pos0)),
        N * ((C + R) * 4 + H * R * 4) + B * 1024 * (C + R) * 2, like="latent_kv_store + query rotation")
    # attention
    keys, kx, vx = rnd(B, S, C + R), rnd(B, S, H * D), rnd(B, S, H * V)
    sink = torch.zeros(H, device=dev)
    for win, tag in ((FULL, "every key visible, sink, output gate"), (1024, "")):
        fl = B * H * sum(min(t + 1, win) for t in range(S)) * 2 * (D + R + V)
        if tag:
            add("latent_prompt_attention, " + tag,
                lambda: seqmix.latent_prompt_attention(q, kx, keys, vx, lens, D, R, V, FULL, 0.07, sink, gate), flops=fl)
        else:
            add("naguzen latent_prompt_attention (window 1024)", lambda: seqmix.latent_prompt_attention(qc, kx, keys, vx, lens, D, R, V, 1024, 0.07),
                flops=fl, like="latent_prompt_attention")
    qa1, q1 = rnd(H, Bd, C), rnd(Bd, 1, H, D + R)
    for L in (2048, 16384):
        kc, pl = rnd(Bd, L, C + R), ints(L - 1, Bd)
        add(f"latent_window_attention, single tokens, {L} cached rows, sink (8 rows)",
            lambda: seqmix.latent_window_attention(qa1, q1, D, kc, s8, pl, l1, FULL, 0.07, sink), bytes_=Bd * L * (C + R) * 2)
    kc1 = rnd(Bd, 1024, C + R)
    add("naguzen latent_window_attention (8 rows, ring 1024)", lambda: seqmix.latent_window_attention(qa1, q1, D, kc1, s8, p8, l1, 1024, 0.07),
        bytes_=Bd * 1024 * (C + R) * 2, like="latent_window_attention")
    qf, cf = qa1.float(), kc1.float()
    add("naguzen latent_window_attention in float32 (8 rows, ring 1024: the scalar kernel)",
        lambda: seqmix.latent_window_attention(qf, q1.float(), D, cf, s8, p8, l1, 1024, 0.07), bytes_=Bd * 1024 * (C + R) * 4)
    ov, g8 = rnd(H, N, V), gate
    add("sigmoid_gate_heads [16, N, 128]", lambda: seqmix.sigmoid_gate_heads(ov, g8), N * H * V * 6)
    hv, hg = rnd(N, H * V), rnd(N, H, dtype=f32)
    add("pulenex sigmoid_gate_mul_ (a gate per head)", lambda: seqmix.sigmoid_gate_mul_(hv, hg), N * H * V * 4, like="sigmoid_gate_heads")
    # router, experts
    lg = rnd(N, E + 1, dtype=f32)
    add("route_topk, 4 groups of 8, 2 kept, renormalised, gate column", lambda: seqmix.route_topk(lg, None, top, E, "sigmoid", 1.0, (4, 2), True, True),
        N * ((E + 1) * 4 + top * 12 + 4))
    lg2 = rnd(N, E, dtype=f32)
    add("naguzen route_topk, sigmoid", lambda: seqmix.route_topk(lg2, None, top, E, "sigmoid"), N * (E * 4 + top * 12), like="route_topk")
    gu = rnd(N * top, 2 * FF)
    add("silu_mul [N x 4, 2 x 704]", lambda: seqmix.silu_mul(gu), N * top * FF * 6)
    mid = rnd(N * top, 1024)
    add("naguzen gelu_erf [N x 4, 1024]", lambda: seqmix.gelu_erf(mid), N * top * 1024 * 4, like="silu_mul")
    up, sel, xs = rnd(E, 2 * FF, W), torch.randint(0, E, (Bd * top,), dtype=i32, device=dev), rnd(Bd * top, W)
    hit = int(sel.unique().numel())
    add("indexed_gemv gated up (8 rows x 4 experts)", lambda: seqmix.indexed_gemv(up, sel, xs, "silu_glu"), hit * 2 * FF * W * 2)
    up1 = rnd(E, 1024, W)
    add("naguzen indexed_gemv up, gelu (8 rows x 4 experts)", lambda: seqmix.indexed_gemv(up1, sel, xs, "gelu"), hit * 1024 * W * 2, like="indexed_gemv")
    return {"peaks": {"hbm_gbs": hbm, "bf16_tflops": tfl, "source": src}, "rows": rows}


def main(args) -> int:
    import torch
    import torch.distributed as dist

    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1"); os.environ.setdefault("MASTER_PORT", "29543")
    dist.init_process_group("nccl", rank=0, world_size=1, device_id=dev)
    from neuronx_distributed_b200.parallel_layers import parallel_state as ps

    ps.initialize_model_parallel(tensor_model_parallel_size=1)
    steps, warmup = max(3, args.steps), max(3, args.warmup)
    out = {"mode": "kulisun", "dtype": "bf16", "data": "synthetic", "steps": steps, "warmup": warmup, "n_gpus": 1,
           "l2": "weights of every model exceed L2; kernel rows flush L2 between iterations"}
    for name, make in (("kulisun", build_kulisun), ("naguzen", base.build_naguzen), ("pulenex", pul.build_pulenex)):
        res = []
        for B, S in ((4, 2048), (1, 8192), (8, 512)):
            model = make(dev, B, S + 64)
            res.append(base.throughput(model, dev, B, S, S, steps, warmup))
            if name == "kulisun" and B == 4:
                out["step_kernels"] = step_profile(model, dev, B, S)
            del model
            torch.cuda.empty_cache()
        out[name] = res
    out["kernels"] = kernel_table(dev, max(steps, 5), warmup)
    print(json.dumps(out), flush=True)
    dist.destroy_process_group()
    return 0
