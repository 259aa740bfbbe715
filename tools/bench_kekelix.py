"""``bench.py --mode kekelix``: serving throughput of the Kekelix design at layer sizes that resemble a real model (random weights), beside
the framework's closest existing models at equal width and depth — Noresun (grouped-query attention through the same kernels, routed
experts) and Kulisun (attention over whole sequences, routed gated experts) — plus every kernel the design added or extended, timed alone
against the measured copy bandwidth / GEMM throughput, beside the like kernel of those paths.  One GPU, bfloat16.  Device time (CUDA
events), >= 3 warm-up iterations; the weights of every model exceed L2, and the kernel timings flush L2 (a 512 MiB write) between
iterations; every kernel row is replayed from a CUDA graph.

Layers (width 2048): differential attention of 8 heads / 2 key-value heads (two maps of 128, value 256) over the whole sequence | chunks of
1024 positions, 16 / 4 heads of 128 whose keys are the values, 64 rotated | the whole sequence, 16 / 4 heads of 128 with biases, rotation
of all coordinates with interpolated frequencies and a sink | the chunked layer again; each beside 32 clamped gated experts of 704, 4 chosen."""
from __future__ import annotations

import json
import math
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "tools"))

import bench_kulisun as kul  # noqa: E402
import bench_naguzen as base  # noqa: E402
import bench_noresun as nor  # noqa: E402

WIDTH, VOCAB = base.WIDTH, base.VOCAB
YARN = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}


def kekelix_layers():
    moe = {"kind": "moe", "expert": {"ff": 704, "limit": 7.0}, "router": {"experts": 32, "top": 4}}
    s = 1.0 / math.sqrt(128)
    diff = {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 256, "scale": s, "diff": 0.3}
    chunk = {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": s, "mask": {"size": 1024}, "rot": {"base": 500000.0, "dims": 64}}
    sink = {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": s, "rot": {"base": 10000.0, "dims": 128, "scaling": YARN}}
    lay = lambda kind, mixer: {"type": kind, "mixer": mixer, "mlp": moe}
    return [lay("attention", diff), lay("attention_3", chunk), lay("attention_2", sink), lay("attention_3", chunk)]


def build_kekelix(dev, batch, max_len):
    import torch

    from neuronx_distributed_b200.models.kekelix import KekelixConfig, KekelixForInference

    cfg = KekelixConfig(vocab=VOCAB, width=WIDTH, layers=kekelix_layers(), norm_eps=1e-6, loop=(0, 2, 1), dtype=torch.bfloat16, device=dev)
    m = KekelixForInference(cfg, batch_size=batch, max_seq_len=max_len).eval()
    g = torch.Generator(device=dev).manual_seed(0)
    with torch.no_grad():
        for name, p in m.named_parameters():
            if p.dim() > 1:
                p.normal_(0.0, 0.02, generator=g)
                if "router" in name:                       # as a checkpoint stored in bfloat16 would hold it
                    p.copy_(p.to(torch.bfloat16).float())
            elif name.endswith("lam"):
                p.fill_(0.4)
        m.lm.embed.normal_(0.0, 1.0, generator=g)
    return m


def kernel_table(dev, steps, warmup):
    """Each kernel the design added or extended, alone at the sizes of the model above (4 x 2048 prompt tokens; 8 decoding rows) → time,
    achieved GB/s or TFLOP/s, fraction of the measured peak; the like kernel of an existing path in the row after it."""
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
    l1, s8 = ints(1, Bd), torch.arange(Bd, dtype=i32, device=dev)
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

    # residual sum of mixer result and expert rows, two norms, the embedding and a vector
    top, E, FF = 4, 32, 704
    x32, y16, vec = rnd(N, W, dtype=f32), rnd(N, W), torch.ones(W, device=dev)
    er, src_i, wt, gw = rnd(N * top, W), torch.randperm(N * top, device=dev).to(i32).view(N, top), rnd(N, top, dtype=f32), rnd(N, dtype=f32)
    table, tok = rnd(VOCAB, W), torch.randint(0, VOCAB, (N,), device=dev)
    add("residual_norm_: 4 expert rows + mixer result, two norms",
        lambda: seqmix.residual_norm_(x32, er, None, vec, None, 1e-6, False, (src_i, None, y16, None), vec), N * W * (top * 2 + 2 + 4 + 4 + 4))
    add("residual_norm_: the same + embedding row + vector", lambda: seqmix.residual_norm_(
        x32, er, None, vec, None, 1e-6, False, (src_i, None, y16, None), vec, (tok, table, vec)), N * W * (top * 2 + 2 + 2 + 4 + 4 + 4))
    add("kulisun residual_norm_: 4 weighted expert rows + shared, layer norm",
        lambda: seqmix.residual_norm_(x32, er, vec, vec, vec, 1e-6, True, (src_i, wt, y16, gw)), N * W * (top * 2 + 2 + 4 + 4 + 2), like="residual_norm_")
    # preparation
    H, G, D, dims, chunk = 16, 4, 128, 64, 1024
    inv, invy, amp = seqmix.rotary_inv_freq(dims, 500000.0, dev), seqmix.rotary_inv_freq(D, 10000.0, dev, YARN), seqmix.rotary_amplitude(YARN)
    p = rnd(B, S, (H + 2 * G) * D)
    q, k, v = p[..., :H * D].unflatten(-1, (H, D)), p[..., H * D:(H + G) * D].unflatten(-1, (G, D)), p[..., (H + G) * D:].unflatten(-1, (G, D))
    kout = torch.empty(B, S, G, D, dtype=bf, device=dev)
    cc, fc = [torch.zeros(B, chunk, G, D, dtype=bf, device=dev) for _ in "kv"], [torch.zeros(B, S, G, D, dtype=bf, device=dev) for _ in "kv"]
    dc = [torch.zeros(B, S, 4, D, dtype=bf, device=dev), torch.zeros(B, S, 2, 2 * D, dtype=bf, device=dev)]
    add("window_qk_prepare: rotation, then unit norm; keys are values, ring 1024", lambda: seqmix.window_qk_prepare(
        q, k, k, None, None, 1e-6, pos0, lens, slots, *cc, inv_freq=inv, rot_dims=dims, unit=True, kout=kout), N * (2 * H + 2 * G) * D * 2 + B * chunk * 2 * G * D * 2)
    add("window_qk_prepare: rotation of all coordinates with an amplitude, every row cached", lambda: seqmix.window_qk_prepare(
        q, k, v, None, None, 1e-6, pos0, lens, slots, *fc, inv_freq=invy, rot_dims=D, amp=amp), N * (2 * H + 5 * G) * D * 2)
    kd, vd = p[..., H * D:H * D + 4 * D].unflatten(-1, (4, D)), p[..., (H + G) * D:(H + G) * D + 4 * D].unflatten(-1, (2, 2 * D))
    add("window_qk_prepare: two maps, no rotation (cache rows only)", lambda: seqmix.window_qk_prepare(
        q, kd, vd, None, None, 1e-6, pos0, lens, slots, *dc), N * 16 * D * 2)
    qwa, kwa = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
    add("noresun window_qk_prepare: one norm over all heads, rotation, ring 1024", lambda: seqmix.window_qk_prepare(
        q, k, v, qwa, kwa, 1e-6, pos0, lens, slots, *cc, norm_all=True, inv_freq=inv, rot_dims=dims), N * (H + G) * D * 4 + B * chunk * G * 2 * D * 4,
        like="window_qk_prepare")
    # prompt attention
    out, sink, lam = torch.empty(N, H * D, dtype=bf, device=dev), torch.zeros(H, device=dev), torch.full((1,), 0.4, device=dev)
    full_pairs, chunk_pairs = B * sum(t + 1 for t in range(S)), B * sum(t % chunk + 1 for t in range(S))
    win_pairs = B * sum(min(t + 1, 1024) for t in range(S))
    diff = (lam, 1e-6, 0.7)
    add("window_attention_prompt: two maps joined, 8/2 heads of 2 x 128, value 256, whole sequence", lambda: seqmix.window_attention_prompt(
        q, kd, vd, None, lens, FULL, 0.088, 0.0, out, 1.0, diff=diff), flops=8 * full_pairs * 2 * 2 * (D + 2 * D))
    add("window_attention_prompt: sink, 16/4 heads of 128, whole sequence", lambda: seqmix.window_attention_prompt(
        q, k, v, None, lens, FULL, 0.088, 0.0, out, 1.0, sink=sink), flops=H * full_pairs * 4 * D)
    add("window_attention_prompt: chunks of 1024, 16/4 heads of 128", lambda: seqmix.window_attention_prompt(
        q, kout, k, None, lens, FULL, 0.088, 0.0, out, 1.0, chunk=chunk), flops=H * chunk_pairs * 4 * D)
    hgate = rnd(B, S, H)
    add("pinirax window_attention_prompt: window 1024, cap, gate", lambda: seqmix.window_attention_prompt(
        q, k, v, hgate, lens, 1024, 0.088, 30.0, out, 0.8), flops=H * win_pairs * 4 * D, like="window_attention_prompt")
    pb = torch.full((H,), -2.0, device=dev)
    add("noresun window_attention_prompt: window 1024, sigmoid weights", lambda: seqmix.window_attention_prompt(
        q, k, v, None, lens, 1024, 0.088, 0.0, out, 1.0, pb), flops=H * win_pairs * 4 * D, like="window_attention_prompt")
    # single tokens
    q1, o1 = rnd(Bd, 1, H, D), torch.empty(Bd, H * D, dtype=bf, device=dev)
    for L in (2048, 16384):
        kc, vc, kc2, vc2, pl = rnd(Bd, L, G, D), rnd(Bd, L, G, D), rnd(Bd, L, 4, D), rnd(Bd, L, 2, 2 * D), ints(L - 1, Bd)
        add(f"window_attention_token: two maps joined, {L} cached (8 rows)", lambda: seqmix.window_attention_token(
            q1, kc2, vc2, None, s8, pl, l1, FULL, 0.088, 0.0, o1, 1.0, diff=diff), bytes_=Bd * L * G * D * 4)
        add(f"window_attention_token: sink, {L} cached (8 rows)", lambda: seqmix.window_attention_token(
            q1, kc, vc, None, s8, pl, l1, FULL, 0.088, 0.0, o1, 1.0, sink=sink), bytes_=Bd * L * G * D * 4)
    kc, vc, pl = rnd(Bd, chunk, G, D), rnd(Bd, chunk, G, D), ints(2047, Bd)
    add("window_attention_token: chunk of 1024 (8 rows)", lambda: seqmix.window_attention_token(
        q1, kc, vc, None, s8, pl, l1, FULL, 0.088, 0.0, o1, 1.0, chunk=chunk), bytes_=Bd * chunk * G * D * 4)
    g1 = rnd(Bd, 1, H)
    add("pinirax window_attention_token: ring 1024, cap, gate (8 rows)", lambda: seqmix.window_attention_token(
        q1, kc, vc, g1, s8, pl, l1, 1024, 0.088, 30.0, o1, 0.8), bytes_=Bd * 1024 * G * D * 4, like="window_attention_token")
    keys, qa1, q1l, pk = rnd(Bd, 2048, 576), rnd(H, Bd, 512), rnd(Bd, 1, H, 192), ints(2047, Bd)
    add("kulisun latent_window_attention, 2048 cached, sink (8 rows)", lambda: seqmix.latent_window_attention(
        qa1, q1l, 128, keys, s8, pk, l1, FULL, 0.07, sink), bytes_=Bd * 2048 * 576 * 2, like="window_attention_token")
    # experts
    gu, rs = rnd(N * top, 2 * FF), torch.rand(N * top, device=dev)
    add("clamped_glu with a number per row [N x 4, 2 x 704]", lambda: seqmix.clamped_glu(gu, 7.0, 1.702, rs), N * top * FF * 6)
    add("kulisun silu_mul [N x 4, 2 x 704]", lambda: seqmix.silu_mul(gu), N * top * FF * 6, like="clamped_glu")
    up, sel, xs, xw = rnd(E, 2 * FF, W), torch.randint(0, E, (Bd * top,), dtype=i32, device=dev), rnd(Bd * top, W), torch.rand(Bd * top, device=dev)
    hit = int(sel.unique().numel())
    add("indexed_gemv clamped gate, weighted input (8 rows x 4 experts)", lambda: seqmix.indexed_gemv(up, sel, xs, "clamped_glu", xw, 7.0, 1.702),
        hit * 2 * FF * W * 2)
    add("kulisun indexed_gemv gated (8 rows x 4 experts)", lambda: seqmix.indexed_gemv(up, sel, xs, "silu_glu"), hit * 2 * FF * W * 2, like="indexed_gemv")
    return {"peaks": {"hbm_gbs": hbm, "bf16_tflops": tfl, "source": src}, "rows": rows}


def main(args) -> int:
    import torch
    import torch.distributed as dist

    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1"); os.environ.setdefault("MASTER_PORT", "29545")
    dist.init_process_group("nccl", rank=0, world_size=1, device_id=dev)
    from neuronx_distributed_b200.parallel_layers import parallel_state as ps

    ps.initialize_model_parallel(tensor_model_parallel_size=1)
    steps, warmup = max(3, args.steps), max(3, args.warmup)
    out = {"mode": "kekelix", "dtype": "bf16", "data": "synthetic", "steps": steps, "warmup": warmup, "n_gpus": 1,
           "l2": "weights of every model exceed L2; kernel rows flush L2 between iterations"}
    for name, make in (("kekelix", build_kekelix), ("noresun", nor.build_noresun), ("kulisun", kul.build_kulisun)):
        res = []
        for B, S in ((4, 2048), (1, 8192), (8, 512)):
            model = make(dev, B, S + 64)
            res.append(base.throughput(model, dev, B, S, S, steps, warmup))
            if name == "kekelix" and B == 4:
                out["step_kernels"] = kul.step_profile(model, dev, B, S)
            del model
            torch.cuda.empty_cache()
        out[name] = res
    out["kernels"] = kernel_table(dev, max(steps, 5), warmup)
    print(json.dumps(out), flush=True)
    dist.destroy_process_group()
    return 0
