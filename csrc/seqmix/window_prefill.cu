// Grouped-query attention (sliding window, aligned chunks or every earlier position) over a prompt as one fused tensor-core kernel
// (bfloat16 operands): scores, score cap, mask, softmax and the weighted sum of values never leave the chip.  A block owns 64
// consecutive queries of one (sequence, query head); its four warps own 16 queries each; the query heads of a group read the same key /
// value head (through L2).  Key / value
// tiles of 64 positions are staged in shared memory by asynchronous copies, one tile ahead of the arithmetic.  Scores come from
// mma.sync m16n8k16 products with float accumulation; they are scaled, capped (cap * tanh(s / cap), the tanh formed from one base-2
// exponential), masked and exponentiated in float with a running maximum and sum per query; the weights are rounded to bfloat16
// only as operands of the value product, whose accumulator is float.  The result is multiplied by sigmoid(gate) and a constant and
// written with a free row stride.  Position i sees j with 0 <= i - j < window and, with chunks, i / chunk == j / chunk: the tiles before a
// block's first chunk are never fetched.  A sink is where the running maximum and sum start.  Queries at or past lens[b] give zeros.
// MAPS = 2 (differential attention): eight warps, four for each score map of the head, share the staged value tiles; at the end the
// second map's results cross over through shared memory and the first four warps write unit(a1 - lam a2) * post.
// SIG: every visible key's weight is sigmoid(score + bias[h]) by itself (no running maximum, no sum, no division at the end).
// Sizes: key and value sizes are multiples of 16 up to 16 * DK16 / 16 * VD16 (template bounds; the real sizes are arguments).
#include "mma_tiles.cuh"
#include "seq_common.cuh"
#include "seqmix.h"
#include "window_rule.cuh"

namespace seqmix {

constexpr int kQT = 64, kKT = 64, kPad = 8;     // queries / keys per tile; row padding (elements) against bank conflicts

template <int DK16, int VD16, bool SIG, int MAPS>
__global__ void __launch_bounds__(128 * MAPS)
window_prompt_mma_kernel(const bf16* __restrict__ q, long q_sb, long q_st, const bf16* __restrict__ k, long k_sb, long k_st,
                         const bf16* __restrict__ v, long v_sb, long v_st, const bf16* __restrict__ gate, long g_sb, long g_st,
                         const int* __restrict__ lens, int S, int H, int G, int DK, int VD,
                         const WindowRule rule, bf16* __restrict__ out, long out_stride, float out_scale) {
    constexpr int NT = 128 * MAPS, NW = 4 * MAPS;
    const float softcap = rule.softcap, scale = rule.scale;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dk16 = DK / 16, vd16 = VD / 16, ldk = DK + kPad, ldv = VD + kPad;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);          // [MAPS][kQT][ldk] queries, then key stage 1 (same size)
    // the blocks of the last queries, which see the most keys, start first
    auto Kst = [&](int st) { return st ? Qs : Qs + MAPS * kQT * ldk; };                        // [MAPS][kKT][ldk] each
    auto Vst = [&](int st) { return Qs + MAPS * (kQT + kKT) * ldk + (st ? kKT * ldv : 0); };   // [kKT][ldv] each
    const int q0 = (gridDim.z - 1 - blockIdx.z) * kQT, h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int hk = h / (H / G), map = warp >> 2;           // this warp's score map
    const int len = min(lens[b], S);
    bf16* ob = out + ((long)b * S) * out_stride + (long)h * VD;
    if (q0 >= len) {                                       // nothing but padding: zeros
        for (int i = tid; i < min(kQT, S - q0) * (VD / 2); i += NT) {
            const int r = i / (VD / 2), c = (i % (VD / 2)) * 2;
            *reinterpret_cast<unsigned*>(ob + (long)(q0 + r) * out_stride + c) = 0u;
        }
        return;
    }
    const uint4 zero4 = make_uint4(0u, 0u, 0u, 0u);
    for (int i = tid; i < MAPS * kQT * (DK / 8); i += NT) {
        const int mr = i / (DK / 8), c = (i % (DK / 8)) * 8, r = mr % kQT, t = q0 + r;
        *reinterpret_cast<uint4*>(Qs + mr * ldk + c) =
            t < S ? *reinterpret_cast<const uint4*>(q + (long)b * q_sb + (long)t * q_st + (long)(h * MAPS + mr / kQT) * DK + c) : zero4;
    }
    __syncthreads();
    const int r0 = (warp & 3) * 16, g = lane >> 2, tq = lane & 3;
    unsigned qa[DK16][4];
#pragma unroll
    for (int kk = 0; kk < DK16; ++kk)
        if (kk < dk16) ldsm4(qa[kk][0], qa[kk][1], qa[kk][2], qa[kk][3], Qs + (map * kQT + r0 + (lane & 15)) * ldk + kk * 16 + (lane >> 4) * 8);
    float oacc[2 * VD16][4];
#pragma unroll
    for (int n = 0; n < 2 * VD16; ++n) oacc[n][0] = oacc[n][1] = oacc[n][2] = oacc[n][3] = 0.f;
    const int i0 = q0 + r0 + g, i1 = i0 + 8;               // this thread's two queries
    const float log2e = 1.4426950408889634f;
    const float start = rule.sink ? rule.sink[h * MAPS + map] * log2e : -INFINITY, lstart = rule.sink && tq == 0 ? 1.f : 0.f;
    float mrow[2] = {start, start}, lrow[2] = {lstart, lstart};      // lrow: this thread's part of the sum
    const int last_lo = first_visible(q0 + r0 + 15, rule.window, rule.chunk);        // of the warp's last query
    const int lo0 = first_visible(i0, rule.window, rule.chunk), lo1 = first_visible(i1, rule.window, rule.chunk);
    const float scale2 = scale * log2e;                    // uncapped scores go straight to base 2
    const float cap_in = softcap > 0.f ? 2.f * log2e * scale / softcap : 0.f, cap_out = softcap * log2e;
    const float sbias2 = SIG ? rule.score_bias[h] * log2e : 0.f;
    const int jlo = first_visible(q0, rule.window, rule.chunk), jhi = min(q0 + kQT - 1, len - 1);
    const bf16* kb = k + (long)b * k_sb + (long)hk * MAPS * DK;        // a group's key heads lie side by side
    const bf16* vb = v + (long)b * v_sb + (long)hk * VD;
    auto fetch = [&](int kt, int st) {
        const int j0 = kt * kKT;
        bf16 *Kd = Kst(st), *Vd = Vst(st);
        for (int c = lane * 8; c < DK; c += 256) {
#pragma unroll 4
            for (int r = warp; r < MAPS * kKT; r += NW) {
                const int j = j0 + r % kKT;
                cp16(Kd + r * ldk + c, kb + (long)min(j, len - 1) * k_st + (MAPS > 1 ? (r / kKT) * DK : 0) + c, j < len);
            }
        }
        for (int c = lane * 8; c < VD; c += 256) {
#pragma unroll 4
            for (int r = warp; r < kKT; r += NW) {
                const int j = j0 + r;
                cp16(Vd + r * ldv + c, vb + (long)min(j, len - 1) * v_st + c, j < len);
            }
        }
        cp_commit();
    };
    const int kt0 = jlo / kKT, kt1 = jhi / kKT;
    __syncthreads();                                       // every warp holds its queries: their room becomes key stage 1
    fetch(kt0, 0);
    for (int kt = kt0; kt <= kt1; ++kt) {
        const int j0 = kt * kKT, st = (kt - kt0) & 1;
        if (kt < kt1) { fetch(kt + 1, st ^ 1); cp_wait<1>(); } else cp_wait<0>();
        __syncthreads();                                   // tile kt has landed for everyone
        const bf16 *Ks = Kst(st) + map * kKT * ldk, *Vs = Vst(st);
        float sacc[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n) sacc[n][0] = sacc[n][1] = sacc[n][2] = sacc[n][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DK16; ++kk) {
            if (kk < dk16) {
#pragma unroll
                for (int np = 0; np < 4; ++np) {           // two 8-key groups per ldmatrix
                    unsigned b0, b1, b2, b3;
                    ldsm4(b0, b1, b2, b3, Ks + (np * 16 + (lane & 7) + ((lane >> 4) << 3)) * ldk + kk * 16 + ((lane >> 3) & 1) * 8);
                    mma16816(sacc[2 * np], qa[kk], b0, b1);
                    mma16816(sacc[2 * np + 1], qa[kk], b2, b3);
                }
            }
        }
        // scale, cap, mask, running softmax (float, in base 2); a thread holds 16 scores of query i0 and 16 of i1.  A tile that every
        // query of the warp sees in full needs no mask.
        const bool full = j0 + kKT - 1 <= q0 + r0 && j0 >= last_lo && j0 + kKT - 1 < len;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                bool vis = true;
                if (!full) {
                    const int j = j0 + n * 8 + tq * 2 + (e & 1);
                    vis = j <= (e < 2 ? i0 : i1) && j >= (e < 2 ? lo0 : lo1) && j < len;
                }
                float sc;
                if (softcap > 0.f) {                       // cap tanh(x) = cap (1 - 2 / (1 + e^(2x))), already times log2(e)
                    const float t = exp2f(fminf(sacc[n][e] * cap_in, 126.f));
                    sc = cap_out * (1.f - __fdividef(2.f, 1.f + t));
                } else {
                    sc = sacc[n][e] * scale2;
                }
                if (SIG) {                                 // sigmoid(x) = 1 / (1 + 2^(-x log2 e)); sc already holds x log2 e
                    sacc[n][e] = vis ? __fdividef(1.f, 1.f + exp2f(fminf(-(sc + sbias2), 126.f))) : 0.f;
                } else {
                    sacc[n][e] = vis ? sc : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], sacc[n][e]);
                }
            }
        float corr[2], base[2];
        if (!SIG) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float mn = fmaxf(mrow[r], mx[r]);
            base[r] = mn == -INFINITY ? 0.f : mn;          // nothing visible so far: every weight is exp(-inf) = 0
            corr[r] = exp2f(mrow[r] - base[r]);
            mrow[r] = mn;
        }
        float ls[2] = {0.f, 0.f};
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                sacc[n][e] = exp2f(sacc[n][e] - base[e >> 1]);
                ls[e >> 1] += sacc[n][e];
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) lrow[r] = lrow[r] * corr[r] + ls[r];
#pragma unroll
        for (int n = 0; n < 2 * VD16; ++n) { oacc[n][0] *= corr[0]; oacc[n][1] *= corr[0]; oacc[n][2] *= corr[1]; oacc[n][3] *= corr[1]; }
        }
#pragma unroll
        for (int kp = 0; kp < 4; ++kp) {
            unsigned pa[4];
            pa[0] = pack2(sacc[2 * kp][0], sacc[2 * kp][1]);
            pa[1] = pack2(sacc[2 * kp][2], sacc[2 * kp][3]);
            pa[2] = pack2(sacc[2 * kp + 1][0], sacc[2 * kp + 1][1]);
            pa[3] = pack2(sacc[2 * kp + 1][2], sacc[2 * kp + 1][3]);
#pragma unroll
            for (int nv = 0; nv < VD16; ++nv) {
                if (nv < vd16) {
                    unsigned b0, b1, b2, b3;
                    ldsm4t(b0, b1, b2, b3, Vs + (kp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + nv * 16 + (lane >> 4) * 8);
                    mma16816(oacc[2 * nv], pa, b0, b1);
                    mma16816(oacc[2 * nv + 1], pa, b2, b3);
                }
            }
        }
        __syncthreads();                                   // the stage may be refilled
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 1);
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 2);
    }
    if (SIG) lrow[0] = lrow[1] = 1.f;
    float inv0 = (i0 < len && lrow[0] > 0.f) ? out_scale / lrow[0] : 0.f, inv1 = (i1 < len && lrow[1] > 0.f) ? out_scale / lrow[1] : 0.f;
    if constexpr (MAPS == 2) {
        // every warp has passed the last tile's barrier: the stages' room takes the second map's results
        float* X = reinterpret_cast<float*>(smem_raw);     // [kQT][VD + 4]
        const int ldx = VD + 4;
        inv0 = (i0 < len && lrow[0] > 0.f) ? 1.f / lrow[0] : 0.f;
        inv1 = (i1 < len && lrow[1] > 0.f) ? 1.f / lrow[1] : 0.f;
        if (map == 1) {
#pragma unroll
            for (int n = 0; n < 2 * VD16; ++n)
                if (n < 2 * vd16) {
                    float* x = X + (r0 + g) * ldx + n * 8 + tq * 2;
                    *reinterpret_cast<float2*>(x) = make_float2(oacc[n][0] * inv0, oacc[n][1] * inv0);
                    *reinterpret_cast<float2*>(x + 8 * ldx) = make_float2(oacc[n][2] * inv1, oacc[n][3] * inv1);
                }
        }
        __syncthreads();
        if (map == 1) return;
        const float lam = rule.lam[0];
        float ss[2] = {0.f, 0.f};
#pragma unroll
        for (int n = 0; n < 2 * VD16; ++n)
            if (n < 2 * vd16) {
                const float* x = X + (r0 + g) * ldx + n * 8 + tq * 2;
                const float2 u = *reinterpret_cast<const float2*>(x), w = *reinterpret_cast<const float2*>(x + 8 * ldx);
                oacc[n][0] = oacc[n][0] * inv0 - lam * u.x; oacc[n][1] = oacc[n][1] * inv0 - lam * u.y;
                oacc[n][2] = oacc[n][2] * inv1 - lam * w.x; oacc[n][3] = oacc[n][3] * inv1 - lam * w.y;
                ss[0] += oacc[n][0] * oacc[n][0] + oacc[n][1] * oacc[n][1];
                ss[1] += oacc[n][2] * oacc[n][2] + oacc[n][3] * oacc[n][3];
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 1);
            ss[r] += __shfl_xor_sync(0xffffffffu, ss[r], 2);
        }
        inv0 = rule.post * out_scale / sqrtf(ss[0] / (float)VD + rule.eps);
        inv1 = rule.post * out_scale / sqrtf(ss[1] / (float)VD + rule.eps);
    }
    if (gate) {
        if (i0 < len) inv0 *= sigmoidf_(__bfloat162float(gate[(long)b * g_sb + (long)i0 * g_st + h]));
        if (i1 < len) inv1 *= sigmoidf_(__bfloat162float(gate[(long)b * g_sb + (long)i1 * g_st + h]));
    }
#pragma unroll
    for (int n = 0; n < 2 * VD16; ++n) {
        if (n < 2 * vd16) {
            const int c = n * 8 + tq * 2;
            if (i0 < S) *reinterpret_cast<unsigned*>(ob + (long)i0 * out_stride + c) = pack2(oacc[n][0] * inv0, oacc[n][1] * inv0);
            if (i1 < S) *reinterpret_cast<unsigned*>(ob + (long)i1 * out_stride + c) = pack2(oacc[n][2] * inv1, oacc[n][3] * inv1);
        }
    }
}

static size_t prompt_smem(int D, int V, int maps) {
    return (size_t)(maps * (kQT + kKT) * (D + kPad) + 2 * kKT * (V + kPad)) * sizeof(bf16);   // the maps' exchange fits into it
}

// The fused kernel takes bfloat16 with key and value sizes in whole 16s up to 256 and 16-byte aligned rows.
bool window_prompt_mma_fits(const void* q, long q_sb, long q_st, const void* k, long k_sb, long k_st, const void* v, long v_sb, long v_st,
                            int D, int V, int maps, const void* out, long out_stride) {
    auto a16 = [](const void* p) { return (uintptr_t)p % 16 == 0; };
    return D % 16 == 0 && V % 16 == 0 && D <= (maps == 2 ? 128 : 256) && V <= 256 && a16(q) && a16(k) && a16(v) && (uintptr_t)out % 4 == 0 &&
           q_sb % 8 == 0 && q_st % 8 == 0 && k_sb % 8 == 0 && k_st % 8 == 0 && v_sb % 8 == 0 && v_st % 8 == 0 && out_stride % 2 == 0;
}

template <int DK16, int VD16, bool SIG, int MAPS>
static void prompt_launch(const bf16* q, long q_sb, long q_st, const bf16* k, long k_sb, long k_st, const bf16* v, long v_sb, long v_st,
                          const bf16* gate, long g_sb, long g_st, const int* lens, int B, int S, int H, int G, int D, int V,
                          const WindowRule& rule, bf16* out, long out_stride, float out_scale, cudaStream_t s) {
    cudaFuncSetAttribute(window_prompt_mma_kernel<DK16, VD16, SIG, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    window_prompt_mma_kernel<DK16, VD16, SIG, MAPS><<<dim3(H, B, (S + kQT - 1) / kQT), 128 * MAPS, prompt_smem(D, V, MAPS), s>>>(
        q, q_sb, q_st, k, k_sb, k_st, v, v_sb, v_st, gate, g_sb, g_st, lens, S, H, G, D, V, rule, out, out_stride, out_scale);
}

void window_prompt_mma(const void* q, long q_sb, long q_st, const void* k, long k_sb, long k_st, const void* v, long v_sb, long v_st,
                       const void* gate, long g_sb, long g_st, const int* lens, int B, int S, int H, int G, int D, int V,
                       const WindowRule& rule, void* out, long out_stride, float out_scale, cudaStream_t s) {
#define SEQMIX_WPM_S(A, Bv, SG, M)                                                                                                    \
    prompt_launch<A, Bv, SG, M>((const bf16*)q, q_sb, q_st, (const bf16*)k, k_sb, k_st, (const bf16*)v, v_sb, v_st, (const bf16*)gate,   \
                                g_sb, g_st, lens, B, S, H, G, D, V, rule, (bf16*)out, out_stride, out_scale, s)
    if (rule.maps == 2) {
        if (D <= 64 && V <= 128) SEQMIX_WPM_S(4, 8, false, 2);
        else if (V <= 128) SEQMIX_WPM_S(8, 8, false, 2);
        else SEQMIX_WPM_S(8, 16, false, 2);
        return;
    }
#define SEQMIX_WPM(A, Bv) do { if (rule.score_bias) SEQMIX_WPM_S(A, Bv, true, 1); else SEQMIX_WPM_S(A, Bv, false, 1); } while (0)
    if (D <= 64 && V <= 64) SEQMIX_WPM(4, 4);
    else if (D <= 128 && V <= 128) SEQMIX_WPM(8, 8);
    else SEQMIX_WPM(16, 16);
#undef SEQMIX_WPM
#undef SEQMIX_WPM_S
}

}  // namespace seqmix
