// Grouped-query attention of single new tokens against their rings on the tensor cores (bfloat16 rows, softmax; window, aligned chunk or
// the whole sequence).  The query heads of one key/value group are the M side of m16n8k16 products (16 at a time), so a group's rows are
// read once for all of them.  With two score maps per head a group's two keys of a position are ONE row of 2 D numbers and each query
// is that long with zeros where the other map's key lies; both maps then share the scores' and the values' products.
// One block = one stretch of the positions a token sees (window and chunk, read on the device, so a long ring costs what is visible and
// a captured graph stays valid while sequences grow) x one group x one tile of 16 heads.  Key and value rows arrive by asynchronous
// copies, 64 positions per tile and up to three tiles ahead.  Per tile: each of the eight warps forms the scores of 8 positions; a warp
// per head turns them into weights (float, running maximum and sum; rounded to bfloat16 only as operands of the value product); each warp
// owns a share of the value columns with float accumulators in registers.
// A stretch leaves its maximum, sum and unnormalised result per head; window_token_merge_kernel (window_attention.cu) folds them.
#include "mma_tiles.cuh"
#include "seq_common.cuh"
#include "seqmix.h"
#include "window_rule.cuh"

namespace seqmix {

static const int kRows = 64;        // positions per tile
static const int kHeads = 16;
static const int kScoreLd = kRows + 4;
static const int kWeightLd = kRows + 8;
static const size_t kTwoPerSm = 110 * 1024, kOnePerSm = 220 * 1024;

static size_t fixed_smem(int KD) {
    return (size_t)kHeads * (KD + 8) * sizeof(bf16) + (size_t)kHeads * kWeightLd * sizeof(bf16) + (size_t)kHeads * (kScoreLd + 1) * sizeof(float);
}
static size_t stage_smem(int KD, int V) { return (size_t)kRows * (KD + V + 16) * sizeof(bf16); }

// how many tiles are staged: as many as leave room for two blocks per SM, two at least
static int stages_of(int KD, int V) {
    const int n = (int)((kTwoPerSm - fixed_smem(KD)) / stage_smem(KD, V));
    return n > 4 ? 4 : (n < 2 ? 2 : n);
}

template <int NP>                   // 16-column value tiles per warp: V <= 128 * NP
__global__ void __launch_bounds__(256)
window_decode_mma_kernel(const bf16* __restrict__ q, long q_sb, const bf16* __restrict__ kcache, const bf16* __restrict__ vcache,
                         const int* __restrict__ slots, const int* __restrict__ pos0, const int* __restrict__ lens, int ring, int H, int G,
                         int D, int V, const WindowRule rule, int stages, int nsplit, float* __restrict__ part_m,
                         float* __restrict__ part_l, float* __restrict__ part_acc) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int M = rule.maps, KD = M * D, ldk = KD + 8, ldv = V + 8, HG = H / G * M, tiles = (HG + kHeads - 1) / kHeads;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);                                  // [kHeads][ldk]
    bf16* Ps = Qs + kHeads * ldk;                                                  // [kHeads][kWeightLd]
    float* Sc = reinterpret_cast<float*>(Ps + kHeads * kWeightLd);                 // [kHeads][kScoreLd]
    float* Corr = Sc + kHeads * kScoreLd;                                          // [kHeads]
    bf16* St = reinterpret_cast<bf16*>(Corr + kHeads);                             // [stages] x ([kRows][ldk], [kRows][ldv])
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int split = blockIdx.x, b = blockIdx.y, gr = blockIdx.z / tiles, h0 = (blockIdx.z - gr * tiles) * kHeads;
    const int nh = min(kHeads, HG - h0);
    const int hq = gr * HG + h0;                                                   // the tile's first query head (maps counted)
    const int p = pos0[b], lo = first_visible(p, rule.window, rule.chunk);
    const int per = ((p - lo + nsplit) / nsplit + kRows - 1) / kRows * kRows;      // positions per stretch, in whole tiles
    const int j0 = lo + split * per, j1 = min(p + 1, j0 + per);
    if (lens[b] <= 0 || j0 >= j1) {
        if (tid < nh) {
            const long o = ((long)b * H * M + hq + tid) * nsplit + split;
            part_m[o] = -INFINITY; part_l[o] = 0.f;
        }
        return;
    }
    const bf16* kb = kcache + ((long)slots[b] * ring * G + gr) * KD;
    const bf16* vb = vcache + ((long)slots[b] * ring * G + gr) * V;
    const int kp8 = KD / 8, row8 = kp8 + V / 8, n = j1 - j0, first = j0 % ring;    // a stretch wraps at most once
    auto fetch = [&](int t) {                                                      // 16-byte pieces of 64 key and value rows
        bf16* Kd = St + (long)(t % stages) * kRows * (ldk + ldv);
        bf16* Vd = Kd + kRows * ldk;
        for (int r = warp; r < kRows; r += 8) {
            const int i = t * kRows + r, at = first + min(i, n - 1);
            const bool on = i < n;
            const long row = (long)(at < ring ? at : at - ring) * G;
            for (int c = lane; c < row8; c += 32) {
                if (c < kp8) cp16(Kd + r * ldk + c * 8, kb + row * KD + c * 8, on);
                else cp16(Vd + r * ldv + (c - kp8) * 8, vb + row * V + (c - kp8) * 8, on);
            }
        }
    };
    const int nt = (j1 - j0 + kRows - 1) / kRows;
    for (int t = 0; t < stages - 1; ++t) {
        if (t < nt) fetch(t);
        cp_commit();
    }
    for (int i = tid; i < kHeads * ldk; i += 256) {                                // queries; zeros where another map's key lies
        const int r = i / ldk, c = i - r * ldk, a = (h0 + r) % M;
        Qs[i] = (r < nh && c >= a * D && c < (a + 1) * D) ? q[(long)b * q_sb + (long)(hq + r) * D + (c - a * D)] : __float2bfloat16_rn(0.f);
    }
    for (int i = tid; i < kHeads * kWeightLd; i += 256) Ps[i] = __float2bfloat16_rn(0.f);
    if (tid < kHeads) Corr[tid] = 1.f;
    const float scale2 = rule.scale * 1.4426950408889634f;
    const int g = lane >> 2, tq = lane & 3;
    float oacc[2 * NP][4];
#pragma unroll
    for (int n = 0; n < 2 * NP; ++n) oacc[n][0] = oacc[n][1] = oacc[n][2] = oacc[n][3] = 0.f;
    float mh[2] = {-INFINITY, -INFINITY}, lh[2] = {0.f, 0.f};                      // heads warp, warp + 8 (lh: this lane's part)
    for (int t = 0; t < nt; ++t) {
        // all but the newest stages - 2 copies have landed: tile t among them
        if (stages == 2) cp_wait<0>(); else if (stages == 3) cp_wait<1>(); else cp_wait<2>();
        __syncthreads();                                                           // for everyone; and everyone has left tile t - 1
        if (t + stages - 1 < nt) fetch(t + stages - 1);
        cp_commit();
        const bf16* Kt = St + (long)(t % stages) * kRows * (ldk + ldv);
        const bf16* Vt = Kt + kRows * ldk;
        float sa[4] = {0.f, 0.f, 0.f, 0.f}, sb[4] = {0.f, 0.f, 0.f, 0.f};
        const bf16* qrow = Qs + (lane & 15) * ldk + (lane >> 4) * 8;
        const bf16* krow = Kt + (warp * 8 + (lane & 7)) * ldk;
        const int ks = KD / 16;
        int k = 0;
#pragma unroll 4
        for (; k + 1 < ks; k += 2) {
            unsigned a[4], c[4], b0, b1, b2, b3;
            ldsm4(b0, b1, b2, b3, krow + k * 16 + (lane >> 3) * 8);
            ldsm4(a[0], a[1], a[2], a[3], qrow + k * 16);
            ldsm4(c[0], c[1], c[2], c[3], qrow + k * 16 + 16);
            mma16816(sa, a, b0, b1);
            mma16816(sb, c, b2, b3);
        }
        if (k < ks) {
            unsigned a[4], b0, b1, b2, b3;
            ldsm4(b0, b1, b2, b3, krow + k * 16 + ((lane >> 3) & 1) * 8);
            ldsm4(a[0], a[1], a[2], a[3], qrow + k * 16);
            mma16816(sa, a, b0, b1);
        }
        float* sd = Sc + g * kScoreLd + warp * 8 + tq * 2;
        *reinterpret_cast<float2*>(sd) = make_float2(sa[0] + sb[0], sa[1] + sb[1]);
        *reinterpret_cast<float2*>(sd + 8 * kScoreLd) = make_float2(sa[2] + sb[2], sa[3] + sb[3]);
        __syncthreads();
        const int left = j1 - (j0 + t * kRows);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = warp + 8 * u;
            if (r >= nh) break;
            const float x = lane < left ? Sc[r * kScoreLd + lane] * scale2 : -INFINITY;
            const float y = lane + 32 < left ? Sc[r * kScoreLd + lane + 32] * scale2 : -INFINITY;
            float mx = fmaxf(x, y);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(mh[u], mx);                                     // finite: a tile has at least one live row
            const float corr = exp2f(mh[u] - mn), ex = exp2f(x - mn), ey = exp2f(y - mn);
            mh[u] = mn;
            lh[u] = fmaf(lh[u], corr, ex + ey);
            Ps[r * kWeightLd + lane] = __float2bfloat16_rn(ex);
            Ps[r * kWeightLd + lane + 32] = __float2bfloat16_rn(ey);
            if (lane == 0) Corr[r] = corr;
        }
        __syncthreads();
        const float c0 = Corr[g], c1 = Corr[g + 8];
#pragma unroll
        for (int n = 0; n < 2 * NP; ++n) { oacc[n][0] *= c0; oacc[n][1] *= c0; oacc[n][2] *= c1; oacc[n][3] *= c1; }
#pragma unroll
        for (int kp = 0; kp < kRows / 16; ++kp) {
            unsigned pa[4];
            ldsm4(pa[0], pa[1], pa[2], pa[3], Ps + (lane & 15) * kWeightLd + kp * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const int c = (warp + i * 8) * 16;
                if (c < V) {
                    unsigned b0, b1, b2, b3;
                    ldsm4t(b0, b1, b2, b3, Vt + (kp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + c + (lane >> 4) * 8);
                    mma16816(oacc[2 * i], pa, b0, b1);
                    mma16816(oacc[2 * i + 1], pa, b2, b3);
                }
            }
        }
    }
    cp_wait<0>();
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int r = warp + 8 * u;
        const float l = warp_sum(lh[u]);
        if (r < nh && lane == 0) {
            const long o = ((long)b * H * M + hq + r) * nsplit + split;
            part_m[o] = mh[u] * 0.69314718055994531f; part_l[o] = l;
        }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int r = g + 8 * u;
        if (r >= nh) continue;
        float* dst = part_acc + (((long)b * H * M + hq + r) * nsplit + split) * V + tq * 2;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int c = (warp + i * 8) * 16;
            if (c < V) {
                *reinterpret_cast<float2*>(dst + c) = make_float2(oacc[2 * i][2 * u], oacc[2 * i][2 * u + 1]);
                *reinterpret_cast<float2*>(dst + c + 8) = make_float2(oacc[2 * i + 1][2 * u], oacc[2 * i + 1][2 * u + 1]);
            }
        }
    }
}

bool window_decode_mma_fits(int D, int V, int maps) {
    const int KD = maps * D;
    return KD % 16 == 0 && D % 8 == 0 && V % 16 == 0 && V <= 512 && fixed_smem(KD) + 2 * stage_smem(KD, V) <= kOnePerSm;
}

// as many stretches as fill the GPU once (one or two blocks per SM), none shorter than two tiles of the ring
int window_decode_mma_splits(int B, int H, int G, int D, int V, int maps, int rows) {
    const int KD = maps * D, units = B * G * ((H / G * maps + kHeads - 1) / kHeads);
    const int per_sm = fixed_smem(KD) + 2 * stage_smem(KD, V) <= kTwoPerSm ? 2 : 1;
    const int want = per_sm * 148 / units, most = (rows + 2 * kRows - 1) / (2 * kRows);
    return want < 1 ? 1 : (want < most ? want : (most < 1 ? 1 : most));
}

void window_decode_mma(const void* q, long q_sb, const void* kcache, const void* vcache, const int* slots, const int* pos0, const int* lens,
                       int ring, int B, int H, int G, int D, int V, const WindowRule& rule, int splits, float* part_m, float* part_l,
                       float* part_acc, cudaStream_t s) {
    const int KD = rule.maps * D, stages = stages_of(KD, V);
    const size_t smem = fixed_smem(KD) + stages * stage_smem(KD, V);
    dim3 grid(splits, B, G * ((H / G * rule.maps + kHeads - 1) / kHeads));
#define SEQMIX_WDM(N)                                                                                                               \
    do {                                                                                                                            \
        cudaFuncSetAttribute(window_decode_mma_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kOnePerSm);             \
        window_decode_mma_kernel<N><<<grid, 256, smem, s>>>((const bf16*)q, q_sb, (const bf16*)kcache, (const bf16*)vcache, slots,  \
                                                            pos0, lens, ring, H, G, D, V, rule, stages, splits, part_m, part_l,     \
                                                            part_acc);                                                              \
    } while (0)
    if (V <= 128) SEQMIX_WDM(1); else if (V <= 256) SEQMIX_WDM(2); else SEQMIX_WDM(4);
#undef SEQMIX_WDM
}

}  // namespace seqmix
