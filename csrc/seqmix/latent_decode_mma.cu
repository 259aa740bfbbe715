// Latent attention for single new tokens (decoding), absorbed form, on the tensor cores (bfloat16 rows).  All heads share a
// sequence's rows, so 16 heads are the M side of m16n8k16 products: scores = queries x rows^T over the C + R coordinates, and the same
// staged rows weighted are the value product over the C latent ones.
// One block = one stretch of a sequence's visible positions x one tile of 16 heads.  The stretches divide what the token sees NOW
// (position and window, read on the device), not the ring, so a long cache costs what the sequence has filled.  Rows arrive by
// asynchronous copies, a tile of 32 ahead of the arithmetic; two blocks share an SM, so one's copies and barriers run under the other's
// arithmetic.  The eight warps split a tile's scores by (8 rows, half of the
// coordinates); each then forms the softmax weights of all 16 x 32 pairs for itself (float; weights are rounded to bfloat16 only as
// operands of the value product) and owns a share of the value columns, with float accumulators in registers.
// A stretch leaves its maximum, sum of weights and unnormalised sums per head; latent_ring_merge_kernel (latent_decode.cu) folds them.
#include "mma_tiles.cuh"
#include "seq_common.cuh"
#include "seqmix.h"

namespace seqmix {

static const int kRows = 32;        // positions per tile
static const int kHeadTile = 16;
static const int kStages = 2;
static const int kWarps = 8;
static const int kScoreLd = kRows + 4;
static const int kMaxRow = 640;     // C + R

template <int NP>                   // pairs of 8-column value tiles per warp: C <= 16 * kWarps * NP
__global__ void __launch_bounds__(32 * kWarps, 2)
latent_decode_mma_kernel(const bf16* __restrict__ qa, long qa_sn, long qa_sh, const bf16* __restrict__ qr, long qr_sn, long qr_sh,
                         const bf16* __restrict__ keys, long key_sb, int ring, const int* __restrict__ key_index,
                         const int* __restrict__ pos0, const int* __restrict__ lens, int H, int C, int R, int window, float scale2,
                         int nsplit, float* __restrict__ part_m, float* __restrict__ part_l, float* __restrict__ part_acc) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int CR = C + R, ld = CR + 8, ks = CR / 16, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);                                  // [kHeadTile][ld]
    bf16* Ks = Qs + kHeadTile * ld;                                                // [kStages][kRows][ld]
    float* Sc = reinterpret_cast<float*>(Ks + kStages * kRows * ld);               // [2 halves][kHeadTile][kScoreLd]
    const int split = blockIdx.x, b = blockIdx.y, h0 = blockIdx.z * kHeadTile, nh = min(kHeadTile, H - h0);
    const long pbase = ((long)b * nsplit + split) * H + h0;
    const int p = pos0[b], lo = max(0, p - window + 1);
    const int per = ((p - lo + nsplit) / nsplit + kRows - 1) / kRows * kRows;      // positions per stretch, in whole tiles
    const int j0 = lo + split * per, j1 = min(p + 1, j0 + per);
    if (lens[b] <= 0 || j0 >= j1) {
        if (tid < nh) { part_m[pbase + tid] = -INFINITY; part_l[pbase + tid] = 0.f; }
        return;
    }
    const bf16* base = keys + (long)(key_index ? key_index[b] : b) * key_sb;
    auto fetch = [&](int t) {                              // a warp per row and pass, a lane per 16-byte piece
        bf16* dst = Ks + (t % kStages) * kRows * ld;
#pragma unroll
        for (int r0 = 0; r0 < kRows; r0 += kWarps) {
            const int r = r0 + warp, j = j0 + t * kRows + r;
            const bf16* src = base + (long)(min(j, j1 - 1) % ring) * CR;
            for (int c = lane * 8; c < CR; c += 256) cp16(dst + r * ld + c, src + c, j < j1);
        }
    };
    const int nt = (j1 - j0 + kRows - 1) / kRows;
    fetch(0);
    cp_commit();
    // the tile's queries: absorbed part, then rotated part; heads past the last are zeros
    for (int i = tid; i < kHeadTile * (C / 8); i += 32 * kWarps) {
        const int h = i / (C / 8), c = (i % (C / 8)) * 8;
        *reinterpret_cast<uint4*>(Qs + h * ld + c) = h < nh ? *reinterpret_cast<const uint4*>(qa + (long)b * qa_sn + (long)(h0 + h) * qa_sh + c)
                                                            : make_uint4(0u, 0u, 0u, 0u);
    }
    for (int i = tid; i < kHeadTile * R; i += 32 * kWarps) {
        const int h = i / R, c = i % R;
        Qs[h * ld + C + c] = h < nh ? qr[(long)b * qr_sn + (long)(h0 + h) * qr_sh + c] : __float2bfloat16_rn(0.f);
    }
    const int g = lane >> 2, tq = lane & 3;
    const int sn = (warp & 3) * 8, kh = warp >> 2;         // this warp's 8 rows of a tile and its half of the coordinates
    const int k0 = kh ? (ks + 1) / 2 : 0, k1 = kh ? ks : (ks + 1) / 2;
    float oacc[2 * NP][4];
#pragma unroll
    for (int n = 0; n < 2 * NP; ++n) oacc[n][0] = oacc[n][1] = oacc[n][2] = oacc[n][3] = 0.f;
    float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
    for (int t = 0; t < nt; ++t) {
        cp_wait<0>();
        __syncthreads();                                   // tile t (and the queries) are here; everyone has left tile t - 1
        if (t + 1 < nt) fetch(t + 1);
        cp_commit();
        const bf16* Kt = Ks + (t % kStages) * kRows * ld;
        float sacc[4] = {0.f, 0.f, 0.f, 0.f}, sacd[4] = {0.f, 0.f, 0.f, 0.f};
        const bf16* qrow = Qs + (lane & 15) * ld + (lane >> 4) * 8;
        const bf16* krow = Kt + (sn + (lane & 7)) * ld;
        int k = k0;
#pragma unroll 4
        for (; k + 1 < k1; k += 2) {                       // two steps of 16 coordinates per row load
            unsigned a[4], c[4], b0, b1, b2, b3;
            ldsm4(b0, b1, b2, b3, krow + k * 16 + (lane >> 3) * 8);
            ldsm4(a[0], a[1], a[2], a[3], qrow + k * 16);
            ldsm4(c[0], c[1], c[2], c[3], qrow + k * 16 + 16);
            mma16816(sacc, a, b0, b1);
            mma16816(sacd, c, b2, b3);
        }
        if (k < k1) {
            unsigned a[4], b0, b1, b2, b3;
            ldsm4(b0, b1, b2, b3, krow + k * 16 + ((lane >> 3) & 1) * 8);
            ldsm4(a[0], a[1], a[2], a[3], qrow + k * 16);
            mma16816(sacc, a, b0, b1);
        }
        float* sd = Sc + (kh * kHeadTile + g) * kScoreLd + sn + tq * 2;
        *reinterpret_cast<float2*>(sd) = make_float2(sacc[0] + sacd[0], sacc[1] + sacd[1]);
        *reinterpret_cast<float2*>(sd + 8 * kScoreLd) = make_float2(sacc[2] + sacd[2], sacc[3] + sacd[3]);
        __syncthreads();
        // weights of heads g and g + 8 for all 32 rows, in the layout of the value product's left operand (base 2)
        float w[2][2][4];                                  // [head][16-row step][2 + 2 columns]
        float mx[2] = {-INFINITY, -INFINITY};
        const int left = j1 - (j0 + t * kRows);
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int kp = 0; kp < 2; ++kp)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int col = kp * 16 + e * 8 + tq * 2;
                    const float* s0 = Sc + (g + 8 * r) * kScoreLd + col;
                    const float2 x = *reinterpret_cast<const float2*>(s0), y = *reinterpret_cast<const float2*>(s0 + kHeadTile * kScoreLd);
                    w[r][kp][2 * e] = col < left ? (x.x + y.x) * scale2 : -INFINITY;
                    w[r][kp][2 * e + 1] = col + 1 < left ? (x.y + y.y) * scale2 : -INFINITY;
                    mx[r] = fmaxf(mx[r], fmaxf(w[r][kp][2 * e], w[r][kp][2 * e + 1]));
                }
        float corr[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float mn = fmaxf(mrow[r], mx[r]);        // finite: a tile has at least one live row
            corr[r] = exp2f(mrow[r] - mn);
            mrow[r] = mn;
            float ls = 0.f;
#pragma unroll
            for (int kp = 0; kp < 2; ++kp)
#pragma unroll
                for (int e = 0; e < 4; ++e) { w[r][kp][e] = exp2f(w[r][kp][e] - mn); ls += w[r][kp][e]; }
            lrow[r] = lrow[r] * corr[r] + ls;
        }
#pragma unroll
        for (int n = 0; n < 2 * NP; ++n) { oacc[n][0] *= corr[0]; oacc[n][1] *= corr[0]; oacc[n][2] *= corr[1]; oacc[n][3] *= corr[1]; }
#pragma unroll
        for (int kp = 0; kp < 2; ++kp) {
            unsigned pa[4];
            pa[0] = pack2(w[0][kp][0], w[0][kp][1]);
            pa[1] = pack2(w[1][kp][0], w[1][kp][1]);
            pa[2] = pack2(w[0][kp][2], w[0][kp][3]);
            pa[3] = pack2(w[1][kp][2], w[1][kp][3]);
#pragma unroll
            for (int i = 0; i < NP; ++i) {
                const int c = (warp + i * kWarps) * 16;
                if (c < C) {
                    unsigned b0, b1, b2, b3;
                    ldsm4t(b0, b1, b2, b3, Kt + (kp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + c + (lane >> 4) * 8);
                    mma16816(oacc[2 * i], pa, b0, b1);
                    mma16816(oacc[2 * i + 1], pa, b2, b3);
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 1);
        lrow[r] += __shfl_xor_sync(0xffffffffu, lrow[r], 2);
        const int h = g + 8 * r;
        if (h >= nh) continue;
        if (warp == 0 && tq == 0) { part_m[pbase + h] = mrow[r] * 0.69314718055994531f; part_l[pbase + h] = lrow[r]; }
        float* dst = part_acc + (pbase + h) * C + tq * 2;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int c = (warp + i * kWarps) * 16;
            if (c < C) {
                *reinterpret_cast<float2*>(dst + c) = make_float2(oacc[2 * i][2 * r], oacc[2 * i][2 * r + 1]);
                *reinterpret_cast<float2*>(dst + c + 8) = make_float2(oacc[2 * i + 1][2 * r], oacc[2 * i + 1][2 * r + 1]);
            }
        }
    }
}

bool latent_decode_mma_fits(int C, int R) { return C % 16 == 0 && R % 16 == 0 && C > 0 && C + R <= kMaxRow; }

// as many stretches as fill the GPU once (two blocks per SM), but none shorter than a tile
int latent_decode_mma_splits(int B, int H, int rows) {
    const int units = B * ((H + kHeadTile - 1) / kHeadTile), want = 2 * 148 / units, most = (rows + kRows - 1) / kRows;
    return want < 1 ? 1 : (want < most ? want : (most < 1 ? 1 : most));
}

void latent_decode_mma(const void* qa, long qa_sn, long qa_sh, const void* qr, long qr_sn, long qr_sh, const void* keys, long key_sb, int ring,
                       const int* key_index, const int* pos0, const int* lens, int B, int H, int C, int R, int window, float scale,
                       int nsplit, float* part_m, float* part_l, float* part_acc, cudaStream_t s) {
    const size_t smem = (size_t)(kHeadTile + kStages * kRows) * (C + R + 8) * sizeof(bf16) + 2 * kHeadTile * kScoreLd * sizeof(float);
    dim3 grid(nsplit, B, (H + kHeadTile - 1) / kHeadTile);
#define SEQMIX_LDM(N)                                                                                                               \
    do {                                                                                                                            \
        cudaFuncSetAttribute(latent_decode_mma_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);                 \
        latent_decode_mma_kernel<N><<<grid, 32 * kWarps, smem, s>>>((const bf16*)qa, qa_sn, qa_sh, (const bf16*)qr, qr_sn, qr_sh,   \
                                                                    (const bf16*)keys, key_sb, ring, key_index, pos0, lens, H, C, R, \
                                                                    window, scale * 1.4426950408889634f, nsplit, part_m, part_l,    \
                                                                    part_acc);                                                      \
    } while (0)
    if (C <= 128) SEQMIX_LDM(1); else if (C <= 256) SEQMIX_LDM(2); else if (C <= 512) SEQMIX_LDM(4); else SEQMIX_LDM(5);
#undef SEQMIX_LDM
}

}  // namespace seqmix
