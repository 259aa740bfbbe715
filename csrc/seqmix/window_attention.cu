// Grouped-query attention over the last `window` positions (or all of them, or an aligned chunk of positions): query position i sees
// j <= i with i - j < window and, when chunks are given, i / chunk == j / chunk; query head h reads key/value head
// h / (H/G).  Scores are q.k * scale, capped as softcap * tanh(score / softcap) when softcap > 0; scores, weights and sums are
// float.  The weights are a softmax over the visible keys (whose denominator also holds exp(sink[h]) when sinks are given), or — when
// a score bias per head is given — sigmoid(score + bias[h]) of
// each visible key by itself, not normalised over the keys.  Each head's result may be multiplied by sigmoid(gate[b,t,h]) and a
// constant before it is written (row stride free: several mixers write side by side into one buffer).
// Two maps per head (differential attention): a head has two queries and a key/value group two keys side by side, each map is a softmax
// of its own over the SAME values, and the head's result is unit(a1 - lam * a2) * post with unit(o) = o / sqrt(mean(o^2) + eps).
// In the kernels below "query head" then counts maps: head * 2 + map.
//   window_qk_prepare      : RMS norm of queries and keys, per head (one weight vector of D numbers each) or over the whole
//                            projection at once (weights of H*D and G*D numbers); then, when frequencies are given, rotation of the
//                            first `dims` coordinates of every head at the token's position (pairs i, i + dims/2; angles in float,
//                            cos and sin times `amp`, formed once per token for all heads); or rotation first and then a norm without
//                            weights per head (`unit`); in place, or the keys to a tensor of their own when the projected keys serve
//                            as the values;
//                            and the last `ring` real tokens' keys and values to the sequence's ring rows (position mod ring);
//                            with no keys given only the queries are prepared (a layer that reads another layer's ring)
//   window_attention_prompt: prompts starting at position 0, keys and values of the call itself.  A block owns 16 consecutive
//                            queries of one head (4 warps x 4 queries); key / value rows come through shared memory 32 at a time;
//                            in the score pass a lane owns one key (4 queries per shared-memory read), in the value pass a lane
//                            owns value columns lane, lane + 32, ...  (float, and bfloat16 of sizes the fused tensor-core kernel
//                            of window_prefill.cu does not take); two maps leave float results that map_combine_kernel joins
//   window_attention_token : one query per (sequence, head) against the ring.  A block owns up to 4 query heads of one key/value
//                            group (a warp each) over one stretch of the visible positions, staged 32 rows at a time for all of them
//                            (bfloat16 softmax without a cap: the tensor-core kernel of window_decode_mma.cu); a
//                            second kernel folds the stretches' partial softmaxes, adds the sink and joins the maps.
#include <math.h>

#include "seq_common.cuh"
#include "seqmix.h"
#include "window_rule.cuh"

namespace seqmix {

template <typename T>
__global__ void window_qk_prepare_kernel(T* q, long q_sb, long q_st, T* k, long k_sb, long k_st, T* kout, long ko_sb, long ko_st,
                                         const T* v, long v_sb, long v_st, const float* __restrict__ qw, const float* __restrict__ kw,
                                         int norm_all, int unit, float eps, const float* __restrict__ inv_freq, int dims, float amp,
                                         const int* __restrict__ pos0, const int* __restrict__ lens, const int* __restrict__ slots,
                                         T* kcache, T* vcache, int ring, int S, int H, int GK, int G, int D, int V) {
    extern __shared__ float trig[];                          // cos, then sin, of the token's angles (times amp)
    __shared__ float red[2][8];
    const int row = blockIdx.x, b = row / S, t = row - b * S, lane = threadIdx.x, tid = threadIdx.y * 32 + lane, nthr = blockDim.y * 32;
    const int len = min(lens[b], S);
    if (t >= len) return;
    const bool keep = k != nullptr && t >= len - ring;
    const int pos = pos0[b] + t, half = inv_freq ? dims / 2 : 0, rot = 2 * half;
    const long cr = k ? (long)slots[b] * ring + pos % ring : 0;
    T* qrow = q + (long)b * q_sb + (long)t * q_st;
    T* krow = k ? k + (long)b * k_sb + (long)t * k_st : nullptr;
    T* korow = k ? kout + (long)b * ko_sb + (long)t * ko_st : nullptr;   // the keys themselves unless they double as values
    for (int i = tid; i < half; i += nthr) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        trig[i] = cs * amp; trig[half + i] = sn * amp;
    }
    float inv_all[2] = {1.f, 1.f};
    if (norm_all) {                                          // one statistic over all heads of the queries, one over all of the keys
        float sq = 0.f, sk = 0.f;
        if (qw) for (int x = tid; x < H * D; x += nthr) { const float e = ldf(qrow + x); sq = fmaf(e, e, sq); }
        if (kw && krow) for (int x = tid; x < GK * D; x += nthr) { const float e = ldf(krow + x); sk = fmaf(e, e, sk); }
        sq = warp_sum(sq); sk = warp_sum(sk);
        if (lane == 0) { red[0][threadIdx.y] = sq; red[1][threadIdx.y] = sk; }
    }
    __syncthreads();
    if (norm_all) {
        float sq = 0.f, sk = 0.f;
        for (int x = 0; x < (int)blockDim.y; ++x) { sq += red[0][x]; sk += red[1][x]; }
        inv_all[0] = 1.f / sqrtf(sq / (float)(H * D) + eps);
        inv_all[1] = 1.f / sqrtf(sk / (float)(GK * D) + eps);
    }
    const int units = krow ? H + GK + G : H;
    for (int u = threadIdx.y; u < units; u += blockDim.y) {
        if (u < H + GK) {
            const bool isq = u < H;
            const int hh = isq ? u : u - H;
            const T* p = (isq ? qrow : krow) + (long)hh * D;
            T* o = (isq ? qrow : korow) + (long)hh * D;
            const float* w = isq ? qw : kw;
            T* dst = (!isq && keep) ? kcache + (cr * GK + hh) * D : nullptr;
            const bool moved = o != p;
            float inv = 1.f;
            if (w && norm_all) {
                inv = inv_all[isq ? 0 : 1];
                w += (long)hh * D;
            } else if (w || unit) {                          // a rotation multiplies the pairs' squares by amp^2 and nothing else
                float ss = 0.f;
                for (int d = lane; d < D; d += 32) { float x = ldf(p + d); if (unit && d < rot) x *= amp; ss = fmaf(x, x, ss); }
                inv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
            }
            if (!(w || dst || rot || unit || moved)) continue;
            for (int i = lane; i < half; i += 32) {          // a lane reads both members of a pair before it writes them
                float x0 = ldf(p + i), x1 = ldf(p + i + half);
                if (w) { x0 *= inv * w[i]; x1 *= inv * w[i + half]; }
                const float cs = trig[i], sn = trig[half + i];
                float y0 = x0 * cs - x1 * sn, y1 = x1 * cs + x0 * sn;
                if (unit) { y0 *= inv; y1 *= inv; }
                stf(o + i, y0); stf(o + i + half, y1);
                if (dst) { stf(dst + i, y0); stf(dst + i + half, y1); }
            }
            for (int d = rot + lane; d < D; d += 32) {
                const float x = w ? ldf(p + d) * inv * w[d] : (unit ? ldf(p + d) * inv : ldf(p + d));
                if (w || unit || moved) stf(o + d, x);
                if (dst) stf(dst + d, x);
            }
        } else if (keep) {
            const int hh = u - H - GK;
            const T* p = v + (long)b * v_sb + (long)t * v_st + (long)hh * V;
            T* dst = vcache + (cr * G + hh) * V;
            for (int d = lane; d < V; d += 32) dst[d] = p[d];
        }
    }
}

// The same for heads of at most 32 E coordinates (E = 4 or 8) whose rows start on whole fours and whose rotated halves are whole E: a warp
// holds a head, E consecutive coordinates per lane, read once; a pair's other half comes from the lane half / E away.
template <typename T, int E>
__global__ void __launch_bounds__(256)
window_qk_prepare_vec_kernel(T* q, long q_sb, long q_st, T* k, long k_sb, long k_st, T* kout, long ko_sb, long ko_st, const T* v, long v_sb,
                             long v_st, const float* __restrict__ qw, const float* __restrict__ kw, int norm_all, int unit, float eps,
                             const float* __restrict__ inv_freq, int dims, float amp, const int* __restrict__ pos0,
                             const int* __restrict__ lens, const int* __restrict__ slots, T* kcache, T* vcache, int ring, int S, int H, int GK,
                             int G, int D, int V) {
    extern __shared__ __align__(16) float trig[];            // cos, then sin, of the token's angles (times amp)
    __shared__ float red[2][8];
    const int row = blockIdx.x, b = row / S, t = row - b * S, lane = threadIdx.x, tid = threadIdx.y * 32 + lane;
    const int len = min(lens[b], S);
    if (t >= len) return;
    const bool keep = k != nullptr && t >= len - ring;
    const int pos = pos0[b] + t, half = inv_freq ? dims / 2 : 0, rot = 2 * half;
    const long cr = k ? (long)slots[b] * ring + pos % ring : 0;
    T* qrow = q + (long)b * q_sb + (long)t * q_st;
    T* krow = k ? k + (long)b * k_sb + (long)t * k_st : nullptr;
    T* korow = k ? kout + (long)b * ko_sb + (long)t * ko_st : nullptr;
    for (int i = tid; i < half; i += 256) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        trig[i] = cs * amp; trig[half + i] = sn * amp;
    }
    if (norm_all) {
        float sq = 0.f, sk = 0.f;
        if (qw) for (int x = tid * 4; x < H * D; x += 1024) { const float4 e = ld4(qrow + x); sq += e.x * e.x + e.y * e.y + e.z * e.z + e.w * e.w; }
        if (kw && krow) for (int x = tid * 4; x < GK * D; x += 1024) { const float4 e = ld4(krow + x); sk += e.x * e.x + e.y * e.y + e.z * e.z + e.w * e.w; }
        sq = warp_sum(sq); sk = warp_sum(sk);
        if (lane == 0) { red[0][threadIdx.y] = sq; red[1][threadIdx.y] = sk; }
    }
    if (norm_all || half) __syncthreads();
    float inv_all[2] = {1.f, 1.f};
    if (norm_all) {
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int x = 0; x < 8; ++x) { sq += red[0][x]; sk += red[1][x]; }
        inv_all[0] = 1.f / sqrtf(sq / (float)(H * D) + eps);
        inv_all[1] = 1.f / sqrtf(sk / (float)(GK * D) + eps);
    }
    auto load = [](float (&x)[E], const T* src) {
#pragma unroll
        for (int e = 0; e < E; e += 4) { const float4 a = ld4(src + e); x[e] = a.x; x[e + 1] = a.y; x[e + 2] = a.z; x[e + 3] = a.w; }
    };
    auto loadf = [](float (&x)[E], const float* src) {
#pragma unroll
        for (int e = 0; e < E; e += 4) { const float4 a = ld4(src + e); x[e] = a.x; x[e + 1] = a.y; x[e + 2] = a.z; x[e + 3] = a.w; }
    };
    auto store = [](T* dst, const float (&x)[E]) {
#pragma unroll
        for (int e = 0; e < E; e += 4) st4(dst + e, make_float4(x[e], x[e + 1], x[e + 2], x[e + 3]));
    };
    const int c = lane * E, shift = half / E;                // this lane's coordinates; lanes between the members of a pair
    const bool in = c < D;
    const bool touch_q = qw || rot || unit;                  // otherwise the queries stay as they are
    const int first = touch_q ? 0 : H, units = krow ? H + GK + (keep ? G : 0) : H;
    for (int u = first + threadIdx.y; u < units; u += 8) {
        if (u < H + GK) {
            const bool isq = u < H;
            const int hh = isq ? u : u - H;
            const T* p = (isq ? qrow : krow) + (long)hh * D;
            T* o = (isq ? qrow : korow) + (long)hh * D;
            const float* w = isq ? qw : kw;
            float x[E];
            if (in) load(x, p + c);
            else {
#pragma unroll
                for (int e = 0; e < E; ++e) x[e] = 0.f;
            }
            float inv = 1.f;
            if (w && norm_all) {
                inv = inv_all[isq ? 0 : 1];
                w += (long)hh * D;
            } else if (w || unit) {
                const float a = unit && c < rot ? amp : 1.f;
                float ss = 0.f;
#pragma unroll
                for (int e = 0; e < E; ++e) ss = fmaf(x[e] * a, x[e] * a, ss);
                inv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
            }
            if (w && in) {
                float g[E];
                loadf(g, w + c);
#pragma unroll
                for (int e = 0; e < E; ++e) x[e] *= inv * g[e];
            }
            if (rot) {
                const bool low = c < half, turn = c < rot;
                const int other = turn ? (low ? lane + shift : lane - shift) : lane;
                float y[E];
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] = __shfl_sync(0xffffffffu, x[e], other);
                if (turn) {
                    const float* cs = trig + (low ? c : c - half);
#pragma unroll
                    for (int e = 0; e < E; ++e) {
                        const float sn = cs[half + e];
                        x[e] = low ? x[e] * cs[e] - y[e] * sn : x[e] * cs[e] + y[e] * sn;
                    }
                }
            }
            if (unit) {
#pragma unroll
                for (int e = 0; e < E; ++e) x[e] *= inv;
            }
            if (!in) continue;
            if (w || rot || unit || o != p) store(o + c, x);
            if (!isq && keep) store(kcache + (cr * GK + hh) * D + c, x);
        } else {
            const int hh = u - H - GK;
            const T* p = v + (long)b * v_sb + (long)t * v_st + (long)hh * V;
            T* dst = vcache + (cr * G + hh) * V;
            for (int d = lane * 4; d < V; d += 128) {
                if (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst + d) = *reinterpret_cast<const uint2*>(p + d);
                else *reinterpret_cast<uint4*>(dst + d) = *reinterpret_cast<const uint4*>(p + d);
            }
        }
    }
}

__device__ __forceinline__ float cap_score(float s, float softcap, float inv_cap) { return softcap > 0.f ? softcap * tanhf(s * inv_cap) : s; }

constexpr int kKeys = 32;       // keys per shared-memory chunk
constexpr int kQW = 4;          // queries per warp (prompts)
constexpr int kWarps = 4;

// shared: Ks [kKeys][D+1], Vs [kKeys][V], Qs [kWarps][D][kQW], Ps [kWarps][kKeys][kQW].  blockIdx.y: head * maps + map; with `fout` the
// results go there as float [B*S, H*maps*V] (no gate, no factor).
template <typename T, int VPL>
__global__ void __launch_bounds__(128) window_prompt_kernel(
    const T* __restrict__ q, long q_sb, long q_st, const T* __restrict__ k, long k_sb, long k_st, const T* __restrict__ v, long v_sb,
    long v_st, const T* __restrict__ gate, long g_sb, long g_st, const int* __restrict__ lens, int S, int H, int G, int D, int V,
    const WindowRule rule, float* __restrict__ fout, T* __restrict__ out, long out_stride, float out_scale) {
    extern __shared__ float sm[];
    const int DP = D + 1;
    float* Ks = sm;
    float* Vs = Ks + kKeys * DP;
    float* Qs = Vs + kKeys * V;
    float* Ps = Qs + kWarps * D * kQW;
    const int i0 = blockIdx.x * (kWarps * kQW), h = blockIdx.y, b = blockIdx.z, g = (h / rule.maps) / (H / G);
    const int gk = g * rule.maps + h % rule.maps;
    const bool sig = rule.score_bias != nullptr;                     // independent sigmoid weights instead of a softmax
    const float sbias = sig ? rule.score_bias[h] : 0.f;
    const int tid = threadIdx.x, lane = tid & 31, wp = tid >> 5;
    const int len = min(lens[b], S);
    const int iq0 = i0 + wp * kQW;                                   // this warp's first query position
    float* Qw = Qs + wp * D * kQW;
    float* Pw = Ps + wp * kKeys * kQW;
    for (int x = lane; x < D * kQW; x += 32) {
        const int d = x / kQW, rq = x - d * kQW, i = iq0 + rq;
        Qw[x] = i < len ? ldf(q + (long)b * q_sb + (long)i * q_st + (long)h * D + d) : 0.f;
    }
    float m[kQW], l[kQW], acc[kQW][VPL];
    int lo[kQW];
#pragma unroll
    for (int rq = 0; rq < kQW; ++rq) {
        m[rq] = rule.sink ? rule.sink[h] : -INFINITY; l[rq] = rule.sink && lane == 0 ? 1.f : 0.f;
        lo[rq] = first_visible(iq0 + rq, rule.window, rule.chunk);
#pragma unroll
        for (int c = 0; c < VPL; ++c) acc[rq][c] = 0.f;
    }
    const float inv_cap = rule.softcap > 0.f ? 1.f / rule.softcap : 0.f;
    const int last = min(i0 + kWarps * kQW, len) - 1;                // last key any query of the block sees
    const int first = first_visible(i0, rule.window, rule.chunk);
    const T* kb = k + (long)b * k_sb + (long)gk * D;
    const T* vb = v + (long)b * v_sb + (long)g * V;
    for (int c0 = first; c0 <= last; c0 += kKeys) {
        __syncthreads();
        for (int x = tid; x < kKeys * D; x += 128) {
            const int jj = x / D, d = x - jj * D, j = c0 + jj;
            Ks[jj * DP + d] = j <= last ? ldf(kb + (long)j * k_st + d) : 0.f;
        }
        for (int x = tid; x < kKeys * V; x += 128) {
            const int jj = x / V, d = x - jj * V, j = c0 + jj;
            Vs[x] = j <= last ? ldf(vb + (long)j * v_st + d) : 0.f;
        }
        __syncthreads();
        // is any of this warp's queries inside the chunk's reach?
        if (c0 > iq0 + kQW - 1 || c0 + kKeys - 1 < lo[0] || iq0 >= len) continue;
        float s[kQW];
#pragma unroll
        for (int rq = 0; rq < kQW; ++rq) s[rq] = 0.f;
        const float* kr = Ks + lane * DP;
        for (int d = 0; d < D; ++d) {
            const float kv = kr[d];
            const float4 qv = *reinterpret_cast<const float4*>(Qw + d * kQW);
            s[0] = fmaf(qv.x, kv, s[0]); s[1] = fmaf(qv.y, kv, s[1]); s[2] = fmaf(qv.z, kv, s[2]); s[3] = fmaf(qv.w, kv, s[3]);
        }
        const int j = c0 + lane;
        float corr[kQW];
#pragma unroll
        for (int rq = 0; rq < kQW; ++rq) {
            const int i = iq0 + rq;
            const bool ok = i < len && j <= i && j >= lo[rq];
            const float sc = ok ? cap_score(s[rq] * rule.scale, rule.softcap, inv_cap) : -INFINITY;
            if (sig) {
                corr[rq] = 1.f;
                Pw[lane * kQW + rq] = ok ? sigmoidf_(sc + sbias) : 0.f;
                continue;
            }
            float mx = sc;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float mn = fmaxf(m[rq], mx);
            const float p = (ok && mn > -INFINITY) ? expf(sc - mn) : 0.f;
            corr[rq] = (m[rq] > -INFINITY) ? expf(m[rq] - mn) : 0.f;
            m[rq] = mn;
            l[rq] = fmaf(l[rq], corr[rq], p);                        // per-lane part of the sum; folded at the end
            Pw[lane * kQW + rq] = p;
        }
#pragma unroll
        for (int rq = 0; rq < kQW; ++rq)
#pragma unroll
            for (int c = 0; c < VPL; ++c) acc[rq][c] *= corr[rq];
        __syncwarp();
        for (int jj = 0; jj < kKeys; ++jj) {
            const float4 p = *reinterpret_cast<const float4*>(Pw + jj * kQW);
#pragma unroll
            for (int c = 0; c < VPL; ++c) {
                const int col = lane + 32 * c;
                const float vv = col < V ? Vs[jj * V + col] : 0.f;
                acc[0][c] = fmaf(p.x, vv, acc[0][c]); acc[1][c] = fmaf(p.y, vv, acc[1][c]);
                acc[2][c] = fmaf(p.z, vv, acc[2][c]); acc[3][c] = fmaf(p.w, vv, acc[3][c]);
            }
        }
        __syncwarp();
    }
#pragma unroll
    for (int rq = 0; rq < kQW; ++rq) {
        const int i = iq0 + rq;
        if (i >= S) continue;
        const float lt = sig ? 1.f : warp_sum(l[rq]);
        float f = 0.f;
        if (i < len && lt > 0.f) {
            f = fout ? 1.f / lt : out_scale / lt;
            if (gate) f *= sigmoidf_(ldf(gate + (long)b * g_sb + (long)i * g_st + h));
        }
        if (fout) {
            float* o = fout + (((long)b * S + i) * H * rule.maps + h) * V;
#pragma unroll
            for (int c = 0; c < VPL; ++c)
                if (lane + 32 * c < V) o[lane + 32 * c] = acc[rq][c] * f;
            continue;
        }
        T* o = out + ((long)b * S + i) * out_stride + (long)h * V;
#pragma unroll
        for (int c = 0; c < VPL; ++c) {
            const int col = lane + 32 * c;
            if (col < V) stf(o + col, acc[rq][c] * f);
        }
    }
}

// a [rows * H, 2, V] float → out[row, h*V..] = unit(a1 - lam * a2) * post * out_scale, a warp per (row, head); zero rows stay zero
template <typename T>
__global__ void map_combine_kernel(const float* __restrict__ a, const float* __restrict__ lam, float eps, float f, long rows, int H, int V,
                                   T* __restrict__ out, long out_stride) {
    const long u = (long)blockIdx.x * blockDim.y + threadIdx.y;
    const int lane = threadIdx.x;
    if (u >= rows * H) return;
    const float* a1 = a + u * 2 * V;
    const float la = lam[0];
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) { const float x = a1[c] - la * a1[V + c]; ss = fmaf(x, x, ss); }
    const float inv = f / sqrtf(warp_sum(ss) / (float)V + eps);
    T* o = out + (u / H) * out_stride + (u % H) * V;
    for (int c = lane; c < V; c += 32) stf(o + c, (a1[c] - la * a1[V + c]) * inv);
}

// ring rows first, first + 1, ... (mod ring); 16 bytes at a time when the row allows it (VEC), else element by element; rows at or past
// `valid` become zeros
template <typename T, bool VEC>
__device__ __forceinline__ void stage_rows(float* dst, int ld, const T* __restrict__ src, long row_stride, int first, int ring, int valid,
                                           int cols, int tid, int nthr) {
    constexpr int E = VEC ? 16 / sizeof(T) : 1;
    const int per = cols / E;
    for (int x = tid; x < kKeys * per; x += nthr) {
        const int jj = x / per, c = (x - jj * per) * E;
        float* d = dst + jj * ld + c;
        int r = first + jj;
        if (r >= ring) r %= ring;
        const T* s = src + (long)r * row_stride + c;
        if (VEC) {
            if (jj < valid) {
                const uint4 raw = *reinterpret_cast<const uint4*>(s);
                const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int u = 0; u < E; ++u) d[u] = ldf(e + u);
            } else {
#pragma unroll
                for (int u = 0; u < E; ++u) d[u] = 0.f;
            }
        } else {
            d[0] = jj < valid ? ldf(s) : 0.f;
        }
    }
}

// Single tokens against their rings.  grid (stretches, head quads, sequences): a block takes up to 4 query heads that read one key
// head (a warp each) over one stretch of the positions the token sees, staged 32 rows at a time for all of them, and leaves a partial
// softmax per head: part_m / part_l [B, heads, splits], part_acc [B, heads, splits, V] (heads counts maps).  shared: Ks [kKeys][D+1],
// Vs [kKeys][V], Qs [4][D], Ps [4][kKeys]
template <typename T, int VPL, bool VEC>
__global__ void __launch_bounds__(128) window_token_kernel(
    const T* __restrict__ q, long q_sb, const T* __restrict__ kcache, const T* __restrict__ vcache, const int* __restrict__ slots,
    const int* __restrict__ pos0, const int* __restrict__ lens, int ring, int H, int G, int D, int V, const WindowRule rule, int splits,
    float* __restrict__ part_m, float* __restrict__ part_l, float* __restrict__ part_acc) {
    extern __shared__ float sm[];
    const int DP = D + 1;
    float* Ks = sm;
    float* Vs = Ks + kKeys * DP;
    float* Qs = Vs + kKeys * V;
    float* Ps = Qs + kWarps * D;
    const int M = rule.maps, split = blockIdx.x, b = blockIdx.z, HG = H / G, qpg = (HG + kWarps - 1) / kWarps;
    const int gk = blockIdx.y / qpg, hq = (blockIdx.y - gk * qpg) * kWarps, g = gk / M;      // key head (counts maps), its value head
    const int tid = threadIdx.x, lane = tid & 31, wp = tid >> 5;
    const bool has = hq + wp < HG;                                   // this warp has a head
    const int h = (g * HG + hq + wp) * M + gk % M;
    const bool sig = rule.score_bias != nullptr;                     // independent sigmoid weights: the partial results are plain sums
    const float sbias = (sig && has) ? rule.score_bias[h] : 0.f;
    const int p = pos0[b], lo = first_visible(p, rule.window, rule.chunk);
    const int n = lens[b] > 0 ? p - lo + 1 : 0;                      // positions the token sees
    int per = (n + splits - 1) / splits;
    per = (per + kKeys - 1) / kKeys * kKeys;
    const int r0 = min(n, split * per), r1 = min(n, r0 + per);
    float* Qw = Qs + wp * D;
    float* Pw = Ps + wp * kKeys;
    if (has)
        for (int d = lane; d < D; d += 32) Qw[d] = ldf(q + (long)b * q_sb + (long)h * D + d);
    float m = -INFINITY, l = 0.f, acc[VPL];
#pragma unroll
    for (int c = 0; c < VPL; ++c) acc[c] = 0.f;
    const float inv_cap = rule.softcap > 0.f ? 1.f / rule.softcap : 0.f;
    const int GK = G * M;
    const T* kb = kcache + (long)slots[b] * ring * GK * D + (long)gk * D;
    const T* vb = vcache + (long)slots[b] * ring * G * V + (long)g * V;
    for (int c0 = r0; c0 < r1; c0 += kKeys) {
        const int first = (lo + c0) % ring;
        __syncthreads();
        stage_rows<T, VEC>(Ks, DP, kb, (long)GK * D, first, ring, r1 - c0, D, tid, 128);
        stage_rows<T, VEC>(Vs, V, vb, (long)G * V, first, ring, r1 - c0, V, tid, 128);
        __syncthreads();
        if (!has) continue;
        float s = 0.f;
        const float* kr = Ks + lane * DP;
        for (int d = 0; d < D; ++d) s = fmaf(Qw[d], kr[d], s);
        const bool ok = c0 + lane < r1;
        const float sc = ok ? cap_score(s * rule.scale, rule.softcap, inv_cap) : -INFINITY;
        float pr, corr;
        if (sig) {
            pr = ok ? sigmoidf_(sc + sbias) : 0.f;
            corr = 1.f;
        } else {
            float mx = sc;
#pragma unroll
            for (int w = 16; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
            const float mn = fmaxf(m, mx);
            pr = (ok && mn > -INFINITY) ? expf(sc - mn) : 0.f;
            corr = (m > -INFINITY) ? expf(m - mn) : 0.f;
            m = mn;
            l = fmaf(l, corr, pr);
        }
        Pw[lane] = pr;
#pragma unroll
        for (int c = 0; c < VPL; ++c) acc[c] *= corr;
        __syncwarp();
        for (int jj = 0; jj < kKeys; ++jj) {
            const float pj = Pw[jj];
#pragma unroll
            for (int c = 0; c < VPL; ++c) {
                const int col = lane + 32 * c;
                acc[c] = fmaf(pj, col < V ? Vs[jj * V + col] : 0.f, acc[c]);
            }
        }
        __syncwarp();
    }
    if (!has) return;
    l = warp_sum(l);
    if (sig) { m = 0.f; l = split == 0 ? 1.f : 0.f; }              // the merge then adds the stretches' sums and divides by one
    const long o = ((long)b * H * M + h) * splits + split;
    if (lane == 0) { part_m[o] = m; part_l[o] = l; }
#pragma unroll
    for (int c = 0; c < VPL; ++c) {
        const int col = lane + 32 * c;
        if (col < V) part_acc[o * V + col] = acc[c];
    }
}

// grid (H, B), 8 warps: the stretches' partial softmaxes of one (sequence, head) folded, with the sink in the denominator; the maps joined;
// gated, scaled and written.  A warp adds every eighth stretch; the warps' sums meet in shared memory.
// shared: sums [8][V], heads [maps][V], one float per warp, weights [maps][splits]
template <typename T>
__global__ void __launch_bounds__(256) window_token_merge_kernel(const float* __restrict__ part_m, const float* __restrict__ part_l,
                                                                 const float* __restrict__ part_acc, const T* __restrict__ gate, long g_sb,
                                                                 int H, int V, int splits, const int* __restrict__ lens,
                                                                 const WindowRule rule, T* __restrict__ out, long out_stride,
                                                                 float out_scale) {
    extern __shared__ __align__(16) float sm[];
    const int M = rule.maps, h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* Rs = sm;
    float* As = Rs + 8 * V;
    float* red = As + M * V;
    float* Ws = red + 8;
    T* dst = out + (long)b * out_stride + (long)h * V;
    if (lens[b] <= 0) {
        for (int c = tid; c < V; c += 256) stf(dst + c, 0.f);
        return;
    }
    for (int a = 0; a < M; ++a) {
        const int hh = h * M + a;
        const long o = ((long)b * H * M + hh) * splits;
        float mt = rule.sink ? rule.sink[hh] : -INFINITY;
        for (int s = lane; s < splits; s += 32) mt = fmaxf(mt, part_m[o + s]);
#pragma unroll
        for (int w = 16; w > 0; w >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, w));
        float lt = 0.f;
        for (int s = lane; s < splits; s += 32) {
            const float pm = part_m[o + s], pl = part_l[o + s], e = pm > -INFINITY ? expf(pm - mt) : 0.f;
            if (warp == 0) Ws[a * splits + s] = e;
            lt = fmaf(pl, e, lt);
        }
        lt = warp_sum(lt);
        if (rule.sink) lt += expf(rule.sink[hh] - mt);
        const float inv = lt > 0.f ? 1.f / lt : 0.f;
        __syncthreads();
        if (V % 4 == 0) {                                            // a stretch that saw nothing left its sums unwritten: not added
            for (int c = lane * 4; c < V; c += 128) {
                float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
                for (int s = warp; s < splits; s += 8) {
                    const float e = Ws[a * splits + s];
                    const float4 x = ld4(part_acc + (o + s) * V + c);
                    acc.x = e > 0.f ? fmaf(x.x, e, acc.x) : acc.x; acc.y = e > 0.f ? fmaf(x.y, e, acc.y) : acc.y;
                    acc.z = e > 0.f ? fmaf(x.z, e, acc.z) : acc.z; acc.w = e > 0.f ? fmaf(x.w, e, acc.w) : acc.w;
                }
                st4(Rs + warp * V + c, acc);
            }
        } else {
            for (int c = lane; c < V; c += 32) {
                float acc = 0.f;
#pragma unroll 4
                for (int s = warp; s < splits; s += 8) {
                    const float e = Ws[a * splits + s], x = part_acc[(o + s) * V + c];
                    acc = e > 0.f ? fmaf(x, e, acc) : acc;
                }
                Rs[warp * V + c] = acc;
            }
        }
        __syncthreads();
        for (int c = tid; c < V; c += 256) {
            float x = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) x += Rs[w * V + c];
            As[a * V + c] = x * inv;
        }
    }
    float f = out_scale;
    if (M == 2) {
        __syncthreads();
        const float la = rule.lam[0];
        float ss = 0.f;
        for (int c = tid; c < V; c += 256) {
            const float x = As[c] - la * As[V + c];
            As[c] = x;
            ss = fmaf(x, x, ss);
        }
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) ss += red[w];
        f *= rule.post / sqrtf(ss / (float)V + rule.eps);
    }
    if (gate) f *= sigmoidf_(ldf(gate + (long)b * g_sb + h));
    for (int c = tid; c < V; c += 256) stf(dst + c, As[c] * f);      // a thread meets its own columns
}

void window_qk_prepare(void* q, long q_sb, long q_st, void* k, long k_sb, long k_st, void* kout, long ko_sb, long ko_st, const void* v,
                       long v_sb, long v_st, int bf, const float* qw, const float* kw, int norm_all, int unit, float eps,
                       const float* inv_freq, int dims, float amp, const int* pos0, const int* lens, const int* slots, void* kcache,
                       void* vcache, int ring, int B, int S, int H, int GK, int G, int D, int V, cudaStream_t s) {
    if (B * S == 0) return;
    dim3 grid(B * S), block(32, 8);
    const size_t smem = inv_freq ? sizeof(float) * dims : 0, a4 = bf ? 8 : 16;
    auto al = [&](const void* p, size_t n) { return p == nullptr || (uintptr_t)p % n == 0; };
    const int half = inv_freq ? dims / 2 : 0, E = D <= 128 && half % 4 == 0 ? 4 : 8;
    const bool vec = D % E == 0 && D <= 32 * E && half % E == 0 && (!k || V % 4 == 0) && al(q, a4) && al(k, a4) && al(kout, a4) && al(v, a4) &&
                     al(kcache, a4) && al(vcache, a4) && al(qw, 16) && al(kw, 16) && q_sb % 4 == 0 && q_st % 4 == 0 && k_sb % 4 == 0 &&
                     k_st % 4 == 0 && ko_sb % 4 == 0 && ko_st % 4 == 0 && v_sb % 4 == 0 && v_st % 4 == 0;
#define SEQMIX_WQP_ARGS(T)                                                                                                            \
    (T*)q, q_sb, q_st, (T*)k, k_sb, k_st, (T*)kout, ko_sb, ko_st, (const T*)v, v_sb, v_st, qw, kw, norm_all, unit, eps, inv_freq, dims,   \
        amp, pos0, lens, slots, (T*)kcache, (T*)vcache, ring, S, H, GK, G, D, V
#define SEQMIX_WQP(T)                                                                                                                 \
    do {                                                                                                                              \
        if (vec && E == 4) window_qk_prepare_vec_kernel<T, 4><<<grid, block, smem, s>>>(SEQMIX_WQP_ARGS(T));                            \
        else if (vec) window_qk_prepare_vec_kernel<T, 8><<<grid, block, smem, s>>>(SEQMIX_WQP_ARGS(T));                                \
        else window_qk_prepare_kernel<T><<<grid, block, smem, s>>>(SEQMIX_WQP_ARGS(T));                                                \
    } while (0)
    if (bf) SEQMIX_WQP(bf16); else SEQMIX_WQP(float);
#undef SEQMIX_WQP
#undef SEQMIX_WQP_ARGS
}

static int value_cols_per_lane(int V) { return V <= 64 ? 2 : (V <= 128 ? 4 : (V <= 256 ? 8 : (V <= 512 ? 16 : 0))); }

template <typename K>
static bool raise_smem(K kernel, size_t smem) {
    if (smem <= 48 * 1024) return true;
    return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) == cudaSuccess;
}

bool window_prompt_fused(const void* q, long q_sb, long q_st, const void* k, long k_sb, long k_st, const void* v, long v_sb, long v_st, int bf,
                         int D, int V, int maps, const void* out, long out_stride) {
    return bf && window_prompt_mma_fits(q, q_sb, q_st, k, k_sb, k_st, v, v_sb, v_st, D, V, maps, out, out_stride);
}

bool window_attention_prompt(const void* q, long q_sb, long q_st, const void* k, long k_sb, long k_st, const void* v, long v_sb, long v_st,
                             const void* gate, long g_sb, long g_st, int bf, const int* lens, int B, int S, int H, int G, int D, int V,
                             const WindowRule& rule, float* maps_room, void* out, long out_stride, float out_scale, cudaStream_t s) {
    const int vpl = value_cols_per_lane(V);
    if (!vpl) return false;
    if (B * S == 0) return true;
    if (window_prompt_fused(q, q_sb, q_st, k, k_sb, k_st, v, v_sb, v_st, bf, D, V, rule.maps, out, out_stride)) {
        window_prompt_mma(q, q_sb, q_st, k, k_sb, k_st, v, v_sb, v_st, gate, g_sb, g_st, lens, B, S, H, G, D, V, rule, out, out_stride,
                          out_scale, s);
        return true;
    }
    const size_t smem = sizeof(float) * ((size_t)kKeys * (D + 1) + (size_t)kKeys * V + (size_t)kWarps * D * kQW + kWarps * kKeys * kQW);
    float* fout = rule.maps == 2 ? maps_room : nullptr;
    dim3 grid((S + kWarps * kQW - 1) / (kWarps * kQW), H * rule.maps, B), block(128);
#define SEQMIX_WP(T, P)                                                                                                               \
    do {                                                                                                                              \
        if (!raise_smem(window_prompt_kernel<T, P>, smem)) return false;                                                              \
        window_prompt_kernel<T, P><<<grid, block, smem, s>>>((const T*)q, q_sb, q_st, (const T*)k, k_sb, k_st, (const T*)v, v_sb, v_st,   \
                                                             (const T*)gate, g_sb, g_st, lens, S, H, G, D, V, rule, fout, (T*)out,      \
                                                             out_stride, out_scale);                                                  \
    } while (0)
#define SEQMIX_WP_T(P) do { if (bf) SEQMIX_WP(bf16, P); else SEQMIX_WP(float, P); } while (0)
    if (vpl == 2) SEQMIX_WP_T(2); else if (vpl == 4) SEQMIX_WP_T(4); else if (vpl == 8) SEQMIX_WP_T(8); else SEQMIX_WP_T(16);
#undef SEQMIX_WP_T
#undef SEQMIX_WP
    if (fout) {
        const long rows = (long)B * S;
        const unsigned blocks = (unsigned)((rows * H + 7) / 8);
        if (bf) map_combine_kernel<bf16><<<blocks, dim3(32, 8), 0, s>>>(fout, rule.lam, rule.eps, rule.post * out_scale, rows, H, V, (bf16*)out, out_stride);
        else map_combine_kernel<float><<<blocks, dim3(32, 8), 0, s>>>(fout, rule.lam, rule.eps, rule.post * out_scale, rows, H, V, (float*)out, out_stride);
    }
    return true;
}

static bool token_on_tensor_cores(int bf, int D, int V, const WindowRule& rule) {
    return bf && rule.softcap <= 0.f && !rule.score_bias && window_decode_mma_fits(D, V, rule.maps);
}

int window_token_splits(int ring, int bf, int B, int H, int G, int D, int V, const WindowRule& rule) {
    if (token_on_tensor_cores(bf, D, V, rule)) return window_decode_mma_splits(B, H, G, D, V, rule.maps, ring);
    const int quads = G * rule.maps * ((H / G + kWarps - 1) / kWarps);
    const int want = (2 * 148 + B * quads - 1) / (B * quads);       // two blocks per SM's worth of work items
    const int most = (ring + 4 * kKeys - 1) / (4 * kKeys);          // a split has at least 4 chunks
    return max(1, min(min(want, most), 64));
}

bool window_attention_token(const void* q, long q_sb, const void* kcache, const void* vcache, const void* gate, long g_sb, int bf,
                            const int* slots, const int* pos0, const int* lens, int ring, int B, int H, int G, int D, int V,
                            const WindowRule& rule, int splits, float* part_m, float* part_l, float* part_acc, void* out, long out_stride,
                            float out_scale, cudaStream_t s) {
    const int vpl = value_cols_per_lane(V), M = rule.maps;
    if (!vpl) return false;
    if (B == 0) return true;
    if (token_on_tensor_cores(bf, D, V, rule)) {
        window_decode_mma(q, q_sb, kcache, vcache, slots, pos0, lens, ring, B, H, G, D, V, rule, splits, part_m, part_l, part_acc, s);
    } else {
        const size_t smem = sizeof(float) * ((size_t)kKeys * (D + 1) + (size_t)kKeys * V + (size_t)kWarps * D + kWarps * kKeys);
        const int quads = G * M * ((H / G + kWarps - 1) / kWarps), per16 = bf ? 8 : 4;
        const bool vec = D % per16 == 0 && V % per16 == 0 && (uintptr_t)kcache % 16 == 0 && (uintptr_t)vcache % 16 == 0;
        dim3 grid(splits, quads, B), block(128);
#define SEQMIX_WT(T, P, VC)                                                                                                           \
    do {                                                                                                                              \
        if (!raise_smem(window_token_kernel<T, P, VC>, smem)) return false;                                                           \
        window_token_kernel<T, P, VC><<<grid, block, smem, s>>>((const T*)q, q_sb, (const T*)kcache, (const T*)vcache, slots, pos0, lens, \
                                                                ring, H, G, D, V, rule, splits, part_m, part_l, part_acc);             \
    } while (0)
#define SEQMIX_WT_V(T, P) do { if (vec) SEQMIX_WT(T, P, true); else SEQMIX_WT(T, P, false); } while (0)
#define SEQMIX_WT_T(P) do { if (bf) SEQMIX_WT_V(bf16, P); else SEQMIX_WT_V(float, P); } while (0)
        if (vpl == 2) SEQMIX_WT_T(2); else if (vpl == 4) SEQMIX_WT_T(4); else if (vpl == 8) SEQMIX_WT_T(8); else SEQMIX_WT_T(16);
#undef SEQMIX_WT_T
#undef SEQMIX_WT_V
#undef SEQMIX_WT
    }
    dim3 mgrid(H, B);
    const size_t msmem = sizeof(float) * ((size_t)M * splits + 8 * V + M * V + 8);
    if (bf) window_token_merge_kernel<bf16><<<mgrid, 256, msmem, s>>>(part_m, part_l, part_acc, (const bf16*)gate, g_sb, H, V, splits, lens, rule, (bf16*)out, out_stride, out_scale);
    else window_token_merge_kernel<float><<<mgrid, 256, msmem, s>>>(part_m, part_l, part_acc, (const float*)gate, g_sb, H, V, splits, lens, rule, (float*)out, out_stride, out_scale);
    return true;
}

}  // namespace seqmix
