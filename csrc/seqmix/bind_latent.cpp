// Python bindings of the latent sliding-window attention kernels.
#include "bind_common.h"

static const float* sink_of(const c10::optional<Tensor>& sink, int H) {
    if (!sink) return nullptr;
    TORCH_CHECK(sink->numel() == H, "one sink per head");
    return f32(*sink);
}

// queries [B,S,H,Dq]: a view with contiguous heads and ONE stride between consecutive tokens of all rows
static void check_q(const Tensor& q, int64_t need) {
    TORCH_CHECK(q.is_cuda() && q.dim() == 4 && q.stride(3) == 1 && need <= q.size(3) && (q.size(0) == 1 || q.size(1) == 1 || q.stride(0) == q.size(1) * q.stride(1)),
                "q must be [B,S,H,Dq] with evenly spaced tokens");
}
static long q_step(const Tensor& q) { return q.size(1) == 1 ? q.stride(0) : q.stride(1); }      // elements between tokens

// kv [B,S,C+R] raw down-projection → normalised latent + rotated shared key, returned as rows [B,S,C+R] (if want_rows) and appended to
// cache [slots, ring, C+R] (if given).  q (optional) [B,S,H,Dq] with one stride between tokens: coordinates [off, off+dims) of every
// head are rotated in place as well.  amp multiplies both cos and sin.
Tensor latent_kv_store(const Tensor& kv, const Tensor& nw, double eps, const Tensor& inv_freq, int64_t dims, const Tensor& pos0,
                       const Tensor& lens, const Tensor& slots, const c10::optional<Tensor>& cache, bool want_rows,
                       const c10::optional<Tensor>& q, int64_t off, double amp) {
    TORCH_CHECK(kv.is_cuda() && kv.dim() == 3 && kv.stride(2) == 1, "kv must be [B,S,C+R]");
    const int B = kv.size(0), S = kv.size(1), C = nw.numel(), R = kv.size(2) - C;
    TORCH_CHECK(R >= 0 && dims % 2 == 0 && dims <= R && inv_freq.numel() == dims / 2, "bad rotary sizes");
    Tensor rows = want_rows ? at::zeros({B, S, C + R}, kv.options()) : Tensor();
    void* cp = nullptr;
    int ring = 1;
    if (cache) {
        TORCH_CHECK(cache->is_contiguous() && cache->scalar_type() == kv.scalar_type() && cache->size(2) == C + R, "bad cache");
        cp = cache->data_ptr();
        ring = cache->size(1);
    }
    char* qp = nullptr;
    long q_sn = 0, q_sh = 0;
    int H = 0;
    if (q) {
        check_q(*q, off + dims);
        TORCH_CHECK(q->scalar_type() == kv.scalar_type() && q->size(0) == B && q->size(1) == S, "queries and keys differ in dtype or rows");
        qp = (char*)q->data_ptr() + off * q->element_size();
        q_sn = q_step(*q);
        q_sh = q->stride(2);
        H = q->size(2);
    }
    seqmix::latent_kv_store(kv.data_ptr(), is_bf(kv), kv.stride(0), kv.stride(1), B, S, C, R, (int)dims, f32(nw), (float)eps, f32(inv_freq),
                            i32(pos0), i32(lens), i32(slots), cp, ring, want_rows ? rows.data_ptr() : nullptr, (float)amp,
                            qp, q_sn, q_sh, H, stream());
    check_launch();
    return rows;
}

// q [B,S,H,Dq]: rotate coordinates [off, off+dims) of every head in place
void rope_q_(Tensor q, int64_t off, int64_t dims, const Tensor& inv_freq, const Tensor& pos0, double amp) {
    check_q(q, off + dims);
    TORCH_CHECK(inv_freq.numel() == dims / 2, "bad rotary sizes");
    const int B = q.size(0), S = q.size(1), H = q.size(2);
    char* p = (char*)q.data_ptr() + off * q.element_size();
    seqmix::rope_q(p, is_bf(q), q_step(q), q.stride(2), B * S, S, H, (int)dims, f32(inv_freq), i32(pos0), (float)amp, stream());
    check_launch();
}

// qa [H, N, C] (absorbed queries, N = B*S), q [B,S,H,Dq] with the rotated part at `off`; keys [blocks, ring, C+R];
// key_index [B] (block of each sequence) or none (block b) → out [H, N, C]
Tensor latent_window_attention(const Tensor& qa, const Tensor& q, int64_t off, const Tensor& keys, const c10::optional<Tensor>& key_index,
                               const Tensor& pos0, const Tensor& lens, int64_t window, double scale, const c10::optional<Tensor>& sink) {
    TORCH_CHECK(qa.is_cuda() && qa.dim() == 3 && qa.is_contiguous() && keys.dim() == 3 && keys.is_contiguous(),
                "bad attention operands");
    check_q(q, off);
    const int H = qa.size(0), N = qa.size(1), C = qa.size(2), B = q.size(0), S = q.size(1), Dq = q.size(3), R = keys.size(2) - C;
    const float* sk = sink_of(sink, H);
    const long q_sn = q_step(q), q_sh = q.stride(2);
    TORCH_CHECK(N == B * S && q.size(2) == H && R >= 0 && off + R <= Dq && C + R <= 640, "bad attention sizes (C + R <= 640)");
    TORCH_CHECK(qa.scalar_type() == q.scalar_type() && q.scalar_type() == keys.scalar_type(), "dtype mismatch");
    Tensor out = at::empty({H, N, C}, qa.options());
    const char* qr = (const char*)q.data_ptr() + off * q.element_size();
    if (S == 1 && seqmix::latent_ring_decode_fits(C, R)) {      // single tokens: split over the ring, partial softmaxes merged
        const int ring = keys.size(1), rows = (int)std::min<int64_t>(ring, window);
        const bool mma = is_bf(qa) && seqmix::latent_decode_mma_fits(C, R);
        const long ns = mma ? seqmix::latent_decode_mma_splits(B, H, rows) : seqmix::latent_ring_decode_splits(ring);
        const auto f = qa.options().dtype(at::kFloat);
        Tensor pm = at::empty({B, ns, H}, f), pl = at::empty({B, ns, H}, f), pa = at::empty({B, ns, H, C}, f);
        seqmix::latent_ring_decode(qa.data_ptr(), is_bf(qa), C, (long)N * C, qr, q_sn, q_sh, keys.data_ptr(), keys.stride(0), ring,
                                   key_index ? i32(*key_index) : nullptr, i32(pos0), i32(lens), B, H, C, R, (int)window, (float)scale, sk,
                                   mma, (int)ns, pm.data_ptr<float>(), pl.data_ptr<float>(), pa.data_ptr<float>(), out.data_ptr(), C,
                                   (long)N * C, stream());
        check_launch();
        return out;
    }
    seqmix::latent_window_attention(qa.data_ptr(), is_bf(qa), C, (long)N * C, qr, q_sn, q_sh, keys.data_ptr(), keys.stride(0),
                                    (int)keys.size(1), key_index ? i32(*key_index) : nullptr, i32(pos0), i32(lens), B, S, H, C, R,
                                    (int)window, (float)scale, sk, out.data_ptr(), C, (long)N * C, stream());
    check_launch();
    return out;
}

bool latent_prompt_attention_fits(int64_t D, int64_t R, int64_t CR, int64_t VD) {
    return seqmix::latent_prompt_attention_fits((int)D, (int)R, (int)CR, (int)VD);
}

// q [B,S,H,D+R] (evenly spaced tokens), kx [B,S,H*D], rows [B,S,CR], v [B,S,H*VD] (bfloat16), gate [B*S, H*VD] (bfloat16, row stride
// free) or none → [B*S, H*VD]
Tensor latent_prompt_attention(const Tensor& q, const Tensor& kx, const Tensor& rows, const Tensor& v, const Tensor& lens, int64_t D,
                               int64_t R, int64_t VD, int64_t window, double scale, const c10::optional<Tensor>& sink,
                               const c10::optional<Tensor>& gate) {
    check_q(q, D + R);
    TORCH_CHECK(q.stride(2) == D + R && q_step(q) % 8 == 0 && (uintptr_t)q.data_ptr() % 16 == 0 && kx.is_contiguous() && rows.is_contiguous() && v.is_contiguous() &&
                    rows.dim() == 3, "bad prompt attention operands");
    TORCH_CHECK(is_bf(q) && is_bf(kx) && is_bf(rows) && is_bf(v), "the fused prompt attention takes bfloat16");
    const int B = q.size(0), S = q.size(1), H = q.size(2), CR = rows.size(2);
    TORCH_CHECK(q.size(3) == D + R && kx.numel() == (long)B * S * H * D && v.numel() == (long)B * S * H * VD && rows.size(0) == B &&
                    rows.size(1) == S && CR >= R, "shape mismatch");
    if (gate)
        TORCH_CHECK(is_bf(*gate) && gate->dim() == 2 && gate->size(0) == (long)B * S && gate->size(1) == H * VD && gate->stride(1) == 1 &&
                        gate->stride(0) % 2 == 0 && (uintptr_t)gate->data_ptr() % 4 == 0, "gate must be bfloat16 [B*S, H*VD]");
    Tensor out = at::empty({(long)B * S, (long)H * VD}, q.options());
    bool ok = seqmix::latent_prompt_attention(q.data_ptr(), q_step(q), kx.data_ptr(), rows.data_ptr(), v.data_ptr(), i32(lens), B, S, H,
                                              (int)D, (int)R, CR, (int)VD, (int)window, (float)scale, sink_of(sink, H),
                                              gate ? gate->data_ptr() : nullptr, gate ? gate->stride(0) : 0, out.data_ptr(), stream());
    TORCH_CHECK(ok, "latent_prompt_attention: sizes do not fit the kernel");
    check_launch();
    return out;
}

// scores float [..., span] (contiguous) → softmax over the visible keys, in `out_bf16`'s dtype.  Band mode: rows (b, block, t, head);
// ring mode: rows (b, head) of single tokens at positions pos0.  sink float [n]: row (b, h)'s sink is number (b * H + h) mod n.
Tensor window_softmax(const Tensor& scores, double scale, bool ring_mode, int64_t H, int64_t Qb, int64_t nblk, int64_t w_eff, int64_t window,
                      const Tensor& pos0, const Tensor& lens, bool out_bf16, const c10::optional<Tensor>& sink) {
    TORCH_CHECK(scores.is_cuda() && scores.is_contiguous() && scores.scalar_type() == at::kFloat, "scores must be contiguous float");
    const int span = scores.size(-1);
    const long rows = scores.numel() / span;
    Tensor out = at::empty(scores.sizes(), scores.options().dtype(out_bf16 ? at::kBFloat16 : at::kFloat));
    seqmix::window_softmax(scores.data_ptr<float>(), rows, span, (float)scale, ring_mode, (int)H, (int)Qb, (int)nblk, (int)w_eff, (int)window,
                           i32(pos0), i32(lens), sink ? f32(*sink) : nullptr, sink ? (int)sink->numel() : 1, out.data_ptr(), out_bf16, stream());
    check_launch();
    return out;
}

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("latent_kv_store", &latent_kv_store);
    m.def("rope_q_", &rope_q_);
    m.def("latent_window_attention", &latent_window_attention);
    m.def("window_softmax", &window_softmax);
    m.def("latent_prompt_attention", &latent_prompt_attention);
    m.def("latent_prompt_attention_fits", &latent_prompt_attention_fits);
}
