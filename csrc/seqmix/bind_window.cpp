// Python bindings of the grouped-query attention kernels (window, chunk or whole sequence).
#include "bind_common.h"

static const float* opt_f32(const c10::optional<Tensor>& t) { return t ? f32(*t) : nullptr; }

// q [B,S,H,D], k [B,S,GK,D], v [B,S,G,V] (views; last dim contiguous, heads one after another; GK = G or, with two score maps, 2 G); caches
// [slots, ring, GK, D], [slots, ring, G, V].  qw / kw: D numbers (a norm per head) or H*D / GK*D numbers (one norm over all heads);
// unit: a norm without weights after the rotation.  inv_freq: dims/2 rotation frequencies; amp multiplies cos and sin.  kout
// (optional): where the prepared keys go, so that v may alias k.  Without k (then also without v and the caches) only the queries.
void window_qk_prepare(Tensor q, const c10::optional<Tensor>& k, const c10::optional<Tensor>& v, const c10::optional<Tensor>& kout,
                       const c10::optional<Tensor>& qw, const c10::optional<Tensor>& kw, bool norm_all, bool unit, double eps,
                       const c10::optional<Tensor>& inv_freq, int64_t dims, double amp, const Tensor& pos0,
                       const Tensor& lens, const Tensor& slots, const c10::optional<Tensor>& kcache, const c10::optional<Tensor>& vcache) {
    TORCH_CHECK(q.is_cuda() && q.dim() == 4 && q.stride(3) == 1, "bad attention operands");
    const int B = q.size(0), S = q.size(1), H = q.size(2), D = q.size(3);
    TORCH_CHECK(H == 1 || q.stride(2) == D, "heads must be laid out one after another");
    TORCH_CHECK(pos0.numel() == B && lens.numel() == B && slots.numel() == B, "one position, length and slot per row");
    int G = 1, GK = 1, V = 1, ring = 1;
    const Tensor* ko = k ? (kout ? &*kout : &*k) : nullptr;
    if (k) {
        TORCH_CHECK(v && kcache && vcache, "keys come with values and both caches");
        TORCH_CHECK(k->dim() == 4 && v->dim() == 4 && k->stride(3) == 1 && v->stride(3) == 1, "bad attention operands");
        GK = k->size(2); G = v->size(2); V = v->size(3); ring = kcache->size(1);
        TORCH_CHECK(k->size(3) == D && G > 0 && GK % G == 0 && H % GK == 0 && (GK == 1 || k->stride(2) == D) && (G == 1 || v->stride(2) == V),
                    "heads must be laid out one after another");
        TORCH_CHECK(k->size(0) == B && k->size(1) == S && v->size(0) == B && v->size(1) == S, "one key and one value per query token");
        TORCH_CHECK(ko->dim() == 4 && ko->sizes() == k->sizes() && ko->stride(3) == 1 && (GK == 1 || ko->stride(2) == D) &&
                        ko->scalar_type() == k->scalar_type(), "the prepared keys have the keys' shape");
        TORCH_CHECK(q.scalar_type() == k->scalar_type() && q.scalar_type() == v->scalar_type() && kcache->scalar_type() == q.scalar_type() &&
                        vcache->scalar_type() == q.scalar_type(), "dtype mismatch");
        TORCH_CHECK(kcache->is_contiguous() && vcache->is_contiguous() && kcache->dim() == 4 && vcache->dim() == 4 &&
                        kcache->size(1) == vcache->size(1) && kcache->size(2) == GK && kcache->size(3) == D && vcache->size(2) == G &&
                        vcache->size(3) == V, "caches must be [slots, ring, heads, D|V]");
    }
    const bool all = norm_all;
    TORCH_CHECK(!unit || (!qw && !kw && !norm_all), "a norm without weights has no weights");
    TORCH_CHECK(!qw || qw->numel() == (all ? (long)H * D : D), "query norm weights must hold D or H*D numbers");
    TORCH_CHECK(!kw || !k || kw->numel() == (all ? (long)GK * D : D), "key norm weights must hold D or GK*D numbers");
    if (inv_freq) TORCH_CHECK(dims >= 0 && dims % 2 == 0 && dims <= D && inv_freq->numel() == dims / 2, "rotation: dims/2 frequencies, dims <= D");
    seqmix::window_qk_prepare(q.data_ptr(), q.stride(0), q.stride(1), k ? k->data_ptr() : nullptr, k ? k->stride(0) : 0, k ? k->stride(1) : 0,
                              ko ? ko->data_ptr() : nullptr, ko ? ko->stride(0) : 0, ko ? ko->stride(1) : 0,
                              v ? v->data_ptr() : nullptr, v ? v->stride(0) : 0, v ? v->stride(1) : 0, is_bf(q), opt_f32(qw),
                              k ? opt_f32(kw) : nullptr, all, unit, (float)eps, inv_freq ? f32(*inv_freq) : nullptr,
                              inv_freq ? (int)dims : 0, (float)amp, i32(pos0), i32(lens), i32(slots), kcache ? kcache->data_ptr() : nullptr,
                              vcache ? vcache->data_ptr() : nullptr, ring, B, S, H, GK, G, D, V, stream());
    check_launch();
}

// Two maps when lam is given: q then holds two queries per head, k two keys per key/value head.
static seqmix::WindowRule make_rule(int heads, int64_t window, int64_t chunk, double scale, double softcap, const c10::optional<Tensor>& score_bias,
                                    const c10::optional<Tensor>& sink, const c10::optional<Tensor>& lam, double eps, double post, bool gated) {
    TORCH_CHECK(!score_bias || (score_bias->numel() == heads && !sink), "the score bias holds one number per query head and goes without sinks");
    TORCH_CHECK(!sink || sink->numel() == heads, "one sink per query head (and map)");
    TORCH_CHECK(window > 0 && chunk >= 0, "a window of at least one position");
    if (lam) TORCH_CHECK(lam->numel() == 1 && softcap <= 0 && !score_bias && !gated && heads % 2 == 0, "two maps: plain softmax scores, no gate");
    return {(int)window, (int)chunk, (float)scale, (float)softcap, opt_f32(score_bias), opt_f32(sink), lam ? 2 : 1, opt_f32(lam), (float)eps, (float)post};
}

static void check_out(const Tensor& out, long rows, long cols, const Tensor& like) {
    TORCH_CHECK(out.is_cuda() && out.dim() == 2 && out.size(0) == rows && out.size(1) >= cols && out.stride(1) == 1 &&
                    out.scalar_type() == like.scalar_type(), "out must be [rows, >= heads * vdim] of the activations' dtype");
}

void window_attention_prompt(const Tensor& q, const Tensor& k, const Tensor& v, const c10::optional<Tensor>& gate, const Tensor& lens,
                             int64_t window, int64_t chunk, double scale, double softcap, const c10::optional<Tensor>& score_bias,
                             const c10::optional<Tensor>& sink, const c10::optional<Tensor>& lam, double eps, double post, Tensor out,
                             double out_scale) {
    TORCH_CHECK(q.is_cuda() && q.dim() == 4 && k.dim() == 4 && v.dim() == 4 && q.stride(3) == 1 && k.stride(3) == 1 && v.stride(3) == 1,
                "bad attention operands");
    const auto rule = make_rule(q.size(2), window, chunk, scale, softcap, score_bias, sink, lam, eps, post, gate.has_value());
    const int B = q.size(0), S = q.size(1), H = q.size(2) / rule.maps, D = q.size(3), G = v.size(2), V = v.size(3);
    TORCH_CHECK(k.size(3) == D && k.size(2) == G * rule.maps && H % G == 0 && (q.size(2) == 1 || q.stride(2) == D) &&
                    (k.size(2) == 1 || k.stride(2) == D) && (G == 1 || v.stride(2) == V), "heads must be laid out one after another");
    TORCH_CHECK(k.size(0) == B && k.size(1) == S && v.size(0) == B && v.size(1) == S && lens.numel() == B, "one key and one value per query token");
    TORCH_CHECK(q.scalar_type() == k.scalar_type() && q.scalar_type() == v.scalar_type(), "dtype mismatch");
    check_out(out, (long)B * S, (long)H * V, q);
    const void* gp = nullptr;
    long g_sb = 0, g_st = 0;
    if (gate) {
        TORCH_CHECK(gate->dim() == 3 && gate->size(2) == H && gate->stride(2) == 1 && gate->scalar_type() == q.scalar_type(), "gate must be [B,S,H]");
        gp = gate->data_ptr(); g_sb = gate->stride(0); g_st = gate->stride(1);
    }
    Tensor room;
    if (rule.maps == 2 && !seqmix::window_prompt_fused(q.data_ptr(), q.stride(0), q.stride(1), k.data_ptr(), k.stride(0), k.stride(1), v.data_ptr(),
                                                       v.stride(0), v.stride(1), is_bf(q), D, V, 2, out.data_ptr(), out.stride(0)))
        room = at::empty({(long)B * S, H, 2, V}, q.options().dtype(at::kFloat));
    bool ok = seqmix::window_attention_prompt(q.data_ptr(), q.stride(0), q.stride(1), k.data_ptr(), k.stride(0), k.stride(1), v.data_ptr(),
                                              v.stride(0), v.stride(1), gp, g_sb, g_st, is_bf(q), i32(lens), B, S, H, G, D, V, rule,
                                              room.defined() ? room.data_ptr<float>() : nullptr, out.data_ptr(), out.stride(0),
                                              (float)out_scale, stream());
    TORCH_CHECK(ok, "window_attention_prompt: sizes do not fit the kernel (vdim <= 512)");
    check_launch();
}

void window_attention_token(const Tensor& q, const Tensor& kcache, const Tensor& vcache, const c10::optional<Tensor>& gate, const Tensor& slots,
                            const Tensor& pos0, const Tensor& lens, int64_t window, int64_t chunk, double scale, double softcap,
                            const c10::optional<Tensor>& score_bias, const c10::optional<Tensor>& sink, const c10::optional<Tensor>& lam,
                            double eps, double post, Tensor out, double out_scale) {
    TORCH_CHECK(q.is_cuda() && q.dim() == 4 && q.size(1) == 1 && q.stride(3) == 1 && kcache.dim() == 4 && vcache.dim() == 4 &&
                    kcache.is_contiguous() && vcache.is_contiguous(), "bad attention operands");
    const auto rule = make_rule(q.size(2), window, chunk, scale, softcap, score_bias, sink, lam, eps, post, gate.has_value());
    const int B = q.size(0), H = q.size(2) / rule.maps, D = q.size(3), G = vcache.size(2), V = vcache.size(3), ring = kcache.size(1);
    TORCH_CHECK(kcache.size(3) == D && kcache.size(2) == G * rule.maps && vcache.size(1) == ring && H % G == 0 &&
                    (q.size(2) == 1 || q.stride(2) == D), "shape mismatch");
    TORCH_CHECK(pos0.numel() == B && lens.numel() == B && slots.numel() == B, "one position, length and slot per row");
    TORCH_CHECK(q.scalar_type() == kcache.scalar_type() && q.scalar_type() == vcache.scalar_type(), "dtype mismatch");
    check_out(out, B, (long)H * V, q);
    const void* gp = nullptr;
    long g_sb = 0;
    if (gate) {
        TORCH_CHECK(gate->dim() == 3 && gate->size(2) == H && gate->stride(2) == 1 && gate->scalar_type() == q.scalar_type(), "gate must be [B,1,H]");
        gp = gate->data_ptr(); g_sb = gate->stride(0);
    }
    const int splits = seqmix::window_token_splits(ring, is_bf(q), B, H, G, D, V, rule), heads = H * rule.maps;
    const auto f = q.options().dtype(at::kFloat);
    Tensor pm = at::empty({B, heads, splits}, f), pl = at::empty({B, heads, splits}, f), pa = at::empty({B, heads, splits, V}, f);
    bool ok = seqmix::window_attention_token(q.data_ptr(), q.stride(0), kcache.data_ptr(), vcache.data_ptr(), gp, g_sb, is_bf(q), i32(slots),
                                             i32(pos0), i32(lens), ring, B, H, G, D, V, rule, splits,
                                             pm.data_ptr<float>(), pl.data_ptr<float>(), pa.data_ptr<float>(), out.data_ptr(),
                                             out.stride(0), (float)out_scale, stream());
    TORCH_CHECK(ok, "window_attention_token: sizes do not fit the kernel (vdim <= 512)");
    check_launch();
}

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("window_qk_prepare", &window_qk_prepare);
    m.def("window_attention_prompt", &window_attention_prompt);
    m.def("window_attention_token", &window_attention_token);
}
