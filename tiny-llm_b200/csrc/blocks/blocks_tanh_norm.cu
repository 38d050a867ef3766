// Elementwise bounded norms around the sublayers of a decoder, n(x) = w tanh(alpha x) + b (alpha one number), fused with what
// surrounds them.  They have no statistics over the row, so a step is a sweep over elements that meets no barrier:
//     y  = a sublayer's output (+ its projection's bias), or the weighted sum of a token's experts, or an embedding row
//     x <- x + n_post(y)                (an embedding row starts the stream: x = n_post(y))
//     h  = n_next(x) rounded to T       (what the next sublayer reads)
// Everything up to the rounding of h is fp32.
#include <initializer_list>

#include "blocks_common.cuh"

namespace tlb {

struct TanhNormArgs {  // one norm; w == NULL: none
    const void *w, *b;
    float alpha;
};

struct MixArgs {  // a token's experts: what tlb_moe_combine sums
    const float *pair_out, *gate, *shared_gate;
    const void *shared, *h_in;
    const int32_t *idx;
    int experts, top;
};

// SRC: where y comes from.
constexpr int kFromRows = 0, kFromTable = 1, kFromExperts = 2, kFromStream = 3;

template <typename T>
__device__ __forceinline__ float tn1(float x, const TanhNormArgs &n, int d) {
    return fmaf(tanhf(n.alpha * x), to_f(((const T *)n.w)[d]), to_f(((const T *)n.b)[d]));
}
template <typename T>
__device__ __forceinline__ float4 tn4(float4 x, const TanhNormArgs &n, int d) {
    const float4 w = load4((const T *)n.w + d), b = load4((const T *)n.b + d);
    return make_float4(fmaf(tanhf(n.alpha * x.x), w.x, b.x), fmaf(tanhf(n.alpha * x.y), w.y, b.y), fmaf(tanhf(n.alpha * x.z), w.z, b.z),
                       fmaf(tanhf(n.alpha * x.w), w.w, b.w));
}
__device__ __forceinline__ float4 axpy4(float a, float4 x, float4 y) {
    return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}

// ids: kFromTable: the table's row of every token; kFromStream: the stream's row of every output row (NULL = the same).
template <typename T, int SRC, bool VEC>
__global__ void __launch_bounds__(256)
tanh_step_kernel(float *__restrict__ x, const float *__restrict__ y, const T *__restrict__ y_bias, const int32_t *__restrict__ ids, const T *__restrict__ table,
                 int vocab, MixArgs mix, TanhNormArgs post, TanhNormArgs next, T *__restrict__ h, long long rows, int dim) {
    constexpr int W = VEC ? 4 : 1;
    const int per_row = dim / W;
    const long long at = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (at >= rows * per_row) return;
    const long long r = at / per_row;
    const int d = (int)(at - r * per_row) * W;
    const size_t e = (size_t)r * dim + d;
    if constexpr (VEC) {
        float4 v;
        if constexpr (SRC == kFromStream) {
            v = load4(x + (size_t)(ids ? ids[r] : r) * dim + d);
        } else {
            float4 u;
            if constexpr (SRC == kFromTable) {
                const int id = ids[r];
                u = load4(table + (size_t)(id < 0 || id >= vocab ? 0 : id) * dim + d);
            } else if constexpr (SRC == kFromExperts) {
                u = make_float4(0.f, 0.f, 0.f, 0.f);
                for (int k = 0; k < mix.top; ++k) {
                    const size_t pair = (size_t)r * mix.top + k;
                    const bool same = mix.idx && mix.idx[pair] >= mix.experts;
                    u = axpy4(mix.gate[pair], same ? load4((const T *)mix.h_in + e) : load4(mix.pair_out + pair * dim + d), u);
                }
                if (mix.shared) u = axpy4(mix.shared_gate ? mix.shared_gate[r] : 1.f, load4((const T *)mix.shared + e), u);
            } else {
                u = load4(y + e);
                if (y_bias) u = axpy4(1.f, load4(y_bias + d), u);
            }
            v = tn4<T>(u, post, d);
            if constexpr (SRC != kFromTable) v = axpy4(1.f, load4(x + e), v);
            store4(x + e, v);
        }
        if (h) store4(h + e, tn4<T>(v, next, d));
    } else {
        float v;
        if constexpr (SRC == kFromStream) {
            v = x[(size_t)(ids ? ids[r] : r) * dim + d];
        } else {
            float u;
            if constexpr (SRC == kFromTable) {
                const int id = ids[r];
                u = to_f(table[(size_t)(id < 0 || id >= vocab ? 0 : id) * dim + d]);
            } else if constexpr (SRC == kFromExperts) {
                u = 0.f;
                for (int k = 0; k < mix.top; ++k) {
                    const size_t pair = (size_t)r * mix.top + k;
                    const bool same = mix.idx && mix.idx[pair] >= mix.experts;
                    u = fmaf(mix.gate[pair], same ? to_f(((const T *)mix.h_in)[e]) : mix.pair_out[pair * dim + d], u);
                }
                if (mix.shared) u = fmaf(mix.shared_gate ? mix.shared_gate[r] : 1.f, to_f(((const T *)mix.shared)[e]), u);
            } else {
                u = y[e] + (y_bias ? to_f(y_bias[d]) : 0.f);
            }
            v = tn1<T>(u, post, d);
            if constexpr (SRC != kFromTable) v += x[e];
            x[e] = v;
        }
        if (h) h[e] = from_f<T>(tn1<T>(v, next, d));
    }
}

template <typename T, int SRC>
static void launch_step(float *x, const float *y, const void *y_bias, const int32_t *ids, const void *table, int vocab, const MixArgs &mix,
                        const TanhNormArgs &post, const TanhNormArgs &next, void *h, long long rows, int dim, cudaStream_t st) {
    bool vec = dim % 4 == 0;
    for (const void *p : std::initializer_list<const void *>{x, y, y_bias, table, mix.pair_out, mix.shared, mix.h_in, post.w, post.b, next.w, next.b, h})
        vec = vec && (!p || tl::aligned16(p));
    const long long threads = rows * (vec ? dim / 4 : dim);
    const unsigned blocks = (unsigned)((threads + 255) / 256);
    if (vec) tanh_step_kernel<T, SRC, true><<<blocks, 256, 0, st>>>(x, y, (const T *)y_bias, ids, (const T *)table, vocab, mix, post, next, (T *)h, rows, dim);
    else tanh_step_kernel<T, SRC, false><<<blocks, 256, 0, st>>>(x, y, (const T *)y_bias, ids, (const T *)table, vocab, mix, post, next, (T *)h, rows, dim);
}

static bool norm_ok(const TanhNormArgs &n) { return n.w && n.b; }

}  // namespace tlb

using namespace tlb;

extern "C" {

int tlb_tanh_embed(const int32_t *ids, const void *table, int vocab, float *x, float post_alpha, const void *post_w, const void *post_b, float next_alpha,
                   const void *next_w, const void *next_b, void *h, int rows, int dim, int dtype, void *stream) {
    if (rows <= 0) return TL_OK;
    TanhNormArgs post{post_w, post_b, post_alpha}, next{next_w, next_b, next_alpha};
    if (!ids || !table || !x || vocab <= 0 || dim <= 0 || !norm_ok(post) || (h && !norm_ok(next))) return tl::fail(TL_EINVAL, "tanh_embed: bad argument");
    TLB_DISPATCH(dtype, "tanh_embed", launch_step<T, kFromTable>(x, nullptr, nullptr, ids, table, vocab, MixArgs{}, post, next, h, rows, dim, as_stream(stream)));
    TL_LAUNCH_CHECK("tanh_embed");
    return TL_OK;
}

int tlb_tanh_step(float *x, const float *y, const void *y_bias, float post_alpha, const void *post_w, const void *post_b, float next_alpha,
                  const void *next_w, const void *next_b, void *h, int rows, int dim, int dtype, void *stream) {
    if (rows <= 0) return TL_OK;
    TanhNormArgs post{post_w, post_b, post_alpha}, next{next_w, next_b, next_alpha};
    if (!x || !y || dim <= 0 || !norm_ok(post) || (h && !norm_ok(next))) return tl::fail(TL_EINVAL, "tanh_step: bad argument");
    TLB_DISPATCH(dtype, "tanh_step", launch_step<T, kFromRows>(x, y, y_bias, nullptr, nullptr, 0, MixArgs{}, post, next, h, rows, dim, as_stream(stream)));
    TL_LAUNCH_CHECK("tanh_step");
    return TL_OK;
}

int tlb_tanh_rows(const float *x, const int32_t *row_ids, float alpha, const void *w, const void *b, void *h, int rows, int dim, int dtype, void *stream) {
    if (rows <= 0) return TL_OK;
    TanhNormArgs next{w, b, alpha};
    if (!x || !h || dim <= 0 || !norm_ok(next)) return tl::fail(TL_EINVAL, "tanh_rows: bad argument");
    TLB_DISPATCH(dtype, "tanh_rows",
                 launch_step<T, kFromStream>(const_cast<float *>(x), nullptr, nullptr, row_ids, nullptr, 0, MixArgs{}, TanhNormArgs{}, next, h, rows, dim,
                                             as_stream(stream)));
    TL_LAUNCH_CHECK("tanh_rows");
    return TL_OK;
}

int tlb_moe_combine_tanh(float *x, const float *pair_out, const float *gate, const void *shared, const float *shared_gate, const int32_t *idx, int experts,
                         const void *h_in, int top, float post_alpha, const void *post_w, const void *post_b, float next_alpha, const void *next_w,
                         const void *next_b, void *h, int rows, int dim, int dtype, void *stream) {
    if (rows <= 0) return TL_OK;
    TanhNormArgs post{post_w, post_b, post_alpha}, next{next_w, next_b, next_alpha};
    if (!x || !pair_out || !gate || top <= 0 || dim <= 0 || (idx && !h_in) || (h && h == h_in) || !norm_ok(post) || (h && !norm_ok(next)))
        return tl::fail(TL_EINVAL, "moe_combine_tanh: bad argument");
    MixArgs mix{pair_out, gate, shared_gate, shared, h_in, idx, experts, top};
    TLB_DISPATCH(dtype, "moe_combine_tanh", launch_step<T, kFromExperts>(x, nullptr, nullptr, nullptr, nullptr, 0, mix, post, next, h, rows, dim, as_stream(stream)));
    TL_LAUNCH_CHECK("moe_combine_tanh");
    return TL_OK;
}

}  // extern "C"
