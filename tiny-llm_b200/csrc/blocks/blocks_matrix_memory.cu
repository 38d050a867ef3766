// The scalar part of a gated matrix memory (mLSTM): from the two gates' projections of every token and head to the numbers its
// recurrence runs on,
//     i_t = cap tanh((zi + bi) / cap)      f_t = log_sigmoid(cap tanh((zf + bf) / cap))      m_t = max(f_t + m_(t-1), i_t)
//     step[t, h] = (exp(f_t + m_(t-1) - m_t), exp(i_t - m_t))        floor[t, h] = exp(-m_t)
// m carried along the sequence in the request's state slot (0 at position 0, whatever the slot held).  The matrix part - decay,
// outer product and read-out - is tlb_decay_scan with these steps.
//
// A token is the map m -> max(f + m, i); two in a row are the map with (f1 + f2, max(f2 + i1, i2)), so a CTA per (sequence, head)
// takes 256 tokens at a time as one scan.  m stays within [-cap, max(0, cap)] from the second token on: sums of f that leave that
// range never win the maximum, and the others are short.
#include "blocks_common.cuh"

namespace tlb {

constexpr int kMmThreads = 256;

// The gates' projections: z [tokens, 2 * heads] (input gates, then forget gates), or, z == NULL, made here from the layer's input
// rows hin [tokens, dim] and w [2 * heads, dim] (launches whose sequences bring a token or two).
template <typename T>
__global__ void __launch_bounds__(kMmThreads)
matrix_memory_gates_kernel(const float *__restrict__ z, long long z_token, const T *__restrict__ hin, long long h_token, const T *__restrict__ w, int dim,
                           const T *__restrict__ bias, float cap, int heads, const int32_t *__restrict__ seq_info, float *__restrict__ state,
                           long long slot_stride, int num_slots, float2 *__restrict__ step, float *__restrict__ floor) {
    __shared__ float s_f[kMmThreads / 32], s_i[kMmThreads / 32], s_m[kMmThreads + 1], s_dot[2][kMmThreads / 32];
    const int s = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int first = seq_info[s * 4 + 0], count = seq_info[s * 4 + 1], start = seq_info[s * 4 + 2], slot = seq_info[s * 4 + 3];
    const bool slot_ok = slot >= 0 && slot < num_slots;
    float *mine = state + (size_t)(slot_ok ? slot : 0) * slot_stride + head;
    const float bi = bias ? to_f(bias[head]) : 0.f, bf = bias ? to_f(bias[heads + head]) : 0.f;
    float carry = start > 0 && slot_ok ? *mine : 0.f;
    const int batch = z ? (int)blockDim.x : 1;  // tokens at a time
    for (int t0 = 0; t0 < count; t0 += batch) {
        const int t = t0 + (int)threadIdx.x;
        const bool live = z ? t < count : threadIdx.x == 0;
        float zi = 0.f, zf = 0.f;
        if (z) {
            if (live) zi = z[(size_t)(first + t) * z_token + head], zf = z[(size_t)(first + t) * z_token + heads + head];
        } else {
            const T *row = hin + (size_t)(first + t0) * h_token, *wi = w + (size_t)head * dim, *wf = w + (size_t)(heads + head) * dim;
            for (int d = threadIdx.x; d < dim; d += blockDim.x) {
                const float x = to_f(row[d]);
                zi = fmaf(x, to_f(wi[d]), zi), zf = fmaf(x, to_f(wf[d]), zf);
            }
            zi = warp_sum(zi), zf = warp_sum(zf);
            if (lane == 0) s_dot[0][warp] = zi, s_dot[1][warp] = zf;
            __syncthreads();
            zi = zf = 0.f;
            for (int i = 0; i < warps; ++i) zi += s_dot[0][i], zf += s_dot[1][i];
        }
        float li = -INFINITY, lf = 0.f;  // a place without a token maps m to itself
        if (live) {
            li = cap * tanhf((zi + bi) / cap);
            lf = log_sigmoid(cap * tanhf((zf + bf) / cap));
        }
        // inclusive scan of (F, I) over the batch's tokens
        float F = lf, I = li;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pf = __shfl_up_sync(0xffffffffu, F, o), pi = __shfl_up_sync(0xffffffffu, I, o);
            if (lane >= o) I = fmaxf(F + pi, I), F = F + pf;
        }
        if (lane == 31) s_f[warp] = F, s_i[warp] = I;
        __syncthreads();
        float before = carry;  // m ahead of this warp's first token
        for (int i = 0; i < warp; ++i) before = fmaxf(s_f[i] + before, s_i[i]);
        const float m = fmaxf(F + before, I);
        s_m[threadIdx.x + 1] = m;
        if (threadIdx.x == 0) s_m[0] = carry;
        __syncthreads();
        if (live) {
            const float prev = s_m[threadIdx.x];
            const size_t at = (size_t)(first + t) * heads + head;
            step[at] = make_float2(expf(lf + prev - m), expf(li - m));
            floor[at] = expf(-m);
        }
        carry = s_m[min(count - t0, batch)];
        __syncthreads();  // s_m, s_f and s_dot are free again
    }
    if (threadIdx.x == 0 && slot_ok) *mine = carry;
}

}  // namespace tlb

using namespace tlb;

extern "C" {

int tlb_matrix_memory_gates(const float *z, long long z_token, const void *hin, long long h_token, const void *w, int dim, const void *bias, float cap, int heads,
                            const int32_t *seq_info, int num_seqs, int max_tokens_per_seq, float *state, long long slot_stride, int num_slots, float *step,
                            float *floor, int dtype, void *stream) {
    if (num_seqs <= 0) return TL_OK;
    if ((z == nullptr) == (hin == nullptr) || (hin && (!w || dim <= 0)) || !(cap > 0.f) || heads <= 0 || !seq_info || !state || num_slots <= 0 || !step || !floor ||
        (uintptr_t)step % 8)
        return tl::fail(TL_EINVAL, "matrix_memory_gates: bad argument");
    int threads = kMmThreads;
    if (z)
        while (threads > 32 && threads / 2 >= max_tokens_per_seq) threads /= 2;
    TLB_DISPATCH(dtype, "matrix_memory_gates",
                 matrix_memory_gates_kernel<T><<<dim3(num_seqs, heads), threads, 0, as_stream(stream)>>>(z, z_token, (const T *)hin, h_token, (const T *)w, dim,
                                                                                                     (const T *)bias, cap, heads, seq_info, state, slot_stride,
                                                                                                     num_slots, (float2 *)step, floor));
    TL_LAUNCH_CHECK("matrix_memory_gates");
    return TL_OK;
}

}  // extern "C"
