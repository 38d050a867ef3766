// Grouped-query attention over the bf16 paged cache with the softmax kept in registers: the serving path of large and small
// steps (same arguments, masks and weights as blocks_paged_attention.cu; mma.sync m16n8k16, fp32 accumulation and softmax).
//
// A query row is one (token, query head); the rows of a CTA belong to a run of consecutive tokens of one sequence x up to
// ROWS query heads of ONE key/value head, and every 64-key tile of that head goes through shared memory once for all of them
// (cp.async, 16 bytes a piece, the next tile loads while this one is computed; one barrier per tile).  Four warps, in one of
// two forms:
//   wide rows (64 rows)   a warp owns 16 rows and computes all 64 keys of a tile for them: prompt portions;
//   split keys (16 rows)  all warps share the 16 rows, each computes 16 keys of every tile with a running maximum and sum of
//                         its own, and the four are combined at the end: single tokens, whose few rows would leave three
//                         warps of the other form without work.
// Scores, probabilities and the output accumulators stay in the warp's registers (the accumulator layout of S is the operand
// layout of P V).  Tiles are 64-aligned in absolute positions and taken in ascending order; those that no row of a warp may
// see are passed over, those that every row sees whole skip the mask.  A row's arithmetic depends on its own position alone,
// so what shares the CTA or the batch leaves no trace, nor does where a prompt was cut.
// When a launch alone would leave SMs idle, a cluster of up to eight CTAs takes the key tiles of one row tile by contiguous
// runs and combines its partial sums through distributed shared memory: no workspace, no second launch.
#include <cooperative_groups.h>

#include "blocks_common.cuh"

namespace tlb {

namespace cg = cooperative_groups;

constexpr int kFWarps = 4;
constexpr int kFKeys = 64;   // keys per tile
constexpr int kFSplits = 8;  // most CTAs of a cluster
constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kOnes = 0x3F803F80u;  // two bf16 ones

struct FlashArgs {
    const bf16 *q;
    long long q_token, q_head;
    const bf16 *slab;
    int num_pages, page_size, dk, dv, heads, kv_heads, hp /* query heads per CTA */;
    const int32_t *block_table;
    int max_pages;
    const int32_t *tiles, *tok_pos;
    int mask, mask_size, keep_first;
    float scale, softcap;
    int sink;
    const bf16 *gate;   // logits of a sigmoid: one per head, or (gate_wide) one per entry of every head
    int gate_wide;
    long long g_token;
    bf16 *out;
    long long o_token, o_head;
    const float *head_bias;
    int weights, k_stride, q_wide /* 16-byte query loads */, o_pairs /* 4-byte output stores */;
};

__device__ __forceinline__ uint32_t f_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void f_ldm_x4(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void f_ldm_x4_trans(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void f_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void f_cp16(uint32_t d, const void *src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ float f_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float f_tanh(float x) {
    float y;
    asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// 2^(a - b) where b is a running maximum: 0 for a = -infinity, also when both are
__device__ __forceinline__ float f_weight(float a, float b) { return a == -INFINITY ? 0.f : f_ex2(a - b); }

// NV: units of 16 value columns; SPLIT: the form (see above); KT: units of 16 query / key columns when known (the queries then
// stay in registers), 0 = any number.
template <int NV, bool SPLIT, int KT>
__global__ void __launch_bounds__(kFWarps * 32, NV <= 8 ? 2 : 1)
paged_attention_flash_kernel(const FlashArgs A) {
    constexpr int ROWS = SPLIT ? 16 : 16 * kFWarps;
    constexpr int NT = SPLIT ? 2 : kFKeys / 8;  // 8-key score tiles per warp
    constexpr int COLS = NV * 16;
    constexpr int VS = COLS + 8;                       // value row stride; (stride / 8) odd: conflict-free ldmatrix rows
    const int KS = KT ? KT * 16 + 8 : A.k_stride;      // query / key row stride
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16 *sq = reinterpret_cast<bf16 *>(smem_raw);     // [ROWS][KS]; with KT only until the queries are in registers
    bf16 *skv = KT ? sq : sq + ROWS * KS;              // [2] x ([64][KS] keys | [64][VS] values)
    const int buf_elems = kFKeys * (KS + VS);

    const int group = A.heads / A.kv_heads, hp = A.hp, parts = (group + hp - 1) / hp;
    const int g = blockIdx.y / parts, part = blockIdx.y % parts;
    const int head0 = g * group + part * hp, nheads = min(hp, group - part * hp);
    const int first = A.tiles[blockIdx.x * 3 + 0], count = A.tiles[blockIdx.x * 3 + 1], seq = A.tiles[blockIdx.x * 3 + 2];
    const int pos0 = A.tok_pos[first];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, t4 = lane & 3;
    const int k_pieces = A.dk / 8, per_row = k_pieces + A.dv / 8;  // 16-byte pieces of a key row, of a cache row's share of this head

    // padding must read as zero in every product: query rows without a token, columns of Q and K past dk
    for (int i = threadIdx.x; i < ((KT ? 0 : ROWS * KS) + 2 * buf_elems) / 8; i += blockDim.x) reinterpret_cast<uint4 *>(sq)[i] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    if (A.q_wide) {
        for (int i = threadIdx.x; i < ROWS * k_pieces; i += blockDim.x) {
            const int r = i / k_pieces, piece = i - r * k_pieces, tq = r / hp, hh = r - tq * hp;
            if (tq < count && hh < nheads)
                *reinterpret_cast<uint4 *>(sq + r * KS + piece * 8) =
                    *reinterpret_cast<const uint4 *>(A.q + (size_t)(first + tq) * A.q_token + (size_t)(head0 + hh) * A.q_head + piece * 8);
        }
    } else {
        for (int i = threadIdx.x; i < ROWS * A.dk; i += blockDim.x) {
            const int r = i / A.dk, d = i - r * A.dk, tq = r / hp, hh = r - tq * hp;
            if (tq < count && hh < nheads) sq[r * KS + d] = A.q[(size_t)(first + tq) * A.q_token + (size_t)(head0 + hh) * A.q_head + d];
        }
    }

    // the key tiles of this row tile: kept first positions that the window does not reach, then from `lo` to the newest key
    const int hi = pos0 + count - 1;
    int lo = 0;
    if (A.mask == 1) lo = max(0, pos0 - A.mask_size + 1);
    if (A.mask == 2) lo = pos0 / A.mask_size * A.mask_size;
    lo = lo / kFKeys * kFKeys;
    const int kept_tiles = A.mask == 1 ? min(lo, (A.keep_first + kFKeys - 1) / kFKeys * kFKeys) / kFKeys : 0;
    const int n_tiles = kept_tiles + (hi - lo) / kFKeys + 1;
    auto tile_key = [&](int tile) { return tile < kept_tiles ? tile * kFKeys : lo + (tile - kept_tiles) * kFKeys; };
    const int per_split = (n_tiles + (int)gridDim.z - 1) / (int)gridDim.z;
    const int tile_begin = min(n_tiles, (int)blockIdx.z * per_split), tile_end = min(n_tiles, tile_begin + per_split);

    const int32_t *table = A.block_table + (size_t)seq * A.max_pages;
    const size_t row_width = (size_t)A.kv_heads * (A.dk + A.dv), k_off = (size_t)g * A.dk, v_off = (size_t)A.kv_heads * A.dk + (size_t)g * A.dv;
    // a warp copies whole rows: `span` lanes a row (a power of two), 32 / span rows at a time, a lane the same 16-byte pieces of
    // every row it takes
    int span = 32;
    while (span / 2 >= per_row) span /= 2;
    const int my_row = warp * (32 / span) + lane / span, my_piece = lane % span, rows_at_once = kFWarps * (32 / span);
    auto stage = [&](int tile, int buf) {
        const uint32_t sk = f_addr(skv + buf * buf_elems), sv = sk + kFKeys * KS * 2;
        const int k0 = tile_key(tile);
#pragma unroll
        for (int h = 0; h < 2; ++h) {  // a page holds a multiple of 32 keys: each half of a tile lies in one page
            const int key = k0 + 32 * h;
            const int page = key <= hi ? table[key / A.page_size] : -1;
            const bool ok = page >= 0 && page < A.num_pages;  // a bad table entry reads as zeros
            const int valid = ok ? min(32, hi - key + 1) : 0;
            for (int piece = my_piece; piece < per_row; piece += 32) {
                const bool is_v = piece >= k_pieces;
                const int col = (is_v ? piece - k_pieces : piece) * 8, stride = is_v ? VS : KS;
                const bf16 *src = A.slab + ((size_t)(ok ? page : 0) * A.page_size + key % A.page_size + my_row) * row_width + (is_v ? v_off : k_off) + col;
                uint32_t dst = (is_v ? sv : sk) + ((32 * h + my_row) * stride + col) * 2;
                const size_t src_step = (size_t)rows_at_once * row_width;
                const uint32_t dst_step = rows_at_once * stride * 2;
                for (int j = my_row; j < 32; j += rows_at_once, src += src_step, dst += dst_step) {
                    if (j < valid) f_cp16(dst, src);
                    else asm volatile("st.shared.v4.b32 [%0], {%1, %1, %1, %1};" ::"r"(dst), "r"(0) : "memory");
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    // scores enter the exponential as 2^(s * mult - maximum * mult): s as the product leaves it where the maximum may be taken
    // over that (a softmax without a cap, a positive scale), else s already scaled and capped and mult = 1
    const float scale2 = A.scale * kLog2e, cap_in = A.softcap > 0.f ? A.scale / A.softcap : 0.f, cap_out = A.softcap * kLog2e;
    const bool raw = A.softcap <= 0.f && A.scale > 0.f && A.weights == 0;
    const float mult = raw ? scale2 : 1.f;
    // the two rows of this thread's quad: what they may see ([see_lo, see_hi] and keys below keep_first) and their running
    // maximum; the running sums are one more accumulator tile, P times a matrix of ones
    const int row0 = SPLIT ? 0 : warp * 16;
    const bool opens = blockIdx.z == 0 && (!SPLIT || warp == 0);  // who counts the sink (or the sigmoid form's constant sum), once
    int see_lo[2], see_hi[2];
    float m[2], hb[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int r = row0 + gq + 8 * h, tq = r / hp, hh = r - tq * hp;
        const bool live = tq < count && hh < nheads;
        const int p = pos0 + tq;
        see_hi[h] = live ? p : -1;
        see_lo[h] = !live ? 0x7fffffff : A.mask == 1 ? max(0, p - A.mask_size + 1) : A.mask == 2 ? p / A.mask_size * A.mask_size : 0;
        hb[h] = A.head_bias && live ? A.head_bias[head0 + hh] * kLog2e : 0.f;
        m[h] = A.weights == 1 ? 0.f : A.sink && opens ? hb[h] / mult : -INFINITY;
    }
    const int first_kept = A.mask == 1 ? A.keep_first : 0;
    // over the warp's live rows: tokens ascend with the row, so the first row's range starts first and the last one's ends last
    int warp_lo, warp_hi, all_lo, all_hi;  // any row sees from / to, every row sees from / to
    {
        int a = min(see_lo[0], see_lo[1]), b = max(see_hi[0], see_hi[1]);
        int c = max(see_hi[0] < 0 ? -1 : see_lo[0], see_hi[1] < 0 ? -1 : see_lo[1]);
        int d = min(see_hi[0] < 0 ? 0x7fffffff : see_hi[0], see_hi[1] < 0 ? 0x7fffffff : see_hi[1]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            a = min(a, __shfl_xor_sync(0xffffffffu, a, o)), b = max(b, __shfl_xor_sync(0xffffffffu, b, o));
            c = max(c, __shfl_xor_sync(0xffffffffu, c, o)), d = min(d, __shfl_xor_sync(0xffffffffu, d, o));
        }
        warp_lo = a, warp_hi = b, all_lo = c, all_hi = d;
    }

    float acc[2 * NV][4], sums[4];
    sums[0] = sums[1] = sums[2] = sums[3] = opens && (A.sink || A.weights == 1) ? 1.f : 0.f;
#pragma unroll
    for (int i = 0; i < 2 * NV; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;

    const int ksteps = KT ? KT : (A.dk + 15) / 16;
    __syncthreads();  // the zero fill and the queries are in place before the first copies land
    const uint32_t q_at = f_addr(sq + (row0 + (lane & 15)) * KS + (lane >> 4) * 8);
    uint32_t qf[KT ? KT : 1][4];
    if constexpr (KT > 0) {
#pragma unroll
        for (int ks = 0; ks < KT; ++ks) f_ldm_x4(qf[ks], q_at + ks * 32);
        __syncthreads();
        for (int i = threadIdx.x; i < ROWS * KS / 8; i += blockDim.x) reinterpret_cast<uint4 *>(sq)[i] = make_uint4(0, 0, 0, 0);  // key padding again
        __syncthreads();
    }
    const uint32_t k_at = ((SPLIT ? warp * 16 : 0) + (lane & 7) + (lane >> 4) * 8) * KS * 2 + ((lane >> 3) & 1) * 16;
    const uint32_t v_at = kFKeys * KS * 2 + ((SPLIT ? warp * 16 : 0) + (lane & 7) + ((lane >> 3) & 1) * 8) * VS * 2 + (lane >> 4) * 16;
    if (tile_begin < tile_end) stage(tile_begin, 0);
    for (int tile = tile_begin; tile < tile_end; ++tile) {
        const int buf = (tile - tile_begin) & 1;
        const uint32_t base_at = f_addr(skv + buf * buf_elems);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // this tile has landed, and every warp is done with the previous one: its buffer may be refilled
        if (tile + 1 < tile_end) stage(tile + 1, buf ^ 1);
        const int key0 = tile_key(tile) + (SPLIT ? warp * 16 : 0), key_end = key0 + NT * 8 - 1;
        if (key0 > warp_hi || (key_end < warp_lo && key0 >= first_kept)) continue;  // no row of the warp sees any of its keys

        float s[NT][4];
#pragma unroll
        for (int i = 0; i < NT; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
        {
            const uint32_t kb = base_at + k_at;
            auto step = [&](int ks, const uint32_t (&a)[4]) {
#pragma unroll
                for (int n = 0; n < NT / 2; ++n) {
                    uint32_t b[4];
                    f_ldm_x4(b, kb + n * 32 * KS + ks * 32);
                    f_mma(s[2 * n], a, b[0], b[1]);
                    f_mma(s[2 * n + 1], a, b[2], b[3]);
                }
            };
            if constexpr (KT > 0) {
#pragma unroll
                for (int ks = 0; ks < KT; ++ks) step(ks, qf[ks]);
            } else {
#pragma unroll 2
                for (int ks = 0; ks < ksteps; ++ks) {
                    uint32_t a[4];
                    f_ldm_x4(a, q_at + ks * 32);
                    step(ks, a);
                }
            }
        }
        if (A.softcap > 0.f) {
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[i][e] = cap_out * f_tanh(s[i][e] * cap_in);
        } else if (!raw) {
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[i][e] *= scale2;
        }
        if (key_end > all_hi || (key0 < all_lo && key_end >= first_kept)) {  // some row does not see all of it
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = key0 + i * 8 + 2 * t4 + (e & 1), h = e >> 1;
                    if (key > see_hi[h] || (key < see_lo[h] && key >= first_kept)) s[i][e] = -INFINITY;
                }
        }
        if (A.weights == 1) {  // every visible key by itself: no maximum, no sum, nothing to rescale
#pragma unroll
            for (int i = 0; i < NT; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[i][e] = s[i][e] == -INFINITY ? 0.f : 1.0f / (1.0f + f_ex2(-(s[i][e] + hb[e >> 1])));
        } else {
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                float mx = m[h];
#pragma unroll
                for (int i = 0; i < NT; ++i) mx = fmaxf(mx, fmaxf(s[i][2 * h], s[i][2 * h + 1]));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float base = mx == -INFINITY ? 0.f : __fmul_rn(mx, mult);
                const float alpha = m[h] == -INFINITY ? 0.f : f_ex2(__fmul_rn(m[h], mult) - base);  // exactly 1 where the maximum stays
                m[h] = mx;
#pragma unroll
                for (int i = 0; i < NT; ++i) s[i][2 * h] = f_ex2(fmaf(s[i][2 * h], mult, -base)), s[i][2 * h + 1] = f_ex2(fmaf(s[i][2 * h + 1], mult, -base));
                if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll
                    for (int i = 0; i < 2 * NV; ++i) acc[i][2 * h] *= alpha, acc[i][2 * h + 1] *= alpha;
                    sums[2 * h] *= alpha, sums[2 * h + 1] *= alpha;
                }
            }
        }
#pragma unroll
        for (int kk = 0; kk < NT / 2; ++kk) {
            const uint32_t a[4] = {tl::pack2<bf16>(s[2 * kk][0], s[2 * kk][1]), tl::pack2<bf16>(s[2 * kk][2], s[2 * kk][3]),
                                   tl::pack2<bf16>(s[2 * kk + 1][0], s[2 * kk + 1][1]), tl::pack2<bf16>(s[2 * kk + 1][2], s[2 * kk + 1][3])};
            if (A.weights == 0) f_mma(sums, a, kOnes, kOnes);  // numerator and denominator see the same rounded weights
            const uint32_t vb = base_at + v_at + kk * 32 * VS;
#pragma unroll
            for (int n = 0; n < NV; ++n) {
                uint32_t b[4];
                f_ldm_x4_trans(b, vb + n * 32);
                f_mma(acc[2 * n], a, b[0], b[1]);
                f_mma(acc[2 * n + 1], a, b[2], b[3]);
            }
        }
    }
    auto factor = [&](int r, float sum) {  // what a row's sums are multiplied by on their way out
        const int tq = r / hp, hh = r - tq * hp;
        float inv = 1.0f / sum;
        if (A.gate && !A.gate_wide) inv *= sigmoid(__bfloat162float(A.gate[(size_t)(first + tq) * A.g_token + head0 + hh]));
        return inv;
    };
    auto put2 = [&](int r, int col, float x, float y) {
        const int tq = r / hp, hh = r - tq * hp;
        if (A.gate_wide) {
            const bf16 *gw = A.gate + (size_t)(first + tq) * A.g_token + (size_t)(head0 + hh) * A.dv + col;
            x *= sigmoid(__bfloat162float(gw[0])), y *= sigmoid(__bfloat162float(gw[1]));
        }
        bf16 *o = A.out + (size_t)(first + tq) * A.o_token + (size_t)(head0 + hh) * A.o_head + col;
        if (A.o_pairs) *reinterpret_cast<uint32_t *>(o) = tl::pack2<bf16>(x, y);
        else o[0] = __float2bfloat16_rn(x), o[1] = __float2bfloat16_rn(y);
    };
    auto row_live = [&](int r) { return r / hp < count && r % hp < nheads; };

    if (!SPLIT && gridDim.z == 1) {  // nothing to combine
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int r = row0 + gq + 8 * h;
            if (!row_live(r)) continue;
            const float inv = factor(r, sums[2 * h]);
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i) {
                const int col = i * 8 + 2 * t4;
                if (col < A.dv) put2(r, col, acc[i][2 * h] * inv, acc[i][2 * h + 1] * inv);
            }
        }
        return;
    }

    // partial sums to shared memory (over the tile buffers, which nobody reads any more)
    constexpr int P = SPLIT ? kFWarps : 1;               // partial results per row in this CTA
    float *so = reinterpret_cast<float *>(skv);          // [P][ROWS][COLS]
    float *sm = so + P * ROWS * COLS, *sl = sm + P * ROWS;  // [P][ROWS]
    __syncthreads();
    {
        const int p = SPLIT ? warp : 0;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int r = row0 + gq + 8 * h;
#pragma unroll
            for (int i = 0; i < 2 * NV; ++i)
                *reinterpret_cast<float2 *>(so + ((size_t)p * ROWS + r) * COLS + i * 8 + 2 * t4) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
            if (t4 == 0) sm[p * ROWS + r] = m[h] == -INFINITY ? m[h] : m[h] * mult, sl[p * ROWS + r] = sums[2 * h];
        }
    }
    cg::cluster_group cluster = cg::this_cluster();
    if (gridDim.z > 1) cluster.sync();  // every CTA of the cluster has its partial sums in place
    else __syncthreads();
    // a thread takes pairs of columns; the CTAs of a cluster share the rows
    const int splits = (int)gridDim.z;
    for (int e = threadIdx.x + (int)blockIdx.z * blockDim.x; e < ROWS * COLS / 2; e += blockDim.x * splits) {
        const int r = e / (COLS / 2), col = (e - r * (COLS / 2)) * 2;
        if (col >= A.dv || !row_live(r)) continue;
        float top = -INFINITY;
        for (int z = 0; z < splits; ++z) {
            const float *zm = splits > 1 ? cluster.map_shared_rank(sm, z) : sm;
            for (int p = 0; p < P; ++p) top = fmaxf(top, zm[p * ROWS + r]);
        }
        float x = 0.f, y = 0.f, sum = 0.f;
        for (int z = 0; z < splits; ++z) {
            const float *zo = splits > 1 ? cluster.map_shared_rank(so, z) : so, *zm = zo + P * ROWS * COLS, *zl = zm + P * ROWS;
            for (int p = 0; p < P; ++p) {
                const float w = f_weight(zm[p * ROWS + r], top);
                const float2 o = *reinterpret_cast<const float2 *>(zo + ((size_t)p * ROWS + r) * COLS + col);
                x = fmaf(w, o.x, x), y = fmaf(w, o.y, y), sum = fmaf(w, zl[p * ROWS + r], sum);
            }
        }
        const float inv = factor(r, sum);
        put2(r, col, x * inv, y * inv);
    }
    if (gridDim.z > 1) cluster.sync();  // nobody leaves while others read its shared memory
}

static int f_units(int dv) {
    int u = ceil_div(dv, 16);
    return u <= 2 ? 2 : u <= 4 ? 4 : u <= 6 ? 6 : u <= 8 ? 8 : u <= 12 ? 12 : 16;
}

template <int NV, bool SPLIT, int KT>
static int f_launch(const FlashArgs &args, int num_tiles, int splits, cudaStream_t st) {
    auto kernel = paged_attention_flash_kernel<NV, SPLIT, KT>;
    const int rows = SPLIT ? 16 : 16 * kFWarps;
    const size_t smem = (size_t)((KT ? 0 : rows * args.k_stride) + 2 * kFKeys * (args.k_stride + NV * 16 + 8)) * sizeof(bf16);
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return tl::fail(TL_ECUDA, "paged_attention_flash: %s", cudaGetErrorString(e));
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(num_tiles, args.kv_heads * ceil_div(args.heads / args.kv_heads, args.hp), splits);
    cfg.blockDim = dim3(kFWarps * 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1, attr[0].val.clusterDim.y = 1, attr[0].val.clusterDim.z = splits;
    cfg.attrs = attr;
    cfg.numAttrs = splits > 1 ? 1 : 0;
    cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, args);
    if (e != cudaSuccess) {
        cudaGetLastError();
        return tl::fail(TL_ECUDA, "paged_attention_flash: kernel launch failed: %s", cudaGetErrorString(e));
    }
    return TL_OK;
}

}  // namespace tlb

using namespace tlb;

extern "C" {

// The most tokens a tile may hold: 64 query rows per CTA, or (split_keys) 16; 0 where the form does not serve the sizes.
int tlb_paged_attention_flash_tile_tokens(int heads, int kv_heads, int split_keys) {
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads) return 0;
    const int group = heads / kv_heads, rows = split_keys ? 16 : 16 * kFWarps;
    if (split_keys && group > rows) return 0;
    return group >= rows ? 1 : rows / group;
}

int tlb_paged_attention_flash_supported(int dk, int dv, int kv_heads, int page_size) {
    return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 256 && kv_heads > 0 && page_size > 0 && page_size % 32 == 0;
}

int tlb_paged_attention_flash(const void *q, long long q_token, long long q_head, const void *slab, int num_pages, int page_size, int dk, int dv, int heads,
                              int kv_heads, const int32_t *block_table, int max_pages, const int32_t *tiles, int num_tiles, const int32_t *tok_pos,
                              int mask, int mask_size, int keep_first, float scale, float softcap, int sink, const void *gate, long long g_token, int gate_wide, void *out,
                              long long o_token, long long o_head, int split_keys, int splits, const float *head_bias, int weights, void *stream) {
    if (num_tiles <= 0) return TL_OK;
    if (weights < 0 || weights > 1 || (weights == 1 && (sink || softcap > 0.f))) return tl::fail(TL_EINVAL, "paged_attention_flash: bad weights mode");
    if (!q || !slab || !block_table || !tiles || !tok_pos || !out || heads <= 0 || kv_heads <= 0 || heads % kv_heads || max_pages <= 0 || num_pages <= 0)
        return tl::fail(TL_EINVAL, "paged_attention_flash: bad argument");
    if (!tlb_paged_attention_flash_supported(dk, dv, kv_heads, page_size))
        return tl::fail(TL_EINVAL, "paged_attention_flash: dk, dv multiples of 8 up to 256 and page_size %% 32 == 0 are required");
    if (mask < 0 || mask > 2 || (mask != 0 && mask_size <= 0) || keep_first < 0 || keep_first > (1 << 30) || (keep_first > 0 && mask != 1))
        return tl::fail(TL_EINVAL, "paged_attention_flash: bad mask");
    if (!tl::aligned16(slab)) return tl::fail(TL_EINVAL, "paged_attention_flash: the cache must be 16-byte aligned");
    if (tlb_paged_attention_flash_tile_tokens(heads, kv_heads, split_keys) == 0) return tl::fail(TL_EINVAL, "paged_attention_flash: too many query heads for this form");
    const int group = heads / kv_heads, rows = split_keys ? 16 : 16 * kFWarps, nv = f_units(dv);
    splits = splits < 1 ? 1 : splits > kFSplits ? kFSplits : splits;
    FlashArgs a;
    a.q = (const bf16 *)q, a.q_token = q_token, a.q_head = q_head, a.slab = (const bf16 *)slab, a.num_pages = num_pages, a.page_size = page_size;
    a.dk = dk, a.dv = dv, a.heads = heads, a.kv_heads = kv_heads, a.hp = group < rows ? group : rows;
    a.block_table = block_table, a.max_pages = max_pages, a.tiles = tiles, a.tok_pos = tok_pos;
    a.mask = mask, a.mask_size = mask_size, a.keep_first = keep_first, a.scale = scale, a.softcap = softcap, a.sink = sink;
    a.gate = (const bf16 *)gate, a.gate_wide = gate && gate_wide, a.g_token = g_token, a.out = (bf16 *)out, a.o_token = o_token, a.o_head = o_head, a.head_bias = head_bias, a.weights = weights;
    a.k_stride = ceil_div(dk, 16) * 16 + 8;  // (stride / 8) odd: conflict-free ldmatrix rows
    a.q_wide = tl::aligned16(q) && q_token % 8 == 0 && q_head % 8 == 0;
    a.o_pairs = (uintptr_t)out % 4 == 0 && o_token % 2 == 0 && o_head % 2 == 0;
    cudaStream_t st = as_stream(stream);
    int rc = TL_OK;
#define TLB_FLASH(N, K) rc = split_keys ? f_launch<N, true, K>(a, num_tiles, splits, st) : f_launch<N, false, K>(a, num_tiles, splits, st)
    const int kt = ceil_div(dk, 16);
    switch (nv) {
        case 2: TLB_FLASH(2, 0); break;
        case 4: if (kt == 4) TLB_FLASH(4, 4); else TLB_FLASH(4, 0); break;
        case 6: TLB_FLASH(6, 0); break;
        case 8: if (kt == 8) TLB_FLASH(8, 8); else TLB_FLASH(8, 0); break;
        case 12: TLB_FLASH(12, 0); break;
        default: TLB_FLASH(16, 0); break;
    }
#undef TLB_FLASH
    if (rc != TL_OK) return rc;
    TL_LAUNCH_CHECK("paged_attention_flash");
    return TL_OK;
}

}  // extern "C"
