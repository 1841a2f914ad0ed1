// What the prompt attention kernels on tcgen05 share: their parameters, the swizzled layouts, the sink, and the
// kernel that puts key ranges together.
#pragma once

#include "common.cuh"
#include "sm100.cuh"

namespace chibi {

using namespace sm100;

struct AttnTcParams {
    const __nv_bfloat16* q;
    __nv_bfloat16* out;
    const int* block_table;
    int table_stride;
    const int* seq_rows;
    const int* q_start;
    const int* ctx_len;
    int nq, nkv, group;
    int page_size;
    long long cache_rows;        // pages * nkv * page_size: rows of the [rows, D] view of a cache
    int num_pages;
    float scale_log2;
    int window;
    int chunk;                     // 0: none; else a row sees only keys of its own block of this many positions
    int skip_single;
    int* error;
    // Options of the score (the kernel with one query tile per CTA only): a soft cap c replaces a
    // scaled score s by c * tanh(s / c); a bias by distance then takes r1 * ln(1 + r2 * (pos - key))
    // off, with r1 and r2 per query head.
    float scale;                   // the plain scale
    float softcap;                 // 0: none
    const float* bias_r1;          // [nq] or null
    const float* bias_r2;
    // The kernel with one query tile per CTA may cut the keys of a row tile into kv_splits ranges,
    // one CTA each (few query rows over a long context would leave most SMs idle otherwise): every
    // CTA then leaves its unnormalised output, maximum and sum per row, and
    // attn_prefill_merge_kernel puts the ranges together.
    int kv_splits;                 // 1: none
    float* part_o;                 // [tokens][nq][kv_splits][D]
    float* part_ml;                // [tokens][nq][kv_splits][2]
    const float* sink;             // [nq] or null: exp(sink[head]) joins the softmax's denominator, once
};

// What the sink adds to a row's sum of weights, which is kept relative to the running maximum
// `m` (in units of log2; -inf while no key has been seen, then the sum is relative to 0).
__device__ __forceinline__ float sink_weight(const float* sink, int head, float m)
{
    return sink ? exp2f(sink[head] * 1.4426950408889634f - (m == -INFINITY ? 0.f : m)) : 0.f;
}

// Byte offset of element (row, col) of a [rows][64] bf16 tile laid out with the
// 128-byte swizzle (what TMA writes and tcgen05.mma reads): 16-byte chunk c of
// row r sits at chunk position c ^ (r % 8).
__device__ __forceinline__ uint32_t swizzled_chunk(int row, int chunk)
{
    return (uint32_t)row * 128u + (uint32_t)((chunk ^ (row & 7)) << 4);
}

__device__ __forceinline__ float fast_exp2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// MN-major operand (here V: [key][d], d contiguous) in the same swizzled tiles:
// leading byte offset = distance between the 64-wide slices of d, stride byte
// offset = 8 keys * 128 B.
__device__ __forceinline__ uint64_t make_mnmajor_sw128_desc(uint32_t smem_byte_addr, uint32_t lbo_bytes)
{
    uint64_t d = 0;
    d |= static_cast<uint64_t>((smem_byte_addr & 0x3ffff) >> 4);
    d |= static_cast<uint64_t>((lbo_bytes >> 4) & 0x3fff) << 16;
    d |= static_cast<uint64_t>(1024 >> 4) << 32;
    d |= static_cast<uint64_t>(1) << 46;
    d |= static_cast<uint64_t>(2) << 61;
    return d;
}

// Puts the key ranges of a row tile together: one block of D threads for each
// (head, token of a sequence); ranges in order, eight at a time.
template <int D>
__global__ void attn_prefill_merge_kernel(const AttnTcParams p)
{
    pdl_trigger();
    const int seq = blockIdx.z, head = blockIdx.x, c = threadIdx.x;
    const int t0 = p.q_start[seq];
    const int q_len = p.q_start[seq + 1] - t0;
    if ((int)blockIdx.y >= q_len || (q_len == 1 && p.skip_single))
        return;
    pdl_wait();
    const size_t slot0 = ((size_t)(t0 + blockIdx.y) * p.nq + head) * p.kv_splits;
    float m_run = -INFINITY, acc = 0.f, lsum = 0.f;
    for (int s0 = 0; s0 < p.kv_splits; s0 += 8) {
        float mv[8], lv[8], ov[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const bool in = s0 + u < p.kv_splits;
            mv[u] = in ? p.part_ml[(slot0 + s0 + u) * 2] : -INFINITY;
            lv[u] = in ? p.part_ml[(slot0 + s0 + u) * 2 + 1] : 0.f;
            ov[u] = in ? p.part_o[(slot0 + s0 + u) * D + c] : 0.f;
        }
        float m_new = m_run;
#pragma unroll
        for (int u = 0; u < 8; ++u)
            m_new = fmaxf(m_new, mv[u]);
        const float base = m_new == -INFINITY ? 0.f : m_new;
        const float keep = exp2f(m_run - base);       // 0 while nothing has been seen
        acc *= keep;
        lsum *= keep;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const float f = exp2f(mv[u] - base);
            acc += ov[u] * f;
            lsum += lv[u] * f;
        }
        m_run = m_new;
    }
    lsum += sink_weight(p.sink, head, m_run);
    p.out[((size_t)(t0 + blockIdx.y) * p.nq + head) * D + c] = __float2bfloat16_rn(lsum > 0.f ? acc / lsum : 0.f);
}

} // namespace chibi
