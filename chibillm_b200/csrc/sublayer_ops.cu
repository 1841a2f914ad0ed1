// The row-wise kernels around the sublayers of a block with norms on the sublayers' results and a weighted
// sum over all layers' results so far:
//
// * sublayer_end: y = sum of a product's partial sums (or one array) + bias; residual += vec * y / rms(y) (or
//   vec * y); then, at a block's end, the new residual is kept as this layer's result X and replaced by
//   sum_j c[j] X_j over the embedding output and all results so far; then the next norm's output.
// * norm_then_gate: x / rms(x over the whole row) * weight * sigmoid(gate).
// * bias_xielu: z = x + bias; z > 0: p z^2 + z / 2, else n (exp(z) - 1 - z) + z / 2.
//
// Sums, statistics, gates and the residual are 32-bit whatever the activations' type is.
#define CHIBI_UNIT sublayer_ops
#define CHIBI_UNIT_ID 13
#include "common.cuh"
#include "sm100.cuh"

namespace chibi {

using namespace sm100;

__device__ __forceinline__ void store4(float* dst, float a, float b, float c, float d)
{
    *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store4(__nv_bfloat16* dst, float a, float b, float c, float d)
{
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<const uint32_t*>(&lo), v.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = v;
}

struct SublayerEnd {
    float* residual;                 // [rows, n]
    const float* delta;              // [splits, rows, n]
    int splits;
    const float* bias;               // [n] or null
    const float* vec;                // [n]
    float y_eps;                     // below 0: y is not normalised
    float* outputs;                  // [.., rows, n]: X_0 .. X_(earlier - 1), then this layer's; null: no depth sum
    const float* weights;            // [earlier + 1]
    int earlier;
    int keep;                        // this layer's result goes to outputs[earlier]
    float eps, offset;               // of the norm that follows
    long long rows;
    int n;
};

// A thread owns V runs of four neighbouring columns of a row (n = 4 V gridDim.x blockDim.x), a run's threads side
// by side; the gridDim.x CTAs of a row form a cluster that adds up its sums of squares through one another's
// shared memory.  Everything a row needs is asked for before its first sum of squares: the earlier results'
// weighted sum does not depend on this layer's.
template <int V, typename TW, typename TO>
__global__ void __launch_bounds__(1024 / V)
sublayer_end_kernel(const SublayerEnd p, const TW* __restrict__ norm_w, TO* __restrict__ out)
{
    pdl_trigger();
    __shared__ float scratch[33];
    __shared__ float sums[2][8];
    const int parts = gridDim.x;
    const int c = 4 * (blockIdx.x * V * blockDim.x + threadIdx.x), step = 4 * blockDim.x;
    const long long t = blockIdx.y + (long long)blockIdx.z * gridDim.y;
    if (t >= p.rows)
        return;                                        // a whole cluster leaves together
    const size_t at = (size_t)t * p.n + c;
    const size_t plane = (size_t)p.rows * p.n;
    auto whole_row = [&](float s, int which) {
        s = block_sum(s, scratch);
        if (parts == 1)
            return s;
        if ((int)threadIdx.x < parts)
            st_peer_shared_f32(smem_addr(&sums[which][cluster_cta_rank()]), threadIdx.x, s);
        cluster_sync();
        float total = 0.f;
        for (int r = 0; r < parts; ++r)
            total += sums[which][r];
        return total;
    };
    auto load4 = [](const float* src) { return *reinterpret_cast<const float4*>(src); };
    if (parts > 1)
        cluster_sync();                                // every CTA of the row has started: its shared memory is there
    pdl_wait();
    float4 r[V], y[V], sum[V];
    float own = 1.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        r[i] = load4(p.residual + at + i * step);
        y[i] = p.bias ? load4(p.bias + c + i * step) : make_float4(0.f, 0.f, 0.f, 0.f);
        sum[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    constexpr int AHEAD = V == 1 ? 8 : 2;              // arrays whose loads are in flight together
    for (int s0 = 0; s0 < p.splits; s0 += AHEAD) {
        float4 q[AHEAD][V];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
#pragma unroll
            for (int i = 0; i < V; ++i)
                q[u][i] = s0 + u < p.splits ? load4(p.delta + (size_t)(s0 + u) * plane + at + i * step)
                                            : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
#pragma unroll
            for (int i = 0; i < V; ++i)
                y[i].x += q[u][i].x, y[i].y += q[u][i].y, y[i].z += q[u][i].z, y[i].w += q[u][i].w;
    }
    if (p.outputs) {
        own = p.weights[p.earlier];
        for (int j0 = 0; j0 < p.earlier; j0 += AHEAD) {
            float4 q[AHEAD][V];
            float k[AHEAD];
#pragma unroll
            for (int u = 0; u < AHEAD; ++u) {
                const bool on = j0 + u < p.earlier;
                k[u] = on ? p.weights[j0 + u] : 0.f;
#pragma unroll
                for (int i = 0; i < V; ++i)
                    q[u][i] = on ? load4(p.outputs + (size_t)(j0 + u) * plane + at + i * step)
                                 : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int u = 0; u < AHEAD; ++u)
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    sum[i].x = fmaf(k[u], q[u][i].x, sum[i].x);
                    sum[i].y = fmaf(k[u], q[u][i].y, sum[i].y);
                    sum[i].z = fmaf(k[u], q[u][i].z, sum[i].z);
                    sum[i].w = fmaf(k[u], q[u][i].w, sum[i].w);
                }
        }
    }
    float inv = 1.f;
    if (p.y_eps >= 0.f) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < V; ++i)
            s = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, s))));
        inv = 1.f / sqrtf(whole_row(s, 0) / (float)p.n + p.y_eps);
    }
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const float4 v = load4(p.vec + c + i * step);
        r[i].x = fmaf(v.x, y[i].x * inv, r[i].x);
        r[i].y = fmaf(v.y, y[i].y * inv, r[i].y);
        r[i].z = fmaf(v.z, y[i].z * inv, r[i].z);
        r[i].w = fmaf(v.w, y[i].w * inv, r[i].w);
        if (p.outputs) {
            if (p.keep)
                *reinterpret_cast<float4*>(p.outputs + (size_t)p.earlier * plane + at + i * step) = r[i];
            r[i].x = fmaf(own, r[i].x, sum[i].x);
            r[i].y = fmaf(own, r[i].y, sum[i].y);
            r[i].z = fmaf(own, r[i].z, sum[i].z);
            r[i].w = fmaf(own, r[i].w, sum[i].w);
        }
        *reinterpret_cast<float4*>(p.residual + at + i * step) = r[i];
        s = fmaf(r[i].x, r[i].x, fmaf(r[i].y, r[i].y, fmaf(r[i].z, r[i].z, fmaf(r[i].w, r[i].w, s))));
    }
    if (!out)
        return;
    const float f = 1.f / sqrtf(whole_row(s, 1) / (float)p.n + p.eps);
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const TW* w = norm_w + c + i * step;
        store4(out + at + i * step, r[i].x * f * (to_f32(w[0]) + p.offset), r[i].y * f * (to_f32(w[1]) + p.offset),
               r[i].z * f * (to_f32(w[2]) + p.offset), r[i].w * f * (to_f32(w[3]) + p.offset));
    }
}

// The same for any width: one block per row, the row in shared memory.
template <typename TW, typename TO>
__global__ void __launch_bounds__(256)
sublayer_end_any_kernel(const SublayerEnd p, const TW* __restrict__ norm_w, TO* __restrict__ out)
{
    pdl_enter();
    extern __shared__ float row[];
    __shared__ float scratch[33];
    const size_t t = blockIdx.x;
    const size_t plane = (size_t)p.rows * p.n;
    float ssq = 0.f;
    for (int c = threadIdx.x; c < p.n; c += blockDim.x) {
        float y = p.bias ? p.bias[c] : 0.f;
        for (int s = 0; s < p.splits; ++s)
            y += p.delta[(size_t)s * plane + t * p.n + c];
        row[c] = y;
        ssq = fmaf(y, y, ssq);
    }
    float inv = 1.f;
    if (p.y_eps >= 0.f)
        inv = 1.f / sqrtf(block_sum(ssq, scratch) / (float)p.n + p.y_eps);
    ssq = 0.f;
    for (int c = threadIdx.x; c < p.n; c += blockDim.x) {
        const size_t at = t * p.n + c;
        float r = fmaf(p.vec[c], row[c] * inv, p.residual[at]);
        if (p.outputs) {
            if (p.keep)
                p.outputs[(size_t)p.earlier * plane + at] = r;
            r *= p.weights[p.earlier];
            for (int j = 0; j < p.earlier; ++j)
                r = fmaf(p.weights[j], p.outputs[(size_t)j * plane + at], r);
        }
        p.residual[at] = r;
        row[c] = r;
        ssq = fmaf(r, r, ssq);
    }
    if (!out)
        return;
    const float f = 1.f / sqrtf(block_sum(ssq, scratch) / (float)p.n + p.eps);
    for (int c = threadIdx.x; c < p.n; c += blockDim.x)
        out[t * p.n + c] = from_f32<TO>(row[c] * f * (to_f32(norm_w[c]) + p.offset));
}

// ---------------------------------------------------------------- norm of a row, then a gate
// One block per row; a thread keeps up to NG_KEEP of its values in registers between the sum of squares and
// the output, a longer row is read again.
constexpr int NG_KEEP = 8;

template <typename TX>
__global__ void __launch_bounds__(512)
norm_then_gate_kernel(const float* __restrict__ x, const TX* __restrict__ gate, long long gate_stride,
                      const float* __restrict__ weight, float eps, TX* __restrict__ out, int n)
{
    pdl_enter();
    __shared__ float scratch[33];
    const size_t t = blockIdx.x;
    const float* xr = x + t * n;
    const TX* gr = gate + t * gate_stride;
    const bool kept = n <= (int)blockDim.x * NG_KEEP;
    float v[NG_KEEP], g[NG_KEEP];
    float ssq = 0.f;
    if (kept) {
#pragma unroll
        for (int k = 0; k < NG_KEEP; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            v[k] = c < n ? xr[c] : 0.f;
            g[k] = c < n ? to_f32(gr[c]) : 0.f;
            ssq = fmaf(v[k], v[k], ssq);
        }
    } else {
        for (int c = threadIdx.x; c < n; c += blockDim.x)
            ssq = fmaf(xr[c], xr[c], ssq);
    }
    const float inv = 1.f / sqrtf(block_sum(ssq, scratch) / (float)n + eps);
    if (kept) {
#pragma unroll
        for (int k = 0; k < NG_KEEP; ++k) {
            const int c = threadIdx.x + k * blockDim.x;
            if (c < n)
                out[t * n + c] = from_f32<TX>(v[k] * inv * weight[c] / (1.f + expf(-g[k])));
        }
        return;
    }
    for (int c = threadIdx.x; c < n; c += blockDim.x)
        out[t * n + c] = from_f32<TX>(xr[c] * inv * weight[c] / (1.f + expf(-to_f32(gr[c]))));
}

// ---------------------------------------------------------------- xIELU
__device__ __forceinline__ float xielu(float z, float pos, float neg)
{
    return z > 0.f ? fmaf(pos * z, z, 0.5f * z) : fmaf(neg, expm1f(z) - z, 0.5f * z);
}

// The same for results that become bfloat16 at once: exp(z) - 1 - z as the first terms of its series next to
// zero (where the difference would cancel) and as the difference of the faster exponential elsewhere; good to
// 1e-4 of the result.
__device__ __forceinline__ float xielu_rounded(float z, float pos, float neg)
{
    const float series = z * z * fmaf(z, fmaf(z, 1.f / 24.f, 1.f / 6.f), 0.5f);
    const float rest = z > -0.0625f ? series : __expf(z) - 1.f - z;
    return z > 0.f ? fmaf(pos * z, z, 0.5f * z) : fmaf(neg, rest, 0.5f * z);
}

// x: [splits, rows, n] (partial sums of a product when there are several) or an array that may be `out`
template <typename TX, typename TO>
__global__ void bias_xielu_kernel(const TX* x, int splits, const float* __restrict__ bias, TO* out, long long rows, int n,
                                  float pos, float neg)
{
    pdl_enter();
    const long long total = rows * n;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total;
         i += (long long)gridDim.x * blockDim.x) {
        float z = bias ? bias[i % n] : 0.f;
        for (int s = 0; s < splits; ++s)
            z += to_f32(x[(size_t)s * total + i]);
        out[i] = from_f32<TO>(xielu(z, pos, neg));
    }
}

// four columns a thread from 32-bit partial sums; n a multiple of 4
template <typename TO>
__global__ void bias_xielu_partial_kernel(const float* __restrict__ x, int splits, const float* __restrict__ bias,
                                          TO* __restrict__ out, long long rows, int n, float pos, float neg)
{
    pdl_enter();
    const int c = 4 * (blockIdx.x * blockDim.x + threadIdx.x);
    if (c >= n)
        return;
    const size_t at = (size_t)blockIdx.y * n + c, plane = (size_t)rows * n;
    float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
    if (bias)
        z = *reinterpret_cast<const float4*>(bias + c);
    for (int s0 = 0; s0 < splits; s0 += 8) {
        float4 q[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            q[u] = s0 + u < splits ? *reinterpret_cast<const float4*>(x + (size_t)(s0 + u) * plane + at)
                                   : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 8; ++u)
            z.x += q[u].x, z.y += q[u].y, z.z += q[u].z, z.w += q[u].w;
    }
    out[at] = from_f32<TO>(xielu(z.x, pos, neg));
    out[at + 1] = from_f32<TO>(xielu(z.y, pos, neg));
    out[at + 2] = from_f32<TO>(xielu(z.z, pos, neg));
    out[at + 3] = from_f32<TO>(xielu(z.w, pos, neg));
}

// bfloat16, 16 bytes a thread; n a multiple of 8, x may be out
__global__ void bias_xielu_wide_kernel(const __nv_bfloat16* x, const float* __restrict__ bias, __nv_bfloat16* out,
                                       long long rows, int n, float pos, float neg)
{
    pdl_enter();
    const int c = 8 * (blockIdx.x * blockDim.x + threadIdx.x);
    if (c >= n)
        return;
    float b[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
        b[j] = bias ? bias[c + j] : 0.f;
    for (long long t = blockIdx.y; t < rows; t += gridDim.y) {
        uint4 raw = *reinterpret_cast<const uint4*>(x + t * n + c);
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 z = __bfloat1622float2(h[j]);
            h[j] = __floats2bfloat162_rn(xielu_rounded(z.x + b[2 * j], pos, neg),
                                         xielu_rounded(z.y + b[2 * j + 1], pos, neg));
        }
        *reinterpret_cast<uint4*>(out + t * n + c) = raw;
    }
}

static inline unsigned sublayer_blocks(long long work, int threads)
{
    const long long b = (work + threads - 1) / threads;
    return (unsigned)(b < 1 ? 1 : (b > 148LL * 16 ? 148LL * 16 : b));
}

} // namespace chibi

using namespace chibi;

// `outputs` null: no depth sum.  y_eps < 0: y is not normalised.  out null: no norm follows.
CHIBI_API int chibi_sublayer_end(float* residual, const float* delta, int splits, const float* bias, const float* vec,
                                 float y_eps, float* outputs, const float* weights, int earlier, int keep,
                                 const void* norm_w, int w_type, float eps, float offset, void* out, int out_type,
                                 long long rows, int n, cudaStream_t stream)
{
    if (rows <= 0)
        return CHIBI_OK;
    if (!residual || !delta || splits < 1 || !vec || n <= 0 || (out && !norm_w) || (outputs && (!weights || earlier < 1)))
        return CHIBI_ERR_ARGUMENT;
    SublayerEnd p = { residual, delta, splits, bias, vec, y_eps, outputs, weights, earlier, keep, eps, offset, rows, n };
    const uintptr_t all = reinterpret_cast<uintptr_t>(residual) | reinterpret_cast<uintptr_t>(delta)
                          | reinterpret_cast<uintptr_t>(bias) | reinterpret_cast<uintptr_t>(vec)
                          | reinterpret_cast<uintptr_t>(outputs);
    const int n4 = n / 4;
    int parts = 0, runs = 1;           // CTAs per row and runs of columns per thread
    if (n % 128 == 0 && (all & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0) {
        if (rows <= 64) {
            // few rows: as many CTAs to a row as divide it evenly
            for (int cand = 1; cand <= 8; ++cand)
                if (n4 % cand == 0 && (n4 / cand) % 32 == 0 && n4 / cand <= 1024)
                    parts = cand;
        } else {
            // many rows: small blocks, several of them to an SM
            runs = n4 % 128 == 0 && n4 >= 512 ? 4 : (n4 % 64 == 0 && n4 >= 256 ? 2 : 1);
            for (int cand = 1; cand <= 8 && parts == 0; ++cand)
                if (n4 % (runs * cand) == 0 && (n4 / (runs * cand)) % 32 == 0 && n4 / (runs * cand) <= 1024 / runs)
                    parts = cand;
        }
    }
    if (parts > 0) {
        const unsigned gy = (unsigned)(rows < 32768 ? rows : 32768), gz = (unsigned)((rows + gy - 1) / gy);
        if (gz > 65535)
            return CHIBI_ERR_UNSUPPORTED;
        const dim3 grid((unsigned)parts, gy, gz), block((unsigned)(n4 / (parts * runs)));
        CHIBI_DISPATCH_TYPE(w_type, TW, CHIBI_DISPATCH_TYPE(out_type, TO, {
            auto kernel = runs == 4 ? sublayer_end_kernel<4, TW, TO>
                                    : runs == 2 ? sublayer_end_kernel<2, TW, TO> : sublayer_end_kernel<1, TW, TO>;
            if (parts > 1)
                launch_cluster_x(kernel, grid, block, 0, stream, parts, p, (const TW*)norm_w, (TO*)out);
            else
                launch(kernel, grid, block, 0, stream, p, (const TW*)norm_w, (TO*)out);
        }));
        return launch_status();
    }
    const size_t smem = (size_t)n * sizeof(float);
    if (smem > 200 * 1024 || rows > 2147483647LL)
        return CHIBI_ERR_UNSUPPORTED;
    CHIBI_DISPATCH_TYPE(w_type, TW, CHIBI_DISPATCH_TYPE(out_type, TO, {
        auto kernel = sublayer_end_any_kernel<TW, TO>;
        if (smem > 47 * 1024)
            cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        launch(kernel, dim3((unsigned)rows), dim3(256), smem, stream, p, (const TW*)norm_w, (TO*)out);
    }));
    return launch_status();
}

CHIBI_API int chibi_norm_then_gate(const float* x, const void* gate, int x_type, long long gate_stride,
                                   const float* weight, float eps, void* out, long long rows, int n, cudaStream_t stream)
{
    if (rows <= 0)
        return CHIBI_OK;
    if (!x || !gate || !weight || !out || n <= 0)
        return CHIBI_ERR_ARGUMENT;
    if (rows > 2147483647LL)
        return CHIBI_ERR_UNSUPPORTED;
    int threads = 64;
    while (threads < 512 && threads * NG_KEEP < n)
        threads <<= 1;
    CHIBI_DISPATCH_TYPE(x_type, TX, {
        launch(norm_then_gate_kernel<TX>, dim3((unsigned)rows), dim3(threads), 0, stream, x, (const TX*)gate, gate_stride,
               weight, eps, (TX*)out, n);
    });
    return launch_status();
}

CHIBI_API int chibi_bias_xielu(const void* x, int x_type, int splits, const float* bias, void* out, int out_type,
                               long long rows, int n, float pos, float neg, cudaStream_t stream)
{
    if (rows <= 0 || n <= 0)
        return CHIBI_OK;
    if (!x || !out || splits < 1 || (splits > 1 && x == out))
        return CHIBI_ERR_ARGUMENT;
    const uintptr_t all = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(bias);
    if (x_type == CHIBI_F32 && x != out && n % 4 == 0 && (all & 15) == 0 && rows <= 65535) {
        CHIBI_DISPATCH_TYPE(out_type, TO, {
            launch(bias_xielu_partial_kernel<TO>, dim3((unsigned)((n / 4 + 127) / 128), (unsigned)rows), dim3(128), 0, stream,
                   (const float*)x, splits, bias, (TO*)out, rows, n, pos, neg);
        });
        return launch_status();
    }
    if (x_type == CHIBI_BF16 && out_type == CHIBI_BF16 && splits == 1 && n % 8 == 0 && (all & 15) == 0) {
        launch(bias_xielu_wide_kernel, dim3((unsigned)((n / 8 + 127) / 128), (unsigned)(rows < 16384 ? rows : 16384)),
               dim3(128), 0, stream, (const __nv_bfloat16*)x, bias, (__nv_bfloat16*)out, rows, n, pos, neg);
        return launch_status();
    }
    CHIBI_DISPATCH_TYPE(x_type, TX, CHIBI_DISPATCH_TYPE(out_type, TO, {
        launch(bias_xielu_kernel<TX, TO>, dim3(sublayer_blocks(rows * n, 256)), dim3(256), 0, stream, (const TX*)x, splits,
               bias, (TO*)out, rows, n, pos, neg);
    }));
    return launch_status();
}
