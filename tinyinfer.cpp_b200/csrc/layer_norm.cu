// Norms of whole rows with a mean, and the sum of two normed rows.
//
//  * layer_norm_rows: out = (x - mean) / sqrt(var + eps) * w + b over rows of n elements, var the mean of the
//    squared deviations from the mean (a pass of its own over the row, which lies in registers); optionally of
//    gathered rows.
//  * norm_sum_rows: residual += scale (rms(a) * wa + rms(b) * wb), where rms(a) is the row over the root of its
//    mean square (+ eps): two sublayers side by side on their way into the residual.  With a layer norm behind it
//    (`then`), the same launch also writes that norm of the new residual rows.
//
// All arithmetic is float32.  A row belongs to a warp or to a block of 256 threads; which of the two depends on n
// and, for bfloat16 results, on the number of rows, so a float32 row's bits depend on the row alone.
#include "common.cuh"

namespace {

constexpr int THREADS = 256;

template <int TPR> __device__ __forceinline__ float row_sum(float v, float* scratch) {
    if constexpr (TPR == 32) return warp_sum(v);
    else return block_sum(v, scratch);
}
__device__ __forceinline__ float sum4(float4 v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float squares4(float4 v) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, v.x * v.x))); }
template <typename TO> __device__ __forceinline__ void put4(TO* p, float4 v) {
    if constexpr (sizeof(TO) == 2) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
    } else {
        *reinterpret_cast<float4*>(p) = v;
    }
}

// the layer norm of a row whose pieces v[j] (quad lane + TPR j) lie in registers
template <typename TO, int TPR, int MAXV>
__device__ __forceinline__ void normed_row(const float4 (&v)[MAXV], int lane, int n, const float* __restrict__ w,
                                           const float* __restrict__ b, float eps, TO* out, float* scratch) {
    const int n4 = n >> 2;
    float s = 0.0f;
#pragma unroll
    for (int j = 0; j < MAXV; ++j)
        if (lane + TPR * j < n4) s += sum4(v[j]);
    const float mean = row_sum<TPR>(s, scratch) / (float)n;
    float q = 0.0f;
#pragma unroll
    for (int j = 0; j < MAXV; ++j)
        if (lane + TPR * j < n4) q += squares4(make_float4(v[j].x - mean, v[j].y - mean, v[j].z - mean, v[j].w - mean));
    const float inv = 1.0f / sqrtf(row_sum<TPR>(q, scratch) / (float)n + eps);
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = lane + TPR * j;
        if (i >= n4) continue;
        const float4 g = __ldg(reinterpret_cast<const float4*>(w) + i), h = __ldg(reinterpret_cast<const float4*>(b) + i);
        put4<TO>(out + 4 * i, make_float4(fmaf((v[j].x - mean) * inv, g.x, h.x), fmaf((v[j].y - mean) * inv, g.y, h.y),
                                          fmaf((v[j].z - mean) * inv, g.z, h.z), fmaf((v[j].w - mean) * inv, g.w, h.w)));
    }
}

template <typename TO, int TPR, int MAXV>
__global__ void __launch_bounds__(THREADS)
layer_norm_rows_kernel(const float* x, const float* __restrict__ w, const float* __restrict__ b,
                       const int* __restrict__ rows, float eps, int n, int num_rows, TO* __restrict__ out) {
    __shared__ float scratch[32];
    pdl_launch();
    pdl_wait();
    const int r = TPR == 32 ? blockIdx.x * (THREADS / 32) + (threadIdx.x >> 5) : blockIdx.x;
    const int lane = TPR == 32 ? threadIdx.x & 31 : threadIdx.x;
    if (r >= num_rows) return;                            // whole warps only: no block-wide sum follows in that form
    const float4* xr = reinterpret_cast<const float4*>(x + (size_t)(rows ? rows[r] : r) * n);
    float4 v[MAXV];
#pragma unroll
    for (int j = 0; j < MAXV; ++j)
        if (lane + TPR * j < (n >> 2)) v[j] = xr[lane + TPR * j];
    normed_row<TO, TPR, MAXV>(v, lane, n, w, b, eps, out + (size_t)r * n, scratch);
}

// any n: a block per row, the row is read again for every pass
template <typename TO>
__global__ void __launch_bounds__(THREADS)
layer_norm_any_kernel(const float* x, const float* __restrict__ w, const float* __restrict__ b,
                      const int* __restrict__ rows, float eps, int n, TO* __restrict__ out) {
    __shared__ float scratch[32];
    pdl_launch();
    pdl_wait();
    const int r = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[r] : r) * n;
    float s = 0.0f;
    for (int i = threadIdx.x; i < n; i += THREADS) s += xr[i];
    const float mean = block_sum(s, scratch) / (float)n;
    float q = 0.0f;
    for (int i = threadIdx.x; i < n; i += THREADS) q = fmaf(xr[i] - mean, xr[i] - mean, q);
    const float inv = 1.0f / sqrtf(block_sum(q, scratch) / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += THREADS)
        out[(size_t)r * n + i] = from_f32<TO>(fmaf((xr[i] - mean) * inv, w[i], b[i]));
}

// What follows the sum in the same launch: a layer norm of the new residual row (out null: nothing).
struct Then { const float* w; const float* b; float eps; };

template <typename TO, int TPR, int MAXV>
__global__ void __launch_bounds__(THREADS)
norm_sum_rows_kernel(const float* a, const float* b, const float* __restrict__ wa, const float* __restrict__ wb,
                     float eps, float scale, float* residual, int res_stride, int n, int num_rows, const Then then,
                     TO* __restrict__ out) {
    __shared__ float scratch[32];
    pdl_launch();
    pdl_wait();
    const int r = TPR == 32 ? blockIdx.x * (THREADS / 32) + (threadIdx.x >> 5) : blockIdx.x;
    const int lane = TPR == 32 ? threadIdx.x & 31 : threadIdx.x;
    if (r >= num_rows) return;
    const int n4 = n >> 2;
    const float4* ar = reinterpret_cast<const float4*>(a + (size_t)r * n);
    const float4* br = reinterpret_cast<const float4*>(b + (size_t)r * n);
    float4* xr = reinterpret_cast<float4*>(residual + (size_t)r * res_stride);
    float4 va[MAXV], vb[MAXV];
#pragma unroll
    for (int j = 0; j < MAXV; ++j)
        if (lane + TPR * j < n4) { va[j] = ar[lane + TPR * j]; vb[j] = br[lane + TPR * j]; }
    float sa = 0.0f, sb = 0.0f;
#pragma unroll
    for (int j = 0; j < MAXV; ++j)
        if (lane + TPR * j < n4) { sa += squares4(va[j]); sb += squares4(vb[j]); }
    const float ia = 1.0f / sqrtf(row_sum<TPR>(sa, scratch) / (float)n + eps);
    const float ib = 1.0f / sqrtf(row_sum<TPR>(sb, scratch) / (float)n + eps);
#pragma unroll
    for (int j = 0; j < MAXV; ++j) {
        const int i = lane + TPR * j;
        if (i >= n4) continue;
        const float4 ga = __ldg(reinterpret_cast<const float4*>(wa) + i), gb = __ldg(reinterpret_cast<const float4*>(wb) + i);
        float4 x = xr[i];
        x.x = fmaf(scale, fmaf(va[j].x * ia, ga.x, vb[j].x * ib * gb.x), x.x);
        x.y = fmaf(scale, fmaf(va[j].y * ia, ga.y, vb[j].y * ib * gb.y), x.y);
        x.z = fmaf(scale, fmaf(va[j].z * ia, ga.z, vb[j].z * ib * gb.z), x.z);
        x.w = fmaf(scale, fmaf(va[j].w * ia, ga.w, vb[j].w * ib * gb.w), x.w);
        xr[i] = x;
        va[j] = x;
    }
    if (out != nullptr)
        normed_row<TO, TPR, MAXV>(va, lane, n, then.w, then.b, then.eps, out + (size_t)r * n, scratch);
}

template <typename TO>
__global__ void __launch_bounds__(THREADS)
norm_sum_any_kernel(const float* a, const float* b, const float* __restrict__ wa, const float* __restrict__ wb,
                    float eps, float scale, float* residual, int res_stride, int n, const Then then,
                    TO* __restrict__ out) {
    __shared__ float scratch[32];
    pdl_launch();
    pdl_wait();
    const size_t r = blockIdx.x;
    const float* ar = a + r * n;
    const float* br = b + r * n;
    float* xr = residual + r * res_stride;
    float sa = 0.0f, sb = 0.0f;
    for (int i = threadIdx.x; i < n; i += THREADS) { sa = fmaf(ar[i], ar[i], sa); sb = fmaf(br[i], br[i], sb); }
    const float ia = 1.0f / sqrtf(block_sum(sa, scratch) / (float)n + eps);
    const float ib = 1.0f / sqrtf(block_sum(sb, scratch) / (float)n + eps);
    float s = 0.0f;
    for (int i = threadIdx.x; i < n; i += THREADS) {       // a thread meets the same elements in every pass
        const float x = fmaf(scale, fmaf(ar[i] * ia, wa[i], br[i] * ib * wb[i]), xr[i]);
        xr[i] = x;
        s += x;
    }
    if (out == nullptr) return;
    const float mean = block_sum(s, scratch) / (float)n;
    float q = 0.0f;
    for (int i = threadIdx.x; i < n; i += THREADS) q = fmaf(xr[i] - mean, xr[i] - mean, q);
    const float inv = 1.0f / sqrtf(block_sum(q, scratch) / (float)n + then.eps);
    for (int i = threadIdx.x; i < n; i += THREADS)
        out[r * n + i] = from_f32<TO>(fmaf((xr[i] - mean) * inv, then.w[i], then.b[i]));
}

bool aligned16(const void* p) { return (uintptr_t)p % 16 == 0; }

// quads of a row per thread and the threads of a row; false: the general kernel
bool form(int n, int num_rows, bool f32, int most_of_a_warp, bool& warp) {
    warp = !f32 && n <= most_of_a_warp && num_rows >= 1024;
    return n % 4 == 0 && n <= 4 * THREADS * 8;
}

}  // namespace

extern "C" int ti_layer_norm_rows(const float* x, const float* w, const float* b, const int* rows, int num_rows, int n,
                                  float eps, void* out, int out_dtype, void* stream) {
    if (num_rows == 0 || n == 0) return 0;
    TI_REQUIRE(out_dtype == TI_F32 || out_dtype == TI_BF16, "layer_norm_rows: output dtype code %d", out_dtype);
    cudaStream_t s = (cudaStream_t)stream;
    bool warp;
    const bool regs = form(n, num_rows, out_dtype == TI_F32, 2048, warp) && aligned16(x) && aligned16(w) && aligned16(b) &&
                      aligned16(out);
    const int quads = (n / 4 + (warp ? 31 : THREADS - 1)) / (warp ? 32 : THREADS);
#define LAUNCH(TO, TPR, MAXV)                                                                                       \
    ti_launch_pdl(layer_norm_rows_kernel<TO, TPR, MAXV>, dim3(TPR == 32 ? (num_rows + 7) / 8 : num_rows), dim3(THREADS), \
                  0, s, x, w, b, rows, eps, n, num_rows, (TO*)out)
#define CALL(TO)                                                                                                    \
    if (!regs) ti_launch_pdl(layer_norm_any_kernel<TO>, dim3(num_rows), dim3(THREADS), 0, s, x, w, b, rows, eps, n, (TO*)out); \
    else if (warp) { if (quads <= 4) LAUNCH(TO, 32, 4); else if (quads <= 8) LAUNCH(TO, 32, 8); else LAUNCH(TO, 32, 16); } \
    else { if (quads <= 1) LAUNCH(TO, 256, 1); else if (quads <= 2) LAUNCH(TO, 256, 2);                              \
           else if (quads <= 4) LAUNCH(TO, 256, 4); else LAUNCH(TO, 256, 8); }
    if (out_dtype == TI_F32) { CALL(float) } else { CALL(bf16) }
#undef CALL
#undef LAUNCH
    return ti_check_launch("layer_norm_rows");
}

// a, b: float32 [num_rows, n]; wa, wb: a weight per element.  out (may be null): the layer norm (then_w, then_b,
// then_eps) of the new residual rows.
extern "C" int ti_norm_sum_rows(const float* a, const float* b, const float* wa, const float* wb, float eps, float scale,
                                float* residual, int res_stride, int num_rows, int n, const float* then_w,
                                const float* then_b, float then_eps, void* out, int out_dtype, void* stream) {
    if (num_rows == 0 || n == 0) return 0;
    TI_REQUIRE(out_dtype == TI_F32 || out_dtype == TI_BF16, "norm_sum_rows: output dtype code %d", out_dtype);
    TI_REQUIRE(out == nullptr || (then_w != nullptr && then_b != nullptr), "norm_sum_rows: the norm behind the sum");
    cudaStream_t s = (cudaStream_t)stream;
    bool warp;
    const bool regs = form(n, num_rows, out_dtype == TI_F32, 512, warp) && res_stride % 4 == 0 && aligned16(a) &&
                      aligned16(b) && aligned16(wa) && aligned16(wb) && aligned16(residual) && aligned16(then_w) &&
                      aligned16(then_b) && aligned16(out);
    const int quads = (n / 4 + (warp ? 31 : THREADS - 1)) / (warp ? 32 : THREADS);
    const Then then{then_w, then_b, then_eps};
#define LAUNCH(TO, TPR, MAXV)                                                                                       \
    ti_launch_pdl(norm_sum_rows_kernel<TO, TPR, MAXV>, dim3(TPR == 32 ? (num_rows + 7) / 8 : num_rows), dim3(THREADS),  \
                  0, s, a, b, wa, wb, eps, scale, residual, res_stride, n, num_rows, then, (TO*)out)
#define CALL(TO)                                                                                                    \
    if (!regs) ti_launch_pdl(norm_sum_any_kernel<TO>, dim3(num_rows), dim3(THREADS), 0, s, a, b, wa, wb, eps, scale,     \
                             residual, res_stride, n, then, (TO*)out);                                              \
    else if (warp) LAUNCH(TO, 32, 4);                                                                               \
    else { if (quads <= 1) LAUNCH(TO, 256, 1); else if (quads <= 2) LAUNCH(TO, 256, 2);                              \
           else if (quads <= 4) LAUNCH(TO, 256, 4); else LAUNCH(TO, 256, 8); }
    if (out_dtype == TI_F32) { CALL(float) } else { CALL(bf16) }
#undef CALL
#undef LAUNCH
    return ti_check_launch("norm_sum_rows");
}
