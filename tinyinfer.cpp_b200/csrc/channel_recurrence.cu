// Linear recurrences per channel and the gates and decays in front of them.  All arithmetic is float32.
//
//  * low_rank_decay: out[t, c] = sigmoid(sum_r low[t, r] a2[c, r] + bias[c])^(1/tau), the decay of a gated
//    linear attention's key channels.  A thread per channel walks the inner width in order.
//  * gated_recurrence: per channel, over a request's tokens in order,
//        a = exp(L sigmoid(zr + br));   S <- a S + sqrt(1 - a^2) sigmoid(zi + bi) u;   out = S gelu(y + by)
//    with L <= 0 a constant of the channel and S in the request's state slot.  One block walks a request's
//    tokens for 8, 16 or 32 channels: fifteen warps turn a tile's inputs into (a, b) pairs and finished
//    states into output rows, one warp does nothing but S <- a S + b.  While it walks tile i, the others
//    prepare tile i + 1, write out tile i - 1 and have the loads of the tiles behind on their way.  Every channel's chain is one multiply-add per token in
//    order, so a row's bits depend neither on the batch nor on how a prompt was cut.
//  * gated_recurrence_single: the same for steps in which every request brings one token, with the block-
//    diagonal products z = W u in front.  A block takes 16 channels of a part: its warps read the 32 rows of W
//    once for up to 16 requests and meet by halving (each exchange halves the sums a lane still holds).
//  * split_rows: a float32 row as three bfloat16 rows that add up to it (24 of its 24 bits), laid out so that
//    one grouped tensor-core product with a weight that repeats itself three times along k gives float32 sums.
#include "common.cuh"

namespace {

// ---- decays ---------------------------------------------------------------------------------------
constexpr int LD_TOKENS = 16, LD_RANK = 32;

template <typename TW>
__global__ void __launch_bounds__(128)
low_rank_decay_kernel(const float* low, int low_stride, int rank, const TW* __restrict__ a2,
                      const float* __restrict__ bias, float inv_tau, int rows, int n, float* __restrict__ out) {
    __shared__ float ls[LD_RANK][LD_TOKENS];
    const int t0 = blockIdx.y * LD_TOKENS, nt = min(LD_TOKENS, rows - t0);
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const TW* wr = a2 + (size_t)min(c, n - 1) * rank;
    float acc[LD_TOKENS];
#pragma unroll
    for (int i = 0; i < LD_TOKENS; ++i) acc[i] = 0.0f;
    for (int r0 = 0; r0 < rank; r0 += LD_RANK) {
        const int nr = min(LD_RANK, rank - r0);
        __syncthreads();
        for (int e = threadIdx.x; e < LD_TOKENS * LD_RANK; e += blockDim.x) {
            const int i = e / LD_RANK, r = e % LD_RANK;
            ls[r][i] = i < nt && r < nr ? low[(size_t)(t0 + i) * low_stride + r0 + r] : 0.0f;
        }
        __syncthreads();
#pragma unroll 8
        for (int r = 0; r < nr; ++r) {
            const float w = to_f32(wr[r0 + r]);
#pragma unroll
            for (int i = 0; i < LD_TOKENS; i += 4) {
                const float4 x = *reinterpret_cast<const float4*>(&ls[r][i]);
                acc[i] = fmaf(x.x, w, acc[i]);
                acc[i + 1] = fmaf(x.y, w, acc[i + 1]);
                acc[i + 2] = fmaf(x.z, w, acc[i + 2]);
                acc[i + 3] = fmaf(x.w, w, acc[i + 3]);
            }
        }
    }
    if (c >= n) return;
    const float b = bias[c];
#pragma unroll
    for (int i = 0; i < LD_TOKENS; ++i) {
        if (i >= nt) break;
        const float z = acc[i] + b;
        const float log_sigmoid = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
        out[(size_t)(t0 + i) * n + c] = expf(log_sigmoid * inv_tau);
    }
}

// ---- the recurrence ---------------------------------------------------------------------------------
struct Channel { float br, bi, log_decay, by; };

__device__ __forceinline__ float sigmoidf_(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }

// (a, b) of S <- a S + b for one token: a = e^l, b = sqrt(1 - a^2) i u, both from e^l - 1 (1 - a^2 = -e (2 + e) keeps its
// digits where a is near 1)
__device__ __forceinline__ float2 gate_pair(const Channel& p, float zr, float zi, float u) {
    const float e = expm1f(p.log_decay * sigmoidf_(zr + p.br));
    return make_float2(1.0f + e, sqrtf(-e * (2.0f + e)) * sigmoidf_(zi + p.bi) * u);
}

// gelu(z), the tanh form: 1/2 (1 + tanh x) = sigmoid(2 x)
__device__ __forceinline__ float gelu_gate(float z) {
    return z * sigmoidf_(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));
}

struct RecurrenceArgs {
    const float* u; int u_stride;
    const float* gates; long long gates_stride, gates_block;   // zr of part b at gates + b * gates_block + t * gates_stride, zi `per` further
    const float* y; int y_stride;
    const float* gate_bias;                                    // [2][width]
    const float* log_decay; const float* y_bias;               // [width]
    int per, width;                                            // channels of a part, of all
    const int* cu_q; const int* slots;
    float* state; long long state_stride;
};

__device__ __forceinline__ Channel channel_of(const RecurrenceArgs& p, int c) {
    return {p.gate_bias[c], p.gate_bias[p.width + c], p.log_decay[c], p.y_bias[c]};
}

// CH channels a block; a warp's lanes are CH channels of 32 / CH neighbouring tokens
constexpr int GR_WARPS = 16, GR_ROWS = 4, GR_BATCH = 12;
template <int CH> struct RecurrenceTile {
    static constexpr int tokens_at_once = 32 / CH;
    static constexpr int tokens_warp = GR_ROWS * tokens_at_once;
    static constexpr int tokens = (GR_WARPS - 1) * tokens_warp;             // 60 x 32 / CH
    static_assert(tokens % GR_BATCH == 0, "whole batches of the walk");
};

template <typename TO, int CH>
__global__ void __launch_bounds__(GR_WARPS * 32)
gated_recurrence_kernel(const RecurrenceArgs p, TO* __restrict__ out) {
    using Tile = RecurrenceTile<CH>;
    constexpr int TT = Tile::tokens;
    __shared__ float2 ab[2][TT][CH];
    __shared__ float ss[2][TT][CH];
    const int req = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = p.cu_q[req], t1 = p.cu_q[req + 1];
    if (t0 >= t1) return;
    const int j = lane % CH, c = blockIdx.y * CH + j;
    const bool live = c < p.width;
    const int cc = live ? c : p.width - 1;                // lanes past the width read the last channel and store nothing
    const Channel ch = channel_of(p, cc);
    const float* gp = p.gates + (size_t)(cc / p.per) * p.gates_block + cc % p.per;
    const float* up = p.u + cc;
    const float* yp = p.y + cc;
    const int tiles = (t1 - t0 + TT - 1) / TT;
    const int row0 = (warp - 1) * Tile::tokens_warp + lane / CH;            // this lane's first token of a tile (warps 1 to 15)
    float* slot = p.state + (size_t)p.slots[req] * p.state_stride + cc;

    float zr[GR_ROWS], zi[GR_ROWS], u[GR_ROWS], y[GR_ROWS], y_next[GR_ROWS];
    auto row = [&](int i) { return row0 + i * Tile::tokens_at_once; };
    auto fetch = [&](int tile) {                          // the inputs of a tile's (a, b), on their way
#pragma unroll
        for (int i = 0; i < GR_ROWS; ++i) {
            const int t = t0 + tile * TT + row(i);
            const bool in = t < t1;
            const float* g = gp + (size_t)(in ? t : t0) * p.gates_stride;
            zr[i] = g[0];
            zi[i] = g[p.per];
            u[i] = up[(size_t)(in ? t : t0) * p.u_stride];
        }
    };
    auto fetch_y = [&](int tile, float (&dst)[GR_ROWS]) {
#pragma unroll
        for (int i = 0; i < GR_ROWS; ++i) {
            const int t = t0 + tile * TT + row(i);
            dst[i] = yp[(size_t)(t < t1 ? t : t0) * p.y_stride];
        }
    };
    auto prepare = [&](int buf) {
#pragma unroll
        for (int i = 0; i < GR_ROWS; ++i) ab[buf][row(i)][j] = gate_pair(ch, zr[i], zi[i], u[i]);
    };
    auto finish = [&](int tile) {
#pragma unroll
        for (int i = 0; i < GR_ROWS; ++i) {
            const int t = t0 + tile * TT + row(i);
            if (t < t1 && live)
                out[(size_t)t * p.width + c] = from_f32<TO>(ss[tile & 1][row(i)][j] * gelu_gate(y[i] + ch.by));
        }
    };
    float S = 0.0f;
    if (warp == 0) {
        S = *slot;
    } else {
        fetch(0);
        prepare(0);
        if (tiles > 1) fetch(1);
        fetch_y(0, y);
    }
    __syncthreads();
    for (int tile = 0; tile < tiles; ++tile) {
        if (warp == 0) {
            if (lane < CH) {
                const int nt = min(TT, t1 - t0 - tile * TT);
                const float2 (*from)[CH] = ab[tile & 1];
                float (*to)[CH] = ss[tile & 1];
                int i = 0;
                for (; i + GR_BATCH <= nt; i += GR_BATCH) {        // a batch's pairs first: the chain then waits for itself alone
                    float2 v[GR_BATCH];
#pragma unroll
                    for (int b = 0; b < GR_BATCH; ++b) v[b] = from[i + b][j];
#pragma unroll
                    for (int b = 0; b < GR_BATCH; ++b) {
                        S = fmaf(v[b].x, S, v[b].y);
                        to[i + b][j] = S;
                    }
                }
                for (; i < nt; ++i) {
                    const float2 v = from[i][j];
                    S = fmaf(v.x, S, v.y);
                    to[i][j] = S;
                }
            }
        } else {
            if (tile > 0) fetch_y(tile, y_next);
            if (tile + 1 < tiles) prepare((tile + 1) & 1);
            if (tile + 2 < tiles) fetch(tile + 2);
            if (tile > 0) {
                finish(tile - 1);
#pragma unroll
                for (int i = 0; i < GR_ROWS; ++i) y[i] = y_next[i];
            }
        }
        __syncthreads();
    }
    if (warp == 0) {
        if (live && lane < CH) *slot = S;
    } else {
        finish(tiles - 1);
    }
}

// ---- one token a request, with the block-diagonal products -------------------------------------------
constexpr int GS_CHANNELS = 16;

template <typename TW, int VEC> __device__ __forceinline__ void load_weights(const TW* p, float (&w)[4]);
template <> __device__ __forceinline__ void load_weights<bf16, 4>(const bf16* p, float (&w)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x);
    const __nv_bfloat162 hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    w[0] = __bfloat162float(lo.x); w[1] = __bfloat162float(lo.y);
    w[2] = __bfloat162float(hi.x); w[3] = __bfloat162float(hi.y);
}
template <> __device__ __forceinline__ void load_weights<float, 4>(const float* p, float (&w)[4]) {
    const float4 raw = *reinterpret_cast<const float4*>(p);
    w[0] = raw.x; w[1] = raw.y; w[2] = raw.z; w[3] = raw.w;
}

// Requests req0 .. req0 + NR of the step, whose token t has the index of its request (one token each).
// w: [parts][2 per][per], the rows of zr first.  A part's width must be a multiple of 4.
template <typename TW, typename TO, int NR>
__global__ void __launch_bounds__(256)
gated_recurrence_single_kernel(const RecurrenceArgs p, const TW* __restrict__ w, int requests, TO* __restrict__ out) {
    extern __shared__ __align__(16) float us[];            // [NR][per]
    __shared__ float z[2 * GS_CHANNELS][NR + 1];
    const int slices = (p.per + GS_CHANNELS - 1) / GS_CHANNELS;
    const int part = blockIdx.x / slices, c0 = blockIdx.x % slices * GS_CHANNELS;      // first channel inside the part
    const int req0 = blockIdx.y * NR, nr = min(NR, requests - req0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const TW* wp = w + (size_t)part * 2 * p.per * p.per;
    // this warp's four rows: channels c0 + 2 warp, + 1 of zr, then of zi (past the part: its last row)
    const TW* rows[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) rows[i] = wp + (size_t)((i >> 1) * p.per + min(c0 + 2 * warp + (i & 1), p.per - 1)) * p.per;
    for (int e = threadIdx.x; e < NR * (p.per / 4); e += 256) {
        const int r = e / (p.per / 4), k = e % (p.per / 4) * 4;
        float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (r < nr) {
            const float* src = p.u + (size_t)p.cu_q[req0 + r] * p.u_stride + (size_t)part * p.per + k;
            x = make_float4(src[0], src[1], src[2], src[3]);
        }
        *reinterpret_cast<float4*>(us + (size_t)r * p.per + k) = x;
    }
    __syncthreads();
    float acc[4 * NR];
#pragma unroll
    for (int i = 0; i < 4 * NR; ++i) acc[i] = 0.0f;
#pragma unroll 2
    for (int k = lane * 4; k < p.per; k += 128) {
        float wv[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) load_weights<TW, 4>(rows[i] + k, wv[i]);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
            const float4 x = *reinterpret_cast<const float4*>(us + (size_t)r * p.per + k);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                float& a = acc[i * NR + r];
                a = fmaf(x.x, wv[i][0], a);
                a = fmaf(x.y, wv[i][1], a);
                a = fmaf(x.z, wv[i][2], a);
                a = fmaf(x.w, wv[i][3], a);
            }
        }
    }
    // halve the sums a lane holds at every exchange: at the end lane l has sums l * NR / 8 .. of the warp's 4 NR
#pragma unroll
    for (int o = 16, held = 2 * NR; o > 0; o >>= 1, held >>= 1) {
#pragma unroll
        for (int i = 0; i < 2 * NR; ++i) {
            if (i >= held) break;
            const bool upper = lane & o;
            const float send = upper ? acc[i] : acc[i + held];
            const float keep = upper ? acc[i + held] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
#pragma unroll
    for (int i = 0; i < NR / 8; ++i) {
        const int at = lane * (NR / 8) + i, row = at / NR, r = at % NR;
        z[(row >> 1) * GS_CHANNELS + 2 * warp + (row & 1)][r] = acc[i];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < NR * GS_CHANNELS; e += 256) {
        const int r = e / GS_CHANNELS, i = e % GS_CHANNELS;
        if (r >= nr || c0 + i >= p.per) continue;
        const int c = part * p.per + c0 + i, req = req0 + r, t = p.cu_q[req];
        const Channel ch = channel_of(p, c);
        float* slot = p.state + (size_t)p.slots[req] * p.state_stride + c;
        const float2 v = gate_pair(ch, z[i][r], z[GS_CHANNELS + i][r], us[(size_t)r * p.per + c0 + i]);
        const float S = fmaf(v.x, *slot, v.y);
        *slot = S;
        out[(size_t)t * p.width + c] = from_f32<TO>(S * gelu_gate(p.y[(size_t)t * p.y_stride + c] + ch.by));
    }
}

// x [rows][width] as three bfloat16 rows that add up to it: out[part][row][3][per] (`rows_padded` rows a part)
__global__ void __launch_bounds__(256)
split_rows_kernel(const float* x, int stride, int rows, int width, int per, int rows_padded, bf16* __restrict__ out) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;      // four neighbouring columns
    const int quads = width / 4;
    if (i >= (size_t)rows * quads) return;
    const int t = (int)(i / quads), c = (int)(i % quads) * 4, part = c / per;
    const float* src = x + (size_t)t * stride + c;
    bf16* dst = out + ((size_t)part * rows_padded + t) * 3 * per + (c - part * per);
    float v[4] = {src[0], src[1], src[2], src[3]};
#pragma unroll
    for (int s = 0; s < 3; ++s) {
        bf16 b[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            b[j] = __float2bfloat16_rn(v[j]);
            v[j] -= __bfloat162float(b[j]);
        }
        uint2 raw;
        __nv_bfloat162 lo(b[0], b[1]), hi(b[2], b[3]);
        raw.x = *reinterpret_cast<unsigned*>(&lo);
        raw.y = *reinterpret_cast<unsigned*>(&hi);
        *reinterpret_cast<uint2*>(dst + (size_t)s * per) = raw;
    }
}

RecurrenceArgs recurrence_args(const float* u, int u_stride, const float* gates, long long gates_stride,
                               long long gates_block, const float* y, int y_stride, const float* gate_bias, int per,
                               const float* log_decay, const float* y_bias, const int* cu_q, const int* slots, int width,
                               float* state, long long state_stride) {
    RecurrenceArgs a;
    a.u = u; a.u_stride = u_stride; a.gates = gates; a.gates_stride = gates_stride; a.gates_block = gates_block;
    a.y = y; a.y_stride = y_stride; a.gate_bias = gate_bias; a.log_decay = log_decay; a.y_bias = y_bias;
    a.per = per; a.width = width; a.cu_q = cu_q; a.slots = slots; a.state = state; a.state_stride = state_stride;
    return a;
}

}  // namespace

extern "C" int ti_low_rank_decay(const float* low, int low_stride, int rank, const void* a2, int a2_dtype,
                                 const float* bias, float inv_tau, int rows, int n, float* out, void* stream) {
    if (rows == 0 || n == 0) return 0;
    TI_REQUIRE(rank >= 1, "low_rank_decay: inner width %d", rank);
    const dim3 grid((n + 127) / 128, (rows + LD_TOKENS - 1) / LD_TOKENS);
    TI_REQUIRE(grid.y <= 65535, "low_rank_decay: %d rows exceed the grid limit", rows);
    cudaStream_t s = (cudaStream_t)stream;
    if (a2_dtype == TI_BF16)
        low_rank_decay_kernel<bf16><<<grid, 128, 0, s>>>(low, low_stride, rank, (const bf16*)a2, bias, inv_tau, rows, n, out);
    else if (a2_dtype == TI_F32)
        low_rank_decay_kernel<float><<<grid, 128, 0, s>>>(low, low_stride, rank, (const float*)a2, bias, inv_tau, rows, n, out);
    else return ti_fail("low_rank_decay: matrix dtype code %d", a2_dtype);
    return ti_check_launch("low_rank_decay");
}

// gates: part b's zr columns of token t at gates + b * gates_block + t * gates_stride, its zi columns `per` further.
extern "C" int ti_gated_recurrence(const float* u, int u_stride, const float* gates, long long gates_stride,
                                   long long gates_block, const float* y, int y_stride, const float* gate_bias, int per,
                                   const float* log_decay, const float* y_bias, const int* cu_q, const int* slots,
                                   int requests, int width, float* state, long long state_stride, void* out,
                                   int out_dtype, void* stream) {
    if (requests == 0 || width == 0) return 0;
    TI_REQUIRE(per >= 1 && width % per == 0, "gated_recurrence: %d channels in parts of %d", width, per);
    const RecurrenceArgs a = recurrence_args(u, u_stride, gates, gates_stride, gates_block, y, y_stride, gate_bias, per,
                                             log_decay, y_bias, cu_q, slots, width, state, state_stride);
    int device = 0, sms = 0;
    cudaGetDevice(&device);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
    // few blocks: fewer channels each, so that more SMs share the gates' exponentials (the bits do not depend on it)
    int ch = 32;
    while (ch > 8 && (long long)requests * ((width + ch / 2 - 1) / (ch / 2)) <= 2LL * sms) ch /= 2;
    const dim3 grid(requests, (width + ch - 1) / ch);
    TI_REQUIRE(grid.y <= 65535, "gated_recurrence: %d channels", width);
    TI_REQUIRE(out_dtype == TI_BF16 || out_dtype == TI_F32, "gated_recurrence: output dtype code %d", out_dtype);
    cudaStream_t s = (cudaStream_t)stream;
#define CALL(CH)                                                                                                     \
    do {                                                                                                             \
        if (out_dtype == TI_BF16) gated_recurrence_kernel<bf16, CH><<<grid, GR_WARPS * 32, 0, s>>>(a, (bf16*)out);     \
        else gated_recurrence_kernel<float, CH><<<grid, GR_WARPS * 32, 0, s>>>(a, (float*)out);                        \
    } while (0)
    if (ch == 32) CALL(32);
    else if (ch == 16) CALL(16);
    else CALL(8);
#undef CALL
    return ti_check_launch("gated_recurrence");
}

// Requests a block takes, and the widest part whose inputs fit the 48 KB of shared memory for eight of them.
extern "C" int ti_gated_recurrence_single_supported(int per) { return per >= 4 && per % 4 == 0 && per * 8 * 4 <= 40 * 1024; }

extern "C" int ti_gated_recurrence_single(const float* u, int u_stride, const void* w, int w_dtype, const float* y,
                                          int y_stride, const float* gate_bias, int per, const float* log_decay,
                                          const float* y_bias, const int* cu_q, const int* slots, int requests,
                                          int width, float* state, long long state_stride, void* out, int out_dtype,
                                          void* stream) {
    if (requests == 0 || width == 0) return 0;
    TI_REQUIRE(width % per == 0 && ti_gated_recurrence_single_supported(per),
               "gated_recurrence_single: %d channels in parts of %d (a multiple of 4, at most 1,280)", width, per);
    TI_REQUIRE((uintptr_t)w % 16 == 0, "gated_recurrence_single: weights must be 16-byte aligned");
    const RecurrenceArgs a = recurrence_args(u, u_stride, nullptr, 0, 0, y, y_stride, gate_bias, per, log_decay, y_bias,
                                             cu_q, slots, width, state, state_stride);
    const int slices = (per + GS_CHANNELS - 1) / GS_CHANNELS;
    const bool wide = requests > 8 && per * 16 * 4 <= 40 * 1024;
    const int nr = wide ? 16 : 8;
    const dim3 grid(width / per * slices, (requests + nr - 1) / nr);
    TI_REQUIRE(grid.y <= 65535, "gated_recurrence_single: %d requests", requests);
    const size_t smem = (size_t)nr * per * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
#define CALL(TW, TO)                                                                                                 \
    do {                                                                                                             \
        if (wide) gated_recurrence_single_kernel<TW, TO, 16><<<grid, 256, smem, s>>>(a, (const TW*)w, requests, (TO*)out); \
        else gated_recurrence_single_kernel<TW, TO, 8><<<grid, 256, smem, s>>>(a, (const TW*)w, requests, (TO*)out); \
    } while (0)
    if (w_dtype == TI_BF16 && out_dtype == TI_BF16) CALL(bf16, bf16);
    else if (w_dtype == TI_BF16 && out_dtype == TI_F32) CALL(bf16, float);
    else if (w_dtype == TI_F32 && out_dtype == TI_BF16) CALL(float, bf16);
    else if (w_dtype == TI_F32 && out_dtype == TI_F32) CALL(float, float);
    else return ti_fail("gated_recurrence_single: dtype codes w=%d out=%d", w_dtype, out_dtype);
#undef CALL
    return ti_check_launch("gated_recurrence_single");
}

extern "C" int ti_split_rows(const float* x, int stride, int rows, int width, int per, int rows_padded, void* out,
                             void* stream) {
    if (rows == 0 || width == 0) return 0;
    TI_REQUIRE(per % 4 == 0 && width % per == 0 && rows <= rows_padded && (uintptr_t)out % 8 == 0,
               "split_rows: parts of %d columns (a multiple of 4) of %d", per, width);
    const long long quads = (long long)rows * (width / 4);
    split_rows_kernel<<<(unsigned)((quads + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, stride, rows, width, per,
                                                                                         rows_padded, (bf16*)out);
    return ti_check_launch("split_rows");
}
