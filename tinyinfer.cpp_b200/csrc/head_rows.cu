// The heads of an attention on their way from a product's float32 row to the kernels that read them.
//
// heads_prepare_store: from rows with the columns [queries | keys | values] and an optional bias per column, each
// query and key head by itself
//    x = head + bias;  x = x / sqrt(mean(x^2) + eps) * weight          (`pre_norm`; weight [dk], shared by the heads)
//    the first `rot` elements turned by the token's position           (neighbouring pairs, or i with i + rot/2;
//                                                                        cosine and sine times `mag`)
//    x = x / sqrt(mean(x^2) + eps)                                      (`post_norm`)
//    queries: x *= 1 + temp_coef * ln(floor((position + 1) / temp_every) + 1)      (temp_every > 0)
// then keys and values go into the token's page and queries into q_out.  `values_from_keys`: there are no value
// columns, a value head is the key head's columns (with their bias) as they are; dv = dk.
//
// A block takes one token, whose cosines and sines it makes once, and a share of its heads; a head belongs to 8, 16 or
// 32 lanes of a warp, which hold it in registers as units of four elements (two pairs), so it is read once.  Sizes
// that do not fall into such units take a kernel with a warp per head and a pass per norm.  All arithmetic is
// float32; a head's bits depend on its row alone.
#include "common.cuh"

namespace {

constexpr int THREADS = 256;
enum { TI_ERR_BAD_PAGE = 1 };
enum { ITEM_QUERY = 0, ITEM_KEY = 1, ITEM_VALUE = 2 };

struct Heads {
    const float* proj; int stride;                    // rows of the step, written by the kernel before this one
    const float* bias; const float* q_weight; const float* k_weight;
    int pre_norm, post_norm; float eps;
    const float* inv_freq; int rot, halves; float mag;
    float temp_coef; int temp_every; int values_from_keys;
    const int* positions; const int* req_of_tok; const int* block_table; int bt_stride;
    int num_pages, page_size, write_kv, num_heads, num_kv_heads, dk, dv;
};

// item: a query head, then, where the cache is written, the key heads and the value heads
struct Item { int kind, head, n, column; };
__device__ __forceinline__ Item item_of(const Heads& p, int i) {
    const int nq = p.num_heads * p.dk, nk = p.num_kv_heads * p.dk;
    if (i < p.num_heads) return {ITEM_QUERY, i, p.dk, i * p.dk};
    i -= p.num_heads;
    if (i < p.num_kv_heads) return {ITEM_KEY, i, p.dk, nq + i * p.dk};
    i -= p.num_kv_heads;
    return {ITEM_VALUE, i, p.dv, p.values_from_keys ? nq + i * p.dk : nq + nk + i * p.dv};
}

__device__ __forceinline__ void fill_table(float2* cs, const Heads& p, float pos) {
    for (int i = threadIdx.x; i < p.rot >> 1; i += blockDim.x) {
        float s, c;
        sincosf(pos * p.inv_freq[i], &s, &c);
        cs[i] = make_float2(c * p.mag, s * p.mag);
    }
}
__device__ __forceinline__ float query_factor(const Heads& p, int pos) {
    return p.temp_every > 0 ? fmaf(p.temp_coef, logf((float)((pos + 1) / p.temp_every + 1)), 1.0f) : 1.0f;
}
// where an item's head starts in q_out or in the token's page (null: nowhere)
template <typename TQ, typename TC>
__device__ __forceinline__ TC* page_head(const Heads& p, const Item& it, TC* page, int slot) {
    TC* base = page + (it.kind == ITEM_VALUE ? (size_t)p.num_kv_heads * p.page_size * p.dk : 0);
    return base + ((size_t)it.head * p.page_size + slot) * it.n;
}
template <typename TC>
__device__ __forceinline__ TC* token_page(const Heads& p, int t, int pos, TC* pages, int* status) {
    const int page = p.block_table[(size_t)p.req_of_tok[t] * p.bt_stride + pos / p.page_size];
    if (page < 0 || page >= p.num_pages) {
        if (threadIdx.x == 0) atomicCAS(status, 0, TI_ERR_BAD_PAGE);
        return nullptr;
    }
    return pages + (size_t)page * p.num_kv_heads * p.page_size * (p.dk + p.dv);
}

template <int LANES> __device__ __forceinline__ float group_sum(float v) {
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Unit u of a head: elements (x0, y0) and (x1, y1) are the pairs of the turn, or four neighbours outside of it.
__device__ __forceinline__ float4 load_unit(const float* p, int u, bool turned, int halves, int half) {
    if (turned && halves) {
        const float2 x = *reinterpret_cast<const float2*>(p + 2 * u), y = *reinterpret_cast<const float2*>(p + 2 * u + half);
        return make_float4(x.x, x.y, y.x, y.y);
    }
    const float4 v = *reinterpret_cast<const float4*>(p + 4 * u);
    return turned ? make_float4(v.x, v.z, v.y, v.w) : v;
}
template <typename T> __device__ __forceinline__ void store2(T* p, float a, float b) {
    if constexpr (sizeof(T) == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
    else *reinterpret_cast<float2*>(p) = make_float2(a, b);
}
template <typename T>
__device__ __forceinline__ void store_unit(T* p, int u, bool turned, int halves, int half, float4 v) {
    if (turned && halves) {
        store2<T>(p + 2 * u, v.x, v.y);
        store2<T>(p + 2 * u + half, v.z, v.w);
        return;
    }
    if (turned) v = make_float4(v.x, v.z, v.y, v.w);
    if constexpr (sizeof(T) == 2) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        *reinterpret_cast<uint2*>(p + 4 * u) = make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
    } else {
        *reinterpret_cast<float4*>(p + 4 * u) = v;
    }
}
__device__ __forceinline__ float squares(float4 v) { return fmaf(v.w, v.w, fmaf(v.z, v.z, fmaf(v.y, v.y, v.x * v.x))); }
__device__ __forceinline__ void times(float4& v, float f) { v.x *= f; v.y *= f; v.z *= f; v.w *= f; }

// What a head of KIND goes through between its row and its destination.  LANES lanes hold it, NU units a lane.
template <int KIND, int LANES, int NU, typename T>
__device__ __forceinline__ void prepare_head(const Heads& p, const float* row, int column, const float2* cs, float factor,
                                             int lane, bool live, T* dst) {
    const int n = KIND == ITEM_VALUE ? p.dv : p.dk;
    const int units = n >> 2, turned_units = KIND == ITEM_VALUE ? 0 : p.rot >> 2, half = p.rot >> 1;
    const float* src = row + column;
    float4 v[NU];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < NU; ++j) {
        const int u = lane + LANES * j;
        v[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (!live || u >= units) continue;
        const bool turned = u < turned_units;
        v[j] = load_unit(src, u, turned, p.halves, half);
        if (p.bias) {
            const float4 b = load_unit(p.bias + column, u, turned, p.halves, half);
            v[j].x += b.x; v[j].y += b.y; v[j].z += b.z; v[j].w += b.w;
        }
        if (KIND != ITEM_VALUE) ss += squares(v[j]);
    }
    if (KIND != ITEM_VALUE) {
        const float mean_of = 1.0f / (float)n;
        float last = KIND == ITEM_QUERY ? factor : 1.0f;
        if (p.pre_norm) {
            const float inv = rsqrtf(fmaf(group_sum<LANES>(ss), mean_of, p.eps));
            const float* w = KIND == ITEM_QUERY ? p.q_weight : p.k_weight;
            if (w) {
#pragma unroll
                for (int j = 0; j < NU; ++j) {
                    const int u = lane + LANES * j;
                    if (u >= units) continue;
                    const float4 g = load_unit(w, u, u < turned_units, p.halves, half);
                    v[j].x *= inv * g.x; v[j].y *= inv * g.y; v[j].z *= inv * g.z; v[j].w *= inv * g.w;
                }
            } else {
#pragma unroll
                for (int j = 0; j < NU; ++j) times(v[j], inv);
            }
        }
#pragma unroll
        for (int j = 0; j < NU; ++j) {
            const int u = lane + LANES * j;
            if (u >= turned_units) continue;
            const float4 f = *reinterpret_cast<const float4*>(cs + 2 * u);     // two pairs' (cosine, sine)
            v[j] = make_float4(v[j].x * f.x - v[j].z * f.y, v[j].y * f.z - v[j].w * f.w,
                               v[j].z * f.x + v[j].x * f.y, v[j].w * f.z + v[j].y * f.w);
        }
        if (p.post_norm) {
            float sq = 0.0f;
#pragma unroll
            for (int j = 0; j < NU; ++j) sq += squares(v[j]);
            last *= rsqrtf(fmaf(group_sum<LANES>(sq), mean_of, p.eps));
        }
#pragma unroll
        for (int j = 0; j < NU; ++j) times(v[j], last);
    }
    if (!live || dst == nullptr) return;
#pragma unroll
    for (int j = 0; j < NU; ++j) {
        const int u = lane + LANES * j;
        if (u < units) store_unit<T>(dst, u, u < turned_units, p.halves, half, v[j]);
    }
}

// LANES lanes of a warp a head, NU units a lane
template <typename TQ, typename TC, int LANES, int NU>
__global__ void __launch_bounds__(THREADS)
heads_prepare_store_kernel(const Heads p, TC* __restrict__ pages, TQ* __restrict__ q_out, int* __restrict__ status) {
    extern __shared__ __align__(16) float2 cs[];
    const int t = blockIdx.x, pos = p.positions[t];
    pdl_launch();
    fill_table(cs, p, (float)pos);                        // of the step's positions: before the wait
    const float factor = query_factor(p, pos);
    TC* page = p.write_kv ? token_page(p, t, pos, pages, status) : nullptr;
    __syncthreads();
    pdl_wait();
    const float* row = p.proj + (size_t)t * p.stride;
    const int slot = pos % p.page_size, nq = p.num_heads * p.dk, nk = p.num_kv_heads * p.dk;
    constexpr int PER_BLOCK = THREADS / LANES;
    const int lane = threadIdx.x % LANES, mine = blockIdx.y * PER_BLOCK + threadIdx.x / LANES, step = gridDim.y * PER_BLOCK;
    const int items = p.num_heads + (p.write_kv ? 2 * p.num_kv_heads : 0);
    // a warp's groups walk on together (they sum in groups): queries, then keys, then values; `at` counts through all
    const int warp_first = mine - (threadIdx.x % 32) / LANES;
    for (int first = warp_first, at = mine; first < items; first += step, at += step) {
        // a warp that holds heads of two kinds takes each kind's path once
        const int last = first + 32 / LANES - 1, k0 = p.num_heads, v0 = p.num_heads + p.num_kv_heads;
        if (first < k0) {
            const bool live = at < k0;
            prepare_head<ITEM_QUERY, LANES, NU, TQ>(p, row, at * p.dk, cs, factor, lane, live,
                                                    q_out + ((size_t)t * p.num_heads + at) * p.dk);
        }
        if (!p.write_kv) continue;
        if (last >= k0 && first < v0) {
            const bool live = at >= k0 && at < v0;
            const int g = at - k0;
            prepare_head<ITEM_KEY, LANES, NU, TC>(p, row, nq + g * p.dk, cs, factor, lane, live,
                                                  page ? page + ((size_t)g * p.page_size + slot) * p.dk : nullptr);
        }
        if (last >= v0) {
            const bool live = at >= v0 && at < items;
            const int g = at - v0;
            TC* base = page ? page + (size_t)p.num_kv_heads * p.page_size * p.dk : nullptr;
            prepare_head<ITEM_VALUE, LANES, NU, TC>(p, row, p.values_from_keys ? nq + g * p.dk : nq + nk + g * p.dv, cs, factor,
                                                    lane, live, base ? base + ((size_t)g * p.page_size + slot) * p.dv : nullptr);
        }
    }
}

// any sizes: a warp a head, an element a lane at a time, the head read again for every pass
template <typename TQ, typename TC>
__global__ void __launch_bounds__(THREADS)
heads_prepare_any_kernel(const Heads p, TC* __restrict__ pages, TQ* __restrict__ q_out, int* __restrict__ status) {
    extern __shared__ float2 cs[];
    const int t = blockIdx.x, pos = p.positions[t];
    pdl_launch();
    fill_table(cs, p, (float)pos);
    const float factor = query_factor(p, pos);
    TC* page = p.write_kv ? token_page(p, t, pos, pages, status) : nullptr;
    __syncthreads();
    pdl_wait();
    const float* row = p.proj + (size_t)t * p.stride;
    const int half = p.rot >> 1, slot = pos % p.page_size, lane = threadIdx.x & 31;
    const int items = p.num_heads + (p.write_kv ? 2 * p.num_kv_heads : 0);
    for (int at = threadIdx.x >> 5; at < items; at += THREADS / 32) {
        const Item it = item_of(p, at);
        const bool value = it.kind == ITEM_VALUE;
        const int rot = value ? 0 : p.rot;
        const float* w = value || !p.pre_norm ? nullptr : it.kind == ITEM_QUERY ? p.q_weight : p.k_weight;
        auto raw = [&](int e) { return row[it.column + e] + (p.bias ? p.bias[it.column + e] : 0.0f); };
        float inv = 1.0f;
        if (p.pre_norm && !value) {
            float ss = 0.0f;
            for (int e = lane; e < it.n; e += 32) ss = fmaf(raw(e), raw(e), ss);
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)it.n + p.eps);
        }
        auto normed = [&](int e) { return w ? raw(e) * inv * w[e] : raw(e) * inv; };
        auto turned = [&](int e) {
            if (e >= rot) return normed(e);
            const bool first = p.halves ? e < half : (e & 1) == 0;
            const int other = p.halves ? (first ? e + half : e - half) : (e ^ 1);
            const float2 f = cs[p.halves ? (first ? e : other) : e >> 1];
            return first ? normed(e) * f.x - normed(other) * f.y : normed(e) * f.x + normed(other) * f.y;
        };
        float last = it.kind == ITEM_QUERY ? factor : 1.0f;
        if (p.post_norm && !value) {
            float ss = 0.0f;
            for (int e = lane; e < it.n; e += 32) { const float y = turned(e); ss = fmaf(y, y, ss); }
            last *= 1.0f / sqrtf(warp_sum(ss) / (float)it.n + p.eps);
        }
        if (it.kind != ITEM_QUERY && page == nullptr) continue;
        if (it.kind == ITEM_QUERY) {
            TQ* dst = q_out + ((size_t)t * p.num_heads + it.head) * p.dk;
            for (int e = lane; e < it.n; e += 32) dst[e] = from_f32<TQ>(turned(e) * last);
        } else {
            TC* dst = page_head<TQ, TC>(p, it, page, slot);
            for (int e = lane; e < it.n; e += 32) dst[e] = from_f32<TC>(turned(e) * last);
        }
    }
}

bool multiple16(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace

extern "C" int ti_heads_prepare_store(const float* proj, int stride, const float* bias, const float* q_weight,
                                      const float* k_weight, int pre_norm, int post_norm, float eps,
                                      const float* inv_freq, int rot, int halves, float mag, float temp_coef,
                                      int temp_every, int values_from_keys, const int* positions,
                                      const int* req_of_tok, const int* block_table, int bt_stride, void* pages,
                                      int cache_dtype, int num_pages, int page_size, int write_kv, int num_tokens,
                                      int num_heads, int num_kv_heads, int dk, int dv, void* q_out, int q_dtype,
                                      int* status, void* stream) {
    if (num_tokens == 0) return 0;
    TI_REQUIRE(rot >= 0 && rot <= dk && rot % 2 == 0, "heads_prepare_store: rotated width %d must be even and at most "
               "the head size %d", rot, dk);
    TI_REQUIRE(rot == 0 || inv_freq != nullptr, "heads_prepare_store: a rotation needs its frequencies");
    TI_REQUIRE(!values_from_keys || dk == dv, "heads_prepare_store: values of %d elements from keys of %d", dv, dk);
    TI_REQUIRE(temp_every >= 0, "heads_prepare_store: a query factor that grows every %d positions", temp_every);
    const Heads p{proj, stride, bias, q_weight, k_weight, pre_norm, post_norm, eps, inv_freq, rot, halves, mag, temp_coef,
                  temp_every, values_from_keys, positions, req_of_tok, block_table, bt_stride, num_pages, page_size,
                  write_kv, num_heads, num_kv_heads, dk, dv};
    const size_t smem = (size_t)(rot / 2) * sizeof(float2);
    TI_REQUIRE(smem <= 48 * 1024, "heads_prepare_store: a rotated width of %d", rot);
    const int widest = dk > dv ? dk : dv;
    const bool units = dk % 4 == 0 && dv % 4 == 0 && rot % 4 == 0 && stride % 4 == 0 && widest <= 512 && multiple16(proj) &&
                       multiple16(bias) && multiple16(q_weight) && multiple16(k_weight) && multiple16(pages) &&
                       multiple16(q_out);
    int lanes = 8;
    while (lanes < 32 && lanes * 4 < widest) lanes *= 2;
    const int nu = (widest / 4 + 31) / 32;
    const int items = num_heads + (write_kv ? 2 * num_kv_heads : 0), per_block = THREADS / lanes;
    // few tokens: a token's heads over several blocks
    const int gy = num_tokens >= 256 ? 1 : (items + per_block - 1) / per_block;
    cudaStream_t s = (cudaStream_t)stream;
#define LAUNCH(TQ, TC, LANES, NU)                                                                                \
    ti_launch_pdl(heads_prepare_store_kernel<TQ, TC, LANES, NU>, dim3(num_tokens, gy), dim3(THREADS), smem, s, p,   \
                  (TC*)pages, (TQ*)q_out, status)
#define CALL(TQ, TC)                                                                                             \
    if (!units) ti_launch_pdl(heads_prepare_any_kernel<TQ, TC>, dim3(num_tokens), dim3(THREADS), smem, s, p,        \
                              (TC*)pages, (TQ*)q_out, status);                                                   \
    else if (lanes <= 8) LAUNCH(TQ, TC, 8, 1); else if (lanes <= 16) LAUNCH(TQ, TC, 16, 1);                       \
    else if (nu <= 1) LAUNCH(TQ, TC, 32, 1); else if (nu <= 2) LAUNCH(TQ, TC, 32, 2); else LAUNCH(TQ, TC, 32, 4)
    if (q_dtype == TI_F32 && cache_dtype == TI_F32) { CALL(float, float); }
    else if (q_dtype == TI_BF16 && cache_dtype == TI_BF16) { CALL(bf16, bf16); }
    else if (q_dtype == TI_F32 && cache_dtype == TI_BF16) { CALL(float, bf16); }
    else if (q_dtype == TI_BF16 && cache_dtype == TI_F32) { CALL(bf16, float); }
    else return ti_fail("heads_prepare_store: dtype codes queries=%d cache=%d are not supported", q_dtype, cache_dtype);
#undef CALL
#undef LAUNCH
    return ti_check_launch("heads_prepare_store");
}
