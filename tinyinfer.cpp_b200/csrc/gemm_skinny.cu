// Matrix product for few rows (M <= 64, the decode step): C[M,N] (+)= A[M,K] * W[N,K]^T, bfloat16
// operands, float32 accumulation.  The work is bound by reading W once from HBM.
//
// A block owns a strip of 16 rows of W (16 outputs per token).  Its 8 warps split K in chunks
// of 32 that they take in turn, so the block reads each W row in contiguous 512-byte pieces.
// Operands go straight from global memory into tensor-core fragments (mma.sync m16n8k16, W as
// the 16-row A operand, tokens as the 8-column B operand): a thread loads 16 bytes = 8
// consecutive k of one W row and of one token, and the contraction index inside a chunk is
// permuted identically for both operands, which a sum over k allows.  The 8 partial sums of a
// block are added in a fixed order in shared memory, so an output does not depend on M, on the
// other rows or on the launch.
//
// Epilogues: store, accumulate into C (the residual stream; optionally through a gate, C += scale
// sigmoid(gate + bias) * sum), or SwiGLU: W holds, in every strip,
// 8 gate rows followed by their 8 up rows, and out[m, j] = silu(gate_j) * up_j in bfloat16; or an activation of
// one value per output.
#include "common.cuh"
#include "glu.cuh"

namespace {

constexpr int WARPS = 8;
constexpr int STRIP = 16;
constexpr int CHUNK = 32;

enum { MODE_STORE = 0, MODE_ACCUMULATE = 1, MODE_SWIGLU = 2, MODE_XIELU = 3, MODE_UNARY = 4 };

__device__ __forceinline__ uint4 ld_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

__device__ __forceinline__ void mma_bf16(float (&c)[4], unsigned a0, unsigned a1, unsigned a2,
                                         unsigned a3, unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 "
                 "{%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// A second product over the same number of rows (with a k of its own) in the same launch: the blocks from `first_block`
// on (0: there is none) store its strips.  Two products of a decode step that depend on nothing of each other (a
// sublayer's first product and its gate) then wait for the kernel before them once.
struct SecondProduct { const bf16* a; const bf16* w; float* c; int n, k, lda, ldw, ldc; unsigned first_block; };

// ROWS = 16: a block owns 16 rows of W.  ROWS = 8: it owns 8 (the upper half of the MMA's A
// operand is zero), which doubles the number of blocks for narrow outputs.
constexpr int SHORT_K = WARPS * CHUNK * 4;     // what four chunks per warp cover: 1,024
// BATCH: chunks of W a warp has in flight.  4 covers K <= 1,024 in one round and leaves registers
// for three blocks per SM (384 blocks of a 6,144-row weight then run as one wave instead of 1.3).
// STORE_ONLY: the kernel without its other two epilogues (the QKV product of a small model's
// decode step, which waits for this kernel once a layer: the shorter the kernel the better).
template <int NT, int ROWS, int BATCH, bool STORE_ONLY = false>
__global__ void __launch_bounds__(WARPS * 32, BATCH == 4 && NT == 1 ? 3 : 2)
gemm_skinny_kernel(const bf16* a, const bf16* __restrict__ w, float* __restrict__ c,
                   bf16* __restrict__ out_act, int m, int n, int k, int lda, int ldw, int ldc,
                   int ld_act, int mode, int glu_kind, float act_p, float act_q, const AddGate add,
                   const SecondProduct second) {
    constexpr int MP = NT * 8;                                  // padded token count
    __shared__ float part[WARPS][ROWS][MP + 1];
    if (STORE_ONLY) mode = MODE_STORE;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, tq = lane & 3;
    int n0 = blockIdx.x * ROWS;
    if (second.first_block > 0 && blockIdx.x >= second.first_block) {      // the blocks of the second product
        n0 = (blockIdx.x - second.first_block) * ROWS;
        a = second.a; w = second.w; c = second.c;
        n = second.n; k = second.k; lda = second.lda; ldw = second.ldw; ldc = second.ldc;
        mode = MODE_STORE;
    }
    // rows past N are read from the last row and never stored
    const bf16* w_lo = w + (size_t)min(n0 + g, n - 1) * ldw + tq * 8;
    const bf16* w_hi = w + (size_t)min(n0 + g + 8, n - 1) * ldw + tq * 8;
    const bf16* a_row[NT];
#pragma unroll
    for (int j = 0; j < NT; ++j) a_row[j] = a + (size_t)min(j * 8 + g, m - 1) * lda + tq * 8;

    float acc[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;

    const int chunks = k / CHUNK;
    pdl_launch();
    for (int c0 = warp; c0 < chunks; c0 += WARPS * BATCH) {
        // all loads of the batch first: the product is bound by memory latency, not by arithmetic
        uint4 wl[BATCH], wh[BATCH];
#pragma unroll
        for (int u = 0; u < BATCH; ++u) {
            const int ch = c0 + u * WARPS;
            if (ch < chunks) {
                wl[u] = ld_stream(w_lo + (size_t)ch * CHUNK);
                if (ROWS == 16) wh[u] = ld_stream(w_hi + (size_t)ch * CHUNK);
            }
        }
        // the weights do not depend on the kernel before this one; the activations do
        if (c0 == warp) pdl_wait();
        if constexpr (NT * BATCH <= 16) {
            // few tokens: all activations of the batch are requested at once (one round trip to
            // L2 behind the wait instead of one per chunk)
            uint4 xr[BATCH][NT];
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const int ch = c0 + u * WARPS;
                if (ch < chunks) {
#pragma unroll
                    for (int j = 0; j < NT; ++j)
                        xr[u][j] = *reinterpret_cast<const uint4*>(a_row[j] + (size_t)ch * CHUNK);
                }
            }
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const int ch = c0 + u * WARPS;
                if (ch >= chunks) break;
                if (ROWS == 8) wh[u] = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    mma_bf16(acc[j], wl[u].x, wh[u].x, wl[u].y, wh[u].y, xr[u][j].x, xr[u][j].y);
                    mma_bf16(acc[j], wl[u].z, wh[u].z, wl[u].w, wh[u].w, xr[u][j].z, xr[u][j].w);
                }
            }
        } else {
#pragma unroll
            for (int u = 0; u < BATCH; ++u) {
                const int ch = c0 + u * WARPS;
                if (ch >= chunks) break;
                if (ROWS == 8) wh[u] = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
                for (int j = 0; j < NT; ++j) {
                    const uint4 x = *reinterpret_cast<const uint4*>(a_row[j] + (size_t)ch * CHUNK);
                    mma_bf16(acc[j], wl[u].x, wh[u].x, wl[u].y, wh[u].y, x.x, x.y);
                    mma_bf16(acc[j], wl[u].z, wh[u].z, wl[u].w, wh[u].w, x.z, x.w);
                }
            }
        }
    }
    // What this thread will add to, requested now: the reads return while the partial sums are
    // exchanged (read one by one between the stores below, each would wait a round trip to L2).
    constexpr int OUT_STEP = WARPS * 32 / ROWS;                 // tokens a pass of the block covers
    float old_c[8 * NT / OUT_STEP > 0 ? 8 * NT / OUT_STEP : 1];
    float gate_c[8 * NT / OUT_STEP > 0 ? 8 * NT / OUT_STEP : 1];
    if (mode == MODE_ACCUMULATE) {
        if (chunks <= warp) pdl_wait();
        const int i = threadIdx.x % ROWS;
#pragma unroll
        for (int it = 0; it < (int)(sizeof(old_c) / sizeof(float)); ++it) {
            const int tok = threadIdx.x / ROWS + it * OUT_STEP;
            old_c[it] = tok < m && n0 + i < n ? __ldcg(c + (size_t)tok * ldc + n0 + i) : 0.0f;
            gate_c[it] = add.gate && tok < m && n0 + i < n ? __ldcg(add.gate + (size_t)tok * add.ld + n0 + i) + add.bias[n0 + i] : 0.0f;
        }
    }
    // acc[j]: [0],[1] = W row g, tokens 8j + 2tq (+1); [2],[3] = W row g + 8
#pragma unroll
    for (int j = 0; j < NT; ++j) {
        part[warp][g][j * 8 + tq * 2] = acc[j][0];
        part[warp][g][j * 8 + tq * 2 + 1] = acc[j][1];
        if (ROWS == 16) {
            part[warp][g + 8][j * 8 + tq * 2] = acc[j][2];
            part[warp][g + 8][j * 8 + tq * 2 + 1] = acc[j][3];
        }
    }
    if (chunks <= warp) pdl_wait();                   // a warp without chunks still orders its writes
    __syncthreads();
    if (mode == MODE_SWIGLU) {
        if (ROWS == 16) {
            const int i = threadIdx.x & 7;                      // gate row i, up row i + 8
            const int col = blockIdx.x * 8 + i;
            for (int tok = threadIdx.x >> 3; tok < m; tok += WARPS * 4) {
                float gate = 0.0f, up = 0.0f;
#pragma unroll
                for (int wp = 0; wp < WARPS; ++wp) {
                    gate += part[wp][i][tok];
                    up += part[wp][(i + 8) % ROWS][tok];
                }
                const float y = glu_activation(glu_kind, gate, up, act_p, act_q);   // limit act_p, factor act_q
                if (n0 + i + 8 < n) out_act[(size_t)tok * ld_act + col] = __float2bfloat16_rn(y);
            }
        }
    } else {
        const int i = threadIdx.x % ROWS;
#pragma unroll
        for (int it = 0; it < (int)(sizeof(old_c) / sizeof(float)); ++it) {
            const int tok = threadIdx.x / ROWS + it * OUT_STEP;
            if (tok >= m) break;
            float sum = 0.0f;
#pragma unroll
            for (int wp = 0; wp < WARPS; ++wp) sum += part[wp][i][tok];
            if (mode == MODE_UNARY) {
                if (n0 + i < n) out_act[(size_t)tok * ld_act + n0 + i] = __float2bfloat16_rn(unary_activation(glu_kind, sum));
            } else if (mode == MODE_XIELU) {          // act_p z^2 + z/2 above zero, act_q (exp(z) - 1 - z) + z/2 below
                const float y = sum > 0.0f ? fmaf(act_p * sum, sum, 0.5f * sum) : fmaf(act_q, expm1f(sum) - sum, 0.5f * sum);
                if (n0 + i < n) out_act[(size_t)tok * ld_act + n0 + i] = __float2bfloat16_rn(y);
            } else if (n0 + i < n) {
                c[(size_t)tok * ldc + n0 + i] = mode == MODE_ACCUMULATE ? add_through(add, old_c[it], sum, gate_c[it], 0.0f) : sum;
            }
        }
    }
}

}  // namespace

extern "C" int ti_gemm_skinny_supported(int m, int n, int k, int lda, int ldw) {
    return m >= 1 && m <= 64 && n >= 1 && k >= CHUNK && k % CHUNK == 0 && lda % 8 == 0 && ldw % 8 == 0;
}

// mode 0: c = a w^T; 1: c += a w^T; 2: out_act[m, n/2] = swiglu over strips of 8 gate + 8 up rows;
// 3: out_act[m, n] = xielu(a w^T) with the activation's two factors.
static int skinny(const void* a, const void* w, float* c, void* out_act, int m, int n, int k, int lda, int ldw,
                  int ldc, int ld_act, int mode, int glu_kind, float act_p, float act_q, void* stream,
                  AddGate add = AddGate{nullptr, 0, nullptr, 1.0f},
                  SecondProduct second = SecondProduct{nullptr, nullptr, nullptr, 0, 0, 0, 0, 0, 0}) {
    if (m == 0 || n == 0) return 0;
    TI_REQUIRE(ti_gemm_skinny_supported(m, n, k, lda, ldw),
               "gemm_skinny: M=%d (1..64), K=%d (multiple of 32) or row strides %d, %d (multiples of 8) "
               "are not supported", m, k, lda, ldw);
    TI_REQUIRE(((uintptr_t)a % 16 == 0) && ((uintptr_t)w % 16 == 0),
               "gemm_skinny: operands must be 16-byte aligned");
    TI_REQUIRE(mode != MODE_SWIGLU || n % 16 == 0, "gemm_skinny: SwiGLU needs N %% 16 == 0, got %d", n);
    cudaStream_t s = (cudaStream_t)stream;
    // narrow outputs get blocks of 8 rows, so that at least about 128 blocks share the reading
    const bool narrow = mode != MODE_SWIGLU && (n + STRIP - 1) / STRIP + (second.n + STRIP - 1) / STRIP < 128;
    const int rows = narrow ? 8 : STRIP;
    unsigned blocks = (unsigned)((n + rows - 1) / rows);
    const int longest = k > second.k ? k : second.k;
    if (second.n > 0) {
        second.first_block = blocks;
        blocks += (unsigned)((second.n + rows - 1) / rows);
    }
#define LAUNCH(NT)                                                                                  \
    if (narrow)                                                                                     \
        ti_launch_pdl(gemm_skinny_kernel<NT, 8, 8>, blocks, WARPS * 32, 0, s,      \
                      (const bf16*)a, (const bf16*)w, c, (bf16*)out_act, m, n, k, lda, ldw, ldc,    \
                      ld_act, mode, glu_kind, act_p, act_q, add, second);                                                                \
    else if (longest <= SHORT_K && mode == MODE_STORE && NT <= 2)                                         \
        ti_launch_pdl((gemm_skinny_kernel<NT <= 2 ? NT : 1, 16, 4, true>), blocks, \
                      WARPS * 32, 0, s, (const bf16*)a, (const bf16*)w, c, (bf16*)out_act, m, n, k, \
                      lda, ldw, ldc, ld_act, mode, glu_kind, act_p, act_q, add, second);                                   \
    else if (longest <= SHORT_K)                                                                          \
        ti_launch_pdl(gemm_skinny_kernel<NT, 16, 4>, blocks,                                        \
                      WARPS * 32, 0, s, (const bf16*)a, (const bf16*)w, c, (bf16*)out_act, m, n, k, \
                      lda, ldw, ldc, ld_act, mode, glu_kind, act_p, act_q, add, second);                                   \
    else                                                                                            \
        ti_launch_pdl(gemm_skinny_kernel<NT, 16, 8>, blocks,                                        \
                      WARPS * 32, 0, s, (const bf16*)a, (const bf16*)w, c, (bf16*)out_act, m, n, k, \
                      lda, ldw, ldc, ld_act, mode, glu_kind, act_p, act_q, add, second)
    if (m <= 8) { LAUNCH(1); }
    else if (m <= 16) { LAUNCH(2); }
    else if (m <= 32) { LAUNCH(4); }
    else { LAUNCH(8); }
#undef LAUNCH
    return ti_check_launch("gemm_skinny");
}

extern "C" int ti_gemm_skinny(const void* a, const void* w, float* c, void* out_act, int m, int n,
                              int k, int lda, int ldw, int ldc, int ld_act, int mode, void* stream) {
    TI_REQUIRE(mode >= MODE_STORE && mode <= MODE_SWIGLU, "gemm_skinny: mode %d", mode);
    return skinny(a, w, c, out_act, m, n, k, lda, ldw, ldc, ld_act, mode, GLU_SILU, 0.0f, 0.0f, stream);
}

// out_act[m, n/2] (bfloat16) = act(gate, up) over strips of 8 gate and 8 up rows of w, with the gated activation
// `glu_kind` of glu.cuh in the epilogue.
extern "C" int ti_gemm_skinny_glu(const void* a, const void* w, void* out_act, int m, int n, int k, int lda, int ldw,
                                  int ld_act, int glu_kind, float glu_limit, float glu_alpha, void* stream) {
    TI_REQUIRE(glu_kind >= GLU_SILU && glu_kind <= GLU_GELU_TANH, "gemm_skinny_glu: activation %d", glu_kind);
    return skinny(a, w, nullptr, out_act, m, n, k, lda, ldw, 0, ld_act, MODE_SWIGLU, glu_kind, glu_limit, glu_alpha, stream);
}

// c += scale sigmoid(gate + bias) * (a w^T), element by element; gate float32 [m, n] (row stride ld_gate), bias [n];
// without a gate c += scale * (a w^T)
extern "C" int ti_gemm_skinny_gated(const void* a, const void* w, float* c, int m, int n, int k, int lda, int ldw,
                                    int ldc, const float* gate, int ld_gate, const float* bias, float scale,
                                    void* stream) {
    TI_REQUIRE((gate != nullptr) == (bias != nullptr), "gemm_skinny_gated: a gate and its bias");
    return skinny(a, w, c, nullptr, m, n, k, lda, ldw, ldc, 0, MODE_ACCUMULATE, GLU_SILU, 0.0f, 0.0f, stream,
                  AddGate{gate, ld_gate, bias, scale});
}

// Two products of m rows in one launch: the first stores its float32 rows into c, or (glu_kind >= 0)
// its gated activation over strips of 8 and 8, or an activation of one value, into out_act; the second stores a2 w2^T into c2.
extern "C" int ti_gemm_skinny_pair(const void* a, const void* w, float* c, void* out_act, int m, int n, int k, int lda,
                                   int ldw, int ldc, int ld_act, int glu_kind, float glu_limit, float glu_alpha,
                                   const void* a2, const void* w2, float* c2, int n2, int k2, int lda2, int ldw2, int ldc2,
                                   void* stream) {
    if (m == 0 || n == 0 || n2 == 0) return 0;
    TI_REQUIRE(glu_kind <= GLU_GELU_TANH || glu_kind == ACT_RELU2, "gemm_skinny_pair: activation %d", glu_kind);
    TI_REQUIRE(ti_gemm_skinny_supported(m, n2, k2, lda2, ldw2) && (uintptr_t)a2 % 16 == 0 && (uintptr_t)w2 % 16 == 0,
               "gemm_skinny_pair: the second product's operands");
    return skinny(a, w, c, out_act, m, n, k, lda, ldw, ldc, ld_act, glu_kind < 0 ? MODE_STORE : act_is_gated(glu_kind) ? MODE_SWIGLU : MODE_UNARY,
                  glu_kind < 0 ? GLU_SILU : glu_kind, glu_limit, glu_alpha, stream, AddGate{nullptr, 0, nullptr, 1.0f},
                  SecondProduct{(const bf16*)a2, (const bf16*)w2, c2, n2, k2, lda2, ldw2, ldc2, 0});
}

// out_act[m, n] (bfloat16) = xielu(a w^T): act_p z^2 + z/2 for z > 0, act_q (exp(z) - 1 - z) + z/2 otherwise
extern "C" int ti_gemm_skinny_xielu(const void* a, const void* w, void* out_act, int m, int n, int k, int lda,
                                    int ldw, int ld_act, float act_p, float act_q, void* stream) {
    return skinny(a, w, nullptr, out_act, m, n, k, lda, ldw, 0, ld_act, MODE_XIELU, GLU_SILU, act_p, act_q, stream);
}

// out_act[m, n] (bfloat16) = act(a w^T) with the activation of one value `act` of glu.cuh
extern "C" int ti_gemm_skinny_unary(const void* a, const void* w, void* out_act, int m, int n, int k, int lda,
                                    int ldw, int ld_act, int act, void* stream) {
    TI_REQUIRE(act == ACT_RELU2, "gemm_skinny_unary: activation %d", act);
    return skinny(a, w, nullptr, out_act, m, n, k, lda, ldw, 0, ld_act, MODE_UNARY, act, 0.0f, 0.0f, stream);
}
