// Entry points of the recurrence over a matrix state (matrix_state.cuh), the launches of the delta rule and the
// gated sum, and the two small kernels behind launches whose columns are cut over several blocks.
#include "matrix_state.cuh"

using namespace matrix_state;

namespace {

// The gated sum's normaliser column and running maximum from `carry` into the slots, after every
// block of the cut launch has read the old ones: one block per (request, head).
__global__ void __launch_bounds__(64)
matrix_state_commit_kernel(const float* __restrict__ carry, const int* __restrict__ cu_q,
                           const int* __restrict__ slots, float* state, long long state_stride, int heads, int dk,
                           int dv) {
    const int req = blockIdx.x, head = blockIdx.y;
    if (cu_q[req] >= cu_q[req + 1]) return;
    const int cols = dv + 1;
    const float* c = carry + ((size_t)req * heads + head) * (dk + 1);
    float* slot = state + (size_t)slots[req] * state_stride;
    for (int i = threadIdx.x; i < dk; i += blockDim.x) slot[((size_t)head * dk + i) * cols + dv] = c[i];
    if (threadIdx.x == 0) slot[(size_t)heads * dk * cols + head] = c[dk];
}

// out[t, head] = o / rms(o) * weight * act(gate) for rows that column-cut blocks left as float32:
// one warp per (token, head).
template <typename TO>
__global__ void __launch_bounds__(256)
matrix_state_finish_kernel(const float* o_raw, const float* __restrict__ norm_weight, int norm_per_row, float eps,
                           const float* gate, int gate_stride, int gate_act, int rows, int heads, int dv,
                           TO* __restrict__ out) {
    const int unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= rows * heads) return;
    const int t = unit / heads, head = unit % heads;
    const float* o = o_raw + (size_t)unit * dv;
    float ss = 0.0f;
    for (int c = lane; c < dv; c += 32) ss = fmaf(o[c], o[c], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + eps);
    for (int c = lane; c < dv; c += 32) {
        float y = o[c] * inv * norm_weight[(norm_per_row ? head * dv : 0) + c];
        if (gate) y *= gate_value(gate[(size_t)t * gate_stride + head * dv + c], gate_act);
        out[(size_t)unit * dv + c] = from_f32<TO>(y);
    }
}

}  // namespace

// Floats of state per request: every head's S (with the normaliser's column in the gated sum) and,
// in the gated sum, one running maximum per head.
extern "C" long long ti_matrix_state_floats(int mode, int heads, int dk, int dv) {
    return mode == MODE_GATED_SUM ? (long long)heads * dk * (dv + 1) + heads : (long long)heads * dk * dv;
}

// col_block: 0 = a head's columns in one block (dv <= 128) with the norm, weight and gate in the same launch;
// 8, 16, 32, 64 or 128 = that many columns a block (16 threads a column up to 32 columns, 4 beyond), o left in
// `o_raw` and finished by a second launch.
extern "C" int ti_matrix_state(int mode, const float* q, const float* k, const float* v, int q_stride, int k_stride,
                               int v_stride, const float* s0, int s0_stride, const float* s1, int s1_stride,
                               const float* decay, int decay_stride, const float* c0, const float* c1, float cap, const float* gate, int gate_stride,
                               int gate_act, const float* norm_weight, int norm_per_row, float eps,
                               const int* cu_q, const int* slots, int requests, int rows, float* state,
                               long long state_stride, int heads, int kv_heads, int dk, int dv, int col_block,
                               void* out, int out_dtype, float* o_raw, float* carry, void* stream) {
    if (requests == 0 || rows == 0) return 0;
    TI_REQUIRE(mode >= MODE_DELTA && mode <= MODE_DECAYED_SUM, "matrix_state: mode %d", mode);
    TI_REQUIRE(mode != MODE_DECAYED_SUM || decay != nullptr, "matrix_state: the decayed sum needs its decays");
    TI_REQUIRE(dk >= 1 && dk <= 256 && dv >= 1 && dv <= 1024, "matrix_state: head sizes %d x %d (keys up to 256, "
               "values up to 1,024)", dk, dv);
    TI_REQUIRE(heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0, "matrix_state: %d heads over %d key heads",
               heads, kv_heads);
    TI_REQUIRE(out_dtype == TI_F32 || out_dtype == TI_BF16, "matrix_state: output dtype code %d", out_dtype);
    TI_REQUIRE(col_block == 0 || col_block == 8 || col_block == 16 || col_block == 32 || col_block == 64 || col_block == 128,
               "matrix_state: %d columns a block", col_block);
    TI_REQUIRE(col_block != 0 || dv <= 128, "matrix_state: %d value columns do not fit one block", dv);
    TI_REQUIRE(col_block == 0 || o_raw != nullptr, "matrix_state: cut columns need the float32 rows");
    TI_REQUIRE(col_block == 0 || mode != MODE_GATED_SUM || carry != nullptr,
               "matrix_state: cut columns of the gated sum need room for the normaliser and the maximum");
    MatrixStateArgs a;
    a.q = q; a.k = k; a.v = v; a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride;
    a.s0 = s0; a.s1 = s1; a.s0_stride = s0_stride; a.s1_stride = s1_stride;
    a.decay = decay; a.decay_stride = decay_stride; a.c0 = c0; a.c1 = c1; a.cap = cap;
    a.gate = gate; a.gate_stride = gate_stride; a.gate_act = gate_act;
    a.norm_weight = norm_weight; a.norm_per_row = norm_per_row; a.eps = eps;
    a.cu_q = cu_q; a.slots = slots; a.state = state; a.state_stride = state_stride;
    a.heads = heads; a.kv_heads = kv_heads; a.dk = dk; a.dv = dv;
    a.out = out; a.out_bf16 = out_dtype == TI_BF16; a.o_raw = o_raw; a.carry = carry;
    a.cut = col_block != 0;
    a.vec4 = ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) % 16 == 0 &&
              reinterpret_cast<uintptr_t>(decay) % 16 == 0 && decay_stride % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 && dk % 4 == 0 && dv % 4 == 0) ? 1 : 0;
    cudaStream_t s = (cudaStream_t)stream;
    int cb = col_block, col_blocks = 1;
    if (cb == 0) cb = dv <= 32 ? 32 : dv <= 64 ? 64 : 128;
    else col_blocks = (dv + cb - 1) / cb;
    if (mode == MODE_DELTA) launch_dk<MODE_DELTA>(a, requests, cb, col_blocks, s);
    else if (mode == MODE_GATED_SUM) launch_dk<MODE_GATED_SUM>(a, requests, cb, col_blocks, s);
    else launch_decayed_sum(a, requests, cb, col_blocks, s);
    if (int rc = ti_check_launch("matrix_state")) return rc;
    if (col_block != 0) {
        if (mode == MODE_GATED_SUM) {
            matrix_state_commit_kernel<<<dim3(requests, heads), 64, 0, s>>>(carry, cu_q, slots, state, state_stride,
                                                                            heads, dk, dv);
            if (int rc = ti_check_launch("matrix_state_commit")) return rc;
        }
        const int blocks = (rows * heads + 7) / 8;
        if (out_dtype == TI_BF16)
            matrix_state_finish_kernel<bf16><<<blocks, 256, 0, s>>>(o_raw, norm_weight, norm_per_row, eps, gate,
                                                                     gate_stride, gate_act, rows, heads, dv, (bf16*)out);
        else
            matrix_state_finish_kernel<float><<<blocks, 256, 0, s>>>(o_raw, norm_weight, norm_per_row, eps, gate,
                                                                      gate_stride, gate_act, rows, heads, dv, (float*)out);
        return ti_check_launch("matrix_state_finish");
    }
    return 0;
}
