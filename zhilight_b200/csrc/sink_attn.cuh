// Parameters of the attention kernels over per-slot caches and the merge of their key splits (sink_attn.cu), shared with
// the kernels that produce the same partial results.
#pragma once
#include "common.cuh"

namespace zl {

struct SinkAttnP {
    const void* q;             // (T, H * d)
    void* const* k_addrs;      // slot -> (max_seq, G, d)
    void* const* v_addrs;      // slot -> (max_seq, G, vd)
    const int32_t *slot, *pos;
    const float* sink;         // (H) or null: sink 0
    const float* gate;         // gate[t * ldg + h] logits or null
    long long ldg;
    void* out;                 // (T, H * vd)
    int H, G, d, vd;
    float scale;
    int splits;
    float* ws;                 // splits > 1: (T, H, splits, 2 + vd) partial (max, sum, weighted values)
    int chunk = 0;             // > 0: keys below (pos / chunk) * chunk are not seen
    const float* dist_bias = nullptr;   // (H, n_dist) added to the scaled score by distance, or null
    int n_dist = 0;
    int no_sink = 0;           // the denominator holds the keys only
    const float* out_table = nullptr;   // (T, vd / 2) pairs (cos, sin): the output of token t is turned back by these angles
    int out_layout = 0;        // ZL_ROT_HALVES: pair (m, m + vd / 2); ZL_ROT_ADJACENT: pair (2m, 2m + 1)
    int window = 0;            // > 0: keys at distance >= window are not seen
    float lambda = 0.f, out_eps = 0.f, out_mul = 1.f;   // two maps: o = a_1 - lambda a_2, out = out_mul o / sqrt(mean(o^2) + out_eps)
    float softcap = 0.f;       // > 0: the scaled score s becomes softcap tanh(s / softcap)
    const float* slopes = nullptr;      // (H): slopes[h] * (pos - key) comes off the score after the cap, or null
    const float* gate_full = nullptr;   // two maps: gate logits, element h * vd + c of row t (row stride ldg), or null
};

// merge of the partial results p.ws (T, H * maps, splits, 2 + vd) into p.out
int sink_attn_merge(const SinkAttnP& p, int maps, int T, int dtype, bool pdl, cudaStream_t stream);

// first key a token at `pos` sees
__device__ __forceinline__ int sa_first_key(const SinkAttnP& p, int pos) {
    if (p.window > 0) return pos >= p.window ? pos - p.window + 1 : 0;
    return p.chunk > 0 ? (pos / p.chunk) * p.chunk : 0;
}

// softcap tanh(s / softcap) through one exponential: tanh(x) = 1 - 2 / (exp(2 x) + 1).  Its absolute error is a few float ulps of
// `softcap`, and absolute is what counts in a score; both limits are right (exp overflows to infinity, underflows to 0).
__device__ __forceinline__ float sa_softcap(float s, float cap, float two_over_cap) {
    return cap - __fdividef(2.0f * cap, __expf(s * two_over_cap) + 1.0f);
}

__device__ __forceinline__ void sa_cp_async16(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void sa_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void sa_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void sa_ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_u32(smem_row)));
}
__device__ __forceinline__ void sa_ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_u32(smem_row)));
}
template <typename T>
__device__ __forceinline__ uint32_t sa_pack(float x, float y) {
    T a = from_f32<T>(x), b = from_f32<T>(y);
    return (uint32_t) * reinterpret_cast<uint16_t*>(&a) | ((uint32_t) * reinterpret_cast<uint16_t*>(&b) << 16);
}

}  // namespace zl
