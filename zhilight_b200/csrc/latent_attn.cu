// Attention over a cache of low-rank key-value latents, in the absorbed form, with a per-head softmax sink.
//
// A layer of this kind caches one latent row c_j (kv_rank numbers) per position; keys and values of head h are
// W_uk,h c_j and W_uv,h c_j.  Instead of expanding the cache, the query is pulled through W_uk,h once
// (qa_h = W_uk,h^T q_h, a per-head GEMM before this kernel), so that score_h(i, j) = scale * qa_h(i) . c_j, and the
// probabilities are applied to the latents themselves (o_h = sum_j p_j c_j); W_uv,h follows as a per-head GEMM.  All
// heads of a token read the same latent rows: multi-query attention with head size kv_rank whose K and V are one array.
// The softmax normaliser of head h has one extra term, exp(sink_h), that belongs to no position: it adds to the sum only,
// unscaled, once per head and query.  It enters the running (max, sum) pair as its initial value (max = sink_h, sum = 1),
// or in the merge when the keys of a token are split over several CTAs.  Scores, probabilities and the accumulation are fp32.
//
// Token t of a step sees the rows 0 .. pos[t] of its slot; the step's own latents are appended before this kernel, so
// one kernel serves prompt portions (consecutive positions of one slot) and decode batches (one token per slot).
//
// General form (zl_latent_attention_ex): a cached row may carry more columns than the value has -- a rotated key part
// shared by the heads behind the latent -- that enter the score only; the sink may be absent (an ordinary softmax); a
// sigmoid gate per head may multiply the output; and the probabilities may enter the 16-bit product as a hi + lo pair,
// so that no weight is rounded to 8 bits; and a sliding window may restrict a token to the last `window` rows up to its own.
// k_latent_rope_append writes such rows and the queries' rotated parts.
#include "common.cuh"

#include <math.h>
#include <stdlib.h>

namespace zl {

constexpr int kLaThreads = 128;
constexpr int kLaKeys = 32;         // keys per tile: one per lane in the score phase
constexpr int kLaMaxElems = 4096;   // (heads per CTA) x kv_rank accumulators, 32 per thread at most

template <typename TC>
struct LaParams {
    const float* qa;       // (T, H, R)
    void* const* slot_addrs;
    const int32_t* slot;
    const int32_t* pos;
    const float* sink;     // (H) or null: no extra term
    void* out;             // (T, H, R) activation dtype
    float* part_acc;       // (T, H, S, R)
    float* part_ml;        // (T, H, S, 2)
    float scale;
    int H, R, HG, S;
    int RS;                // columns of a cached row and of qa: the score runs over all of them, the value is the first R
    const float* gate = nullptr;   // gate[t * ldg + h] logits or null
    long long ldg = 0;
    int window = 0;                // > 0: rows at distance >= window are not seen
};

// first row a token at `pos` sees
template <typename TC>
__device__ __forceinline__ int la_first_row(const LaParams<TC>& p, int pos) {
    return p.window > 0 && pos >= p.window ? pos - p.window + 1 : 0;
}

__device__ __forceinline__ float la_gate(const float* gate, long long ldg, int t, int h) {
    return gate ? 1.0f / (1.0f + expf(-gate[(size_t)t * ldg + h])) : 1.0f;
}

template <typename TC, int EPT>
__global__ void __launch_bounds__(kLaThreads) k_latent_attn(LaParams<TC> p) {
    extern __shared__ float smem[];
    const int R = p.R, RS = p.RS, RP = RS + 1;
    float* sq = smem;                       // [HG][RS]
    float* sc = sq + p.HG * RS;             // [32][RS + 1]
    float* sp = sc + kLaKeys * RP;          // [HG][32]
    float* sm = sp + p.HG * kLaKeys;        // [HG] running max
    float* sl = sm + p.HG;                  // [HG] running sum
    float* scorr = sl + p.HG;               // [HG]
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, h0 = blockIdx.y * p.HG, split = blockIdx.z;
    const int hg = min(p.HG, p.H - h0);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int len = p.pos[t] + 1;
    const TC* cache = static_cast<const TC*>(p.slot_addrs[p.slot[t]]);
    int lo = la_first_row(p, len - 1), hi = len;
    if (p.S > 1) {
        const int per = cdiv(cdiv(len - lo, p.S), kLaKeys) * kLaKeys;
        lo += split * per;
        hi = min(len, lo + per);
    }
    for (int i = tid; i < hg * RS; i += kLaThreads) sq[i] = p.qa[((size_t)t * p.H + h0) * RS + i];
    for (int i = tid; i < hg; i += kLaThreads) {
        sm[i] = p.S > 1 || !p.sink ? -INFINITY : p.sink[h0 + i];
        sl[i] = p.S > 1 || !p.sink ? 0.f : 1.f;
    }
    float acc[EPT];
#pragma unroll
    for (int k = 0; k < EPT; ++k) acc[k] = 0.f;

    for (int j0 = lo; j0 < hi; j0 += kLaKeys) {
        __syncthreads();   // previous tile fully consumed (and sq / sm / sl initialised)
        for (int i = tid; i < kLaKeys * RS; i += kLaThreads) {
            const int j = i / RS, r = i - j * RS;
            sc[j * RP + r] = (j0 + j < hi) ? to_f32<TC>(cache[(size_t)(j0 + j) * RS + r]) : 0.f;
        }
        __syncthreads();
        for (int hh = warp; hh < hg; hh += kLaThreads / 32) {
            const float* q = sq + hh * RS;
            const float* c = sc + lane * RP;
            float s = 0.f;
            for (int r = 0; r < RS; ++r) s = fmaf(q[r], c[r], s);
            const bool valid = j0 + lane < hi;
            s = valid ? s * p.scale : -INFINITY;
            const float m_old = sm[hh];
            const float m_new = fmaxf(m_old, warp_max(s));
            const float pj = valid ? expf(s - m_new) : 0.f;
            const float ps = warp_sum(pj);
            sp[hh * kLaKeys + lane] = pj;
            __syncwarp();
            if (lane == 0) {
                const float corr = m_old == -INFINITY ? 0.f : expf(m_old - m_new);
                scorr[hh] = corr;
                sl[hh] = sl[hh] * corr + ps;
                sm[hh] = m_new;
            }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < EPT; ++k) {
            const int e = tid + k * kLaThreads;
            if (e < hg * R) {
                const int hh = e / R, r = e - hh * R;
                float a = acc[k] * scorr[hh];
                const float* pr = sp + hh * kLaKeys;
#pragma unroll 8
                for (int j = 0; j < kLaKeys; ++j) a = fmaf(pr[j], sc[j * RP + r], a);
                acc[k] = a;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
        const int e = tid + k * kLaThreads;
        if (e < hg * R) {
            const int hh = e / R, r = e - hh * R;
            const size_t th = (size_t)t * p.H + h0 + hh;
            if (p.S > 1) p.part_acc[(th * p.S + split) * R + r] = acc[k];
            else static_cast<TC*>(p.out)[th * R + r] = from_f32<TC>(acc[k] / sl[hh] * la_gate(p.gate, p.ldg, t, h0 + hh));
        }
    }
    for (int i = tid; p.S > 1 && i < hg; i += kLaThreads) {
        const size_t th = (size_t)t * p.H + h0 + i;
        p.part_ml[(th * p.S + split) * 2 + 0] = sm[i];
        p.part_ml[(th * p.S + split) * 2 + 1] = sl[i];
    }
}

// grid (H, T): merge the S <= 64 partial (max, sum, accumulator) triples of one (token, head) and the sink
template <typename TC>
__global__ void k_latent_attn_merge(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                    const float* __restrict__ sink, const float* __restrict__ gate, long long ldg,
                                    TC* __restrict__ out, int H, int R, int S) {
    __shared__ float wgt[64];
    pdl_trigger();
    pdl_wait();
    const size_t th = (size_t)blockIdx.y * H + blockIdx.x;
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        const float* ml = part_ml + th * S * 2;
        const float sk = sink ? sink[blockIdx.x] : -INFINITY;
        const float m0 = lane < S ? ml[2 * lane] : -INFINITY, m1 = lane + 32 < S ? ml[2 * (lane + 32)] : -INFINITY;
        const float l0 = lane < S ? ml[2 * lane + 1] : 0.f, l1 = lane + 32 < S ? ml[2 * (lane + 32) + 1] : 0.f;
        const float M = fmaxf(sk, warp_max(fmaxf(m0, m1)));
        const float e0 = m0 == -INFINITY ? 0.f : expf(m0 - M), e1 = m1 == -INFINITY ? 0.f : expf(m1 - M);
        const float L = expf(sk - M) + warp_sum(l0 * e0 + l1 * e1);
        const float gl = la_gate(gate, ldg, blockIdx.y, blockIdx.x) / L;
        wgt[lane] = e0 * gl;
        wgt[lane + 32] = e1 * gl;
    }
    __syncthreads();
    const float* pa = part_acc + th * S * R;
    for (int r = threadIdx.x; r < R; r += blockDim.x) {
        float a = 0.f;
#pragma unroll 4
        for (int s = 0; s < S; ++s) a = fmaf(pa[(size_t)s * R + r], wgt[s], a);
        out[th * R + r] = from_f32<TC>(a);
    }
}

// ---- tensor-core variant (bfloat16 caches, kv_rank a multiple of 64 up to 512) -------------------------------------------
// One CTA = one token x 16 heads x one key range; 4 warps.  The 32-key latent tile is staged once in shared memory
// (cp.async, three tiles in flight) and serves both products: S = Qa C^T (contraction over kv_rank, split in quarters over the
// warps, the partial 16 x 32 score tiles summed through shared memory in a fixed order) and O += P C (each warp owns a
// quarter of the kv_rank output columns; C is read through ldmatrix.trans).  Scores, softmax and O are fp32; Qa and P
// enter the MMAs as bfloat16.
constexpr int kLmKeys = 32;
constexpr int kLmRows = 16;
// latent tiles in flight per CTA; the general form's longer rows leave room for two if two CTAs are to share an SM
template <bool EX>
constexpr int lm_stages() { return EX ? 2 : 3; }

__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
    __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_u32(smem_row)));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"(smem_u32(smem_row)));
}

// NK: the value has 64 * NK columns, every warp contracts over 16 * NK of them and owns 16 * NK output columns.  EX: the
// general form -- up to 64 score-only columns behind them (16 per warp), no sink, gate, probabilities as a hi + lo pair.
template <int NK, bool EX>
__global__ void __launch_bounds__(128) k_latent_attn_mma(LaParams<__nv_bfloat16> p) {
    constexpr int RQ = 16 * NK, R = 4 * RQ;
    const int RS = EX ? p.RS : R, RP = RS + 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* sc = reinterpret_cast<__nv_bfloat16*>(smem_raw);                       // [stages][32][RP]
    constexpr int STG = lm_stages<EX>();
    float* ss = reinterpret_cast<float*>(smem_raw + (size_t)STG * kLmKeys * RP * 2);   // [4][16][34]
    pdl_trigger();
    pdl_wait();
    const int h0 = blockIdx.x * kLmRows, t = blockIdx.y, split = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int len = p.pos[t] + 1;
    const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.slot_addrs[p.slot[t]]);
    int lo = la_first_row(p, len - 1), hi = len;
    if (p.S > 1) {
        const int per = cdiv(cdiv(len - lo, p.S), kLmKeys) * kLmKeys;
        lo += split * per;
        hi = min(len, lo + per);
    }
    const int ha = h0 + g, hb = h0 + g + 8;   // the two heads (rows) this lane holds
    // query fragments of this warp's contraction quarter
    uint32_t qf[NK][4];
    {
        const float* qa = p.qa + ((size_t)t * p.H) * RS + warp * RQ;
#pragma unroll
        for (int ks = 0; ks < NK; ++ks) {
            const int k = ks * 16 + 2 * q4;
            const float2 z = make_float2(0.f, 0.f);
            const float2 a0 = ha < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)ha * RS + k) : z;
            const float2 a1 = hb < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)hb * RS + k) : z;
            const float2 a2 = ha < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)ha * RS + k + 8) : z;
            const float2 a3 = hb < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)hb * RS + k + 8) : z;
            qf[ks][0] = pack_bf16(a0.x, a0.y), qf[ks][1] = pack_bf16(a1.x, a1.y);
            qf[ks][2] = pack_bf16(a2.x, a2.y), qf[ks][3] = pack_bf16(a3.x, a3.y);
        }
    }
    const bool extra = EX && warp * 16 < RS - R;   // this warp's 16 score-only columns
    uint32_t qx[4] = {0, 0, 0, 0};
    if (extra) {
        const float* qa = p.qa + ((size_t)t * p.H) * RS + R + warp * 16 + 2 * q4;
        const float2 z = make_float2(0.f, 0.f);
        const float2 a0 = ha < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)ha * RS) : z;
        const float2 a1 = hb < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)hb * RS) : z;
        const float2 a2 = ha < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)ha * RS + 8) : z;
        const float2 a3 = hb < p.H ? *reinterpret_cast<const float2*>(qa + (size_t)hb * RS + 8) : z;
        qx[0] = pack_bf16(a0.x, a0.y), qx[1] = pack_bf16(a1.x, a1.y);
        qx[2] = pack_bf16(a2.x, a2.y), qx[3] = pack_bf16(a3.x, a3.y);
    }
    float m_run[2], l_run[2];
    const bool with_sink = p.S == 1 && (!EX || p.sink);
    m_run[0] = !with_sink ? -INFINITY : (ha < p.H ? p.sink[ha] : 0.f);
    m_run[1] = !with_sink ? -INFINITY : (hb < p.H ? p.sink[hb] : 0.f);
    l_run[0] = l_run[1] = with_sink ? 1.f : 0.f;
    float o[2 * NK][4];
#pragma unroll
    for (int i = 0; i < 2 * NK; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[i][c] = 0.f;

    auto stage = [&](int j0, int buf) {   // 32 keys x R bf16 in 16-byte pieces; keys past `hi` are zero rows
        __nv_bfloat16* dst = sc + (size_t)buf * kLmKeys * RP;
        for (int i = tid; i < kLmKeys * (RS / 8); i += 128) {
            const int j = i / (RS / 8), c8 = (i - j * (RS / 8)) * 8;
            if (j0 + j < hi) cp_async16(dst + j * RP + c8, cache + (size_t)(j0 + j) * RS + c8);
            else *reinterpret_cast<uint4*>(dst + j * RP + c8) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    };
    const int n_tiles = hi > lo ? cdiv(hi - lo, kLmKeys) : 0;
#pragma unroll
    for (int i = 0; i < STG - 1; ++i) {
        if (i < n_tiles) stage(lo + i * kLmKeys, i);
        else cp_async_commit();
    }
    for (int it = 0; it < n_tiles; ++it) {
        const int j0 = lo + it * kLmKeys, buf = it % STG;
        cp_async_wait<STG - 2>();   // all but the younger groups: tile `it` has landed
        __syncthreads();      // ... for every thread; every warp is done with round it - 1 (its buffer, the score tiles)
        if (it + STG - 1 < n_tiles) stage(j0 + (STG - 1) * kLmKeys, (it + STG - 1) % STG);   // ahead of the math
        else cp_async_commit();
        const __nv_bfloat16* ct = sc + (size_t)buf * kLmKeys * RP;
        // partial scores over this warp's quarter of kv_rank
        float s[4][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
#pragma unroll
            for (int c = 0; c < 4; ++c) s[nt][c] = 0.f;
            const __nv_bfloat16* krow = ct + (nt * 8 + g) * RP + warp * RQ + 2 * q4;
#pragma unroll
            for (int ks = 0; ks < NK; ++ks) {
                const uint32_t b0 = *reinterpret_cast<const uint32_t*>(krow + ks * 16);
                const uint32_t b1 = *reinterpret_cast<const uint32_t*>(krow + ks * 16 + 8);
                mma_16816_bf16(s[nt], qf[ks], b0, b1, s[nt]);
            }
            if (extra) {
                const __nv_bfloat16* xrow = ct + (nt * 8 + g) * RP + R + warp * 16 + 2 * q4;
                const uint32_t b0 = *reinterpret_cast<const uint32_t*>(xrow);
                const uint32_t b1 = *reinterpret_cast<const uint32_t*>(xrow + 8);
                mma_16816_bf16(s[nt], qx, b0, b1, s[nt]);
            }
        }
        float* mine = ss + warp * (kLmRows * 34);
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            *reinterpret_cast<float2*>(mine + g * 34 + nt * 8 + 2 * q4) = make_float2(s[nt][0], s[nt][1]);
            *reinterpret_cast<float2*>(mine + (g + 8) * 34 + nt * 8 + 2 * q4) = make_float2(s[nt][2], s[nt][3]);
        }
        __syncthreads();
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            float2 ra = make_float2(0.f, 0.f), rb = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < 4; ++w) {   // same order in every warp: identical sums
                const float2 xa = *reinterpret_cast<const float2*>(ss + w * (kLmRows * 34) + g * 34 + nt * 8 + 2 * q4);
                const float2 xb = *reinterpret_cast<const float2*>(ss + w * (kLmRows * 34) + (g + 8) * 34 + nt * 8 + 2 * q4);
                ra.x += xa.x, ra.y += xa.y, rb.x += xb.x, rb.y += xb.y;
            }
            const int j = j0 + nt * 8 + 2 * q4;
            s[nt][0] = j < hi ? ra.x * p.scale : -INFINITY;
            s[nt][1] = j + 1 < hi ? ra.y * p.scale : -INFINITY;
            s[nt][2] = j < hi ? rb.x * p.scale : -INFINITY;
            s[nt][3] = j + 1 < hi ? rb.y * p.scale : -INFINITY;
            mx[0] = fmaxf(mx[0], fmaxf(s[nt][0], s[nt][1]));
            mx[1] = fmaxf(mx[1], fmaxf(s[nt][2], s[nt][3]));
        }
        float corr[2], sum[2] = {0.f, 0.f};
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            const float m_new = fmaxf(m_run[r], mx[r]);
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            corr[r] = expf(m_run[r] - m_use);
            m_run[r] = m_new;
            mx[r] = m_use;
        }
        uint32_t pf[2][4], pl[2][4];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
            const float p0 = expf(s[nt][0] - mx[0]), p1 = expf(s[nt][1] - mx[0]);
            const float p2 = expf(s[nt][2] - mx[1]), p3 = expf(s[nt][3] - mx[1]);
            sum[0] += p0 + p1;
            sum[1] += p2 + p3;
            pf[nt >> 1][(nt & 1) * 2 + 0] = pack_bf16(p0, p1);
            pf[nt >> 1][(nt & 1) * 2 + 1] = pack_bf16(p2, p3);
            if constexpr (EX) {
                auto lo = [](float v) { return v - __bfloat162float(__float2bfloat16_rn(v)); };
                pl[nt >> 1][(nt & 1) * 2 + 0] = pack_bf16(lo(p0), lo(p1));
                pl[nt >> 1][(nt & 1) * 2 + 1] = pack_bf16(lo(p2), lo(p3));
            }
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
            sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
            l_run[r] = l_run[r] * corr[r] + sum[r];
        }
        // O (16 x RQ columns of this warp) = O * corr + P (16 x 32 keys) C (32 keys x RQ)
#pragma unroll
        for (int nt = 0; nt < 2 * NK; ++nt) {
            o[nt][0] *= corr[0], o[nt][1] *= corr[0], o[nt][2] *= corr[1], o[nt][3] *= corr[1];
            uint32_t bv[4];
            ldmatrix_x4_trans(bv, ct + lane * RP + warp * RQ + nt * 8);
            mma_16816_bf16(o[nt], pf[0], bv[0], bv[1], o[nt]);
            mma_16816_bf16(o[nt], pf[1], bv[2], bv[3], o[nt]);
            if constexpr (EX) {
                mma_16816_bf16(o[nt], pl[0], bv[0], bv[1], o[nt]);
                mma_16816_bf16(o[nt], pl[1], bv[2], bv[3], o[nt]);
            }
        }
    }
    const size_t tha = (size_t)t * p.H + ha, thb = (size_t)t * p.H + hb;
    float fa = 1.0f / l_run[0], fb = 1.0f / l_run[1];
    if (EX && p.S == 1 && p.gate) {
        if (ha < p.H) fa *= la_gate(p.gate, p.ldg, t, ha);
        if (hb < p.H) fb *= la_gate(p.gate, p.ldg, t, hb);
    }
#pragma unroll
    for (int nt = 0; nt < 2 * NK; ++nt) {
        const int col = warp * RQ + nt * 8 + 2 * q4;
        if (p.S > 1) {
            if (ha < p.H) *reinterpret_cast<float2*>(p.part_acc + (tha * p.S + split) * R + col) = make_float2(o[nt][0], o[nt][1]);
            if (hb < p.H) *reinterpret_cast<float2*>(p.part_acc + (thb * p.S + split) * R + col) = make_float2(o[nt][2], o[nt][3]);
        } else {
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
            if (ha < p.H)
                *reinterpret_cast<uint32_t*>(out + tha * R + col) = pack_bf16(o[nt][0] * fa, o[nt][1] * fa);
            if (hb < p.H)
                *reinterpret_cast<uint32_t*>(out + thb * R + col) = pack_bf16(o[nt][2] * fb, o[nt][3] * fb);
        }
    }
    if (p.S > 1 && warp == 0 && q4 == 0) {
        if (ha < p.H) p.part_ml[(tha * p.S + split) * 2] = m_run[0], p.part_ml[(tha * p.S + split) * 2 + 1] = l_run[0];
        if (hb < p.H) p.part_ml[(thb * p.S + split) * 2] = m_run[1], p.part_ml[(thb * p.S + split) * 2 + 1] = l_run[1];
    }
}

// ---- prompt form of the general tensor-core kernel ---------------------------------------------------------------------
// One CTA = 64 rows = (consecutive tokens of one run) x (heads), one key range; 8 warps in pairs of the same 16 rows.  Every
// 32-key latent tile serves all 64 rows (cp.async, two tiles in flight; the queries stay in shared memory).  S: a warp takes
// 16 of the 32 keys over the whole contraction; the pair exchanges its score halves through shared memory; both warps then
// hold the same softmax state, and each owns half of the value columns of O += P C.
constexpr int kLtRows = 64, kLtKeys = 32, kLtStages = 2, kLtSp = kLtKeys + 4;

struct LaTileP {
    LaParams<__nv_bfloat16> a;
    const int32_t *run_row0, *run_len;
    int hb, nq;   // heads and tokens per tile
};

template <int NK>
__global__ void __launch_bounds__(256, 1) k_latent_tile_mma(LaTileP pp) {
    constexpr int R = 64 * NK, NT = 4 * NK;   // value columns; 8-column tiles per warp
    const LaParams<__nv_bfloat16>& p = pp.a;
    const int RS = p.RS, RP = RS + 8, H = p.H;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    __nv_bfloat16* sq = reinterpret_cast<__nv_bfloat16*>(smem_raw);          // [64][RP]
    __nv_bfloat16* sc = sq + (size_t)kLtRows * RP;                           // [stages][32][RP]
    float* ss = reinterpret_cast<float*>(sc + (size_t)kLtStages * kLtKeys * RP);   // [64][kLtSp]
    pdl_trigger();
    pdl_wait();
    const int run = blockIdx.z / p.S, split = blockIdx.z - run * p.S, h0 = blockIdx.x * pp.hb;
    const int len = pp.run_len[run], t0 = (int)(gridDim.y - 1 - blockIdx.y) * pp.nq;   // the tiles with the most keys start first
    if (t0 >= len) return;
    const int ntok = min(pp.nq, len - t0), row0 = pp.run_row0[run] + t0, hb = pp.hb, hn = min(hb, H - h0);
    const int pos0 = p.pos[row0];
    const __nv_bfloat16* cache = static_cast<const __nv_bfloat16*>(p.slot_addrs[p.slot[row0]]);
    // row tiles start at multiples of kLtKeys from row 0 whatever the step, so a token's sums do not depend on the cut
    int lo = la_first_row(p, pos0) / kLtKeys * kLtKeys, hi = pos0 + ntok;
    if (p.S > 1) {
        const int per = cdiv(cdiv(hi - lo, p.S), kLtKeys) * kLtKeys;
        lo += split * per;
        hi = min(hi, lo + per);
    }
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
    const int rb = warp >> 1, hf = warp & 1;
    const int n8 = RS / 8;
    auto stage = [&](int j0, int buf) {   // keys past `hi` are zero rows
        __nv_bfloat16* dst = sc + (size_t)buf * kLtKeys * RP;
        for (int j = warp; j < kLtKeys; j += 8)
            for (int c = lane; c < n8; c += 32) {
                if (j0 + j < hi) cp_async16(dst + j * RP + c * 8, cache + (size_t)(j0 + j) * RS + c * 8);
                else *reinterpret_cast<uint4*>(dst + j * RP + c * 8) = make_uint4(0, 0, 0, 0);
            }
        cp_async_commit();
    };
    int t_of[2], h_of[2], pos_of[2], first_of[2];
    bool ok[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = rb * 16 + g + i * 8, tk = r / hb;
        t_of[i] = row0 + tk;
        h_of[i] = h0 + r - tk * hb;
        ok[i] = tk < ntok && h_of[i] < H;
        pos_of[i] = ok[i] ? pos0 + tk : -1;
        first_of[i] = la_first_row(p, pos_of[i]);
    }
    float m_run[2], l_run[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const bool with_sink = p.S == 1 && p.sink && ok[i];
        m_run[i] = with_sink ? p.sink[h_of[i]] : -INFINITY;
        l_run[i] = with_sink ? 1.f : 0.f;
    }
    float o[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[i][c] = 0.f;
    const int n_tiles = hi > lo ? cdiv(hi - lo, kLtKeys) : 0;
    if (n_tiles > 0) {
        stage(lo, 0);
        for (int r = warp; r < kLtRows; r += 8) {
            const int tk = r / hb, h = r - tk * hb;
            const bool in = tk < ntok && h < hn;
            const float* src = p.qa + ((size_t)(row0 + (in ? tk : 0)) * H + h0 + (in ? h : 0)) * RS;
            for (int c = lane; c < RS / 4; c += 32) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (in) v = reinterpret_cast<const float4*>(src)[c];
                *reinterpret_cast<uint2*>(sq + (size_t)r * RP + c * 4) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
            }
        }
    }
    for (int it = 0; it < n_tiles; ++it) {
        const int j0 = lo + it * kLtKeys;
        cp_async_wait<0>();
        __syncthreads();   // tile `it` (and the queries) are in place; every warp is done with the other buffer and the scores
        if (it + 1 < n_tiles) stage(j0 + kLtKeys, (it + 1) & 1);
        const __nv_bfloat16* ct = sc + (size_t)(it & 1) * kLtKeys * RP;
        float s[4][4];   // two 8-key tiles, each in two chains over alternating contraction steps
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[i][c] = 0.f;
        const __nv_bfloat16* qrow = sq + (size_t)(rb * 16 + (lane & 15)) * RP + (lane >> 4) * 8;
        const __nv_bfloat16* krow = ct + (size_t)(hf * 16 + (lane & 7) + (lane >> 4) * 8) * RP + ((lane >> 3) & 1) * 8;
#pragma unroll 4
        for (int ks = 0; ks < RS / 16; ++ks) {
            uint32_t a[4], b[4];
            ldmatrix_x4(a, qrow + ks * 16);
            ldmatrix_x4(b, krow + ks * 16);
            if (ks & 1) {
                mma_16816_bf16(s[2], a, b[0], b[1], s[2]);
                mma_16816_bf16(s[3], a, b[2], b[3], s[3]);
            } else {
                mma_16816_bf16(s[0], a, b[0], b[1], s[0]);
                mma_16816_bf16(s[1], a, b[2], b[3], s[1]);
            }
        }
        float* sr = ss + (size_t)rb * 16 * kLtSp;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            float* d = sr + (size_t)g * kLtSp + hf * 16 + i * 8 + 2 * q4;
            *reinterpret_cast<float2*>(d) = make_float2(s[i][0] + s[i + 2][0], s[i][1] + s[i + 2][1]);
            *reinterpret_cast<float2*>(d + 8 * kLtSp) = make_float2(s[i][2] + s[i + 2][2], s[i][3] + s[i + 2][3]);
        }
        asm volatile("bar.sync %0, 64;" ::"r"(1 + rb) : "memory");   // the pair's halves are in place
        float v[4][4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float2 x = *reinterpret_cast<const float2*>(sr + (size_t)(g + i * 8) * kLtSp + nt * 8 + 2 * q4);
                const int j = j0 + nt * 8 + 2 * q4;
                v[nt][2 * i] = j < hi && j <= pos_of[i] && j >= first_of[i] ? x.x * p.scale : -INFINITY;
                v[nt][2 * i + 1] = j + 1 < hi && j + 1 <= pos_of[i] && j + 1 >= first_of[i] ? x.y * p.scale : -INFINITY;
                mx[i] = fmaxf(mx[i], fmaxf(v[nt][2 * i], v[nt][2 * i + 1]));
            }
        float corr[2], sum[2] = {0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            const float m_new = fmaxf(m_run[i], mx[i]), m_use = m_new == -INFINITY ? 0.f : m_new;
            corr[i] = expf(m_run[i] - m_use);
            m_run[i] = m_new;
            mx[i] = m_use;
        }
        uint32_t ph[2][4], pl[2][4];
        auto rest = [](float x) { return x - __bfloat162float(__float2bfloat16_rn(x)); };
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const float x = expf(v[nt][2 * i] - mx[i]), y = expf(v[nt][2 * i + 1] - mx[i]);
                sum[i] += x + y;
                ph[nt >> 1][(nt & 1) * 2 + i] = pack_bf16(x, y);
                pl[nt >> 1][(nt & 1) * 2 + i] = pack_bf16(rest(x), rest(y));
            }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
            sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
            l_run[i] = l_run[i] * corr[i] + sum[i];
        }
        if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
            for (int nt = 0; nt < NT; ++nt) o[nt][0] *= corr[0], o[nt][1] *= corr[0], o[nt][2] *= corr[1], o[nt][3] *= corr[1];
        }
        const __nv_bfloat16* vrow = ct + (size_t)lane * RP + hf * (R / 2);
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            uint32_t bv[4];
            ldmatrix_x4_trans(bv, vrow + nt * 8);
            mma_16816_bf16(o[nt], ph[0], bv[0], bv[1], o[nt]);
            mma_16816_bf16(o[nt], ph[1], bv[2], bv[3], o[nt]);
            mma_16816_bf16(o[nt], pl[0], bv[0], bv[1], o[nt]);
            mma_16816_bf16(o[nt], pl[1], bv[2], bv[3], o[nt]);
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        if (!ok[i]) continue;
        const size_t th = (size_t)t_of[i] * H + h_of[i];
        const float f = p.S > 1 ? 1.f : la_gate(p.gate, p.ldg, t_of[i], h_of[i]) / l_run[i];
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            const int col = hf * (R / 2) + nt * 8 + 2 * q4;
            if (p.S > 1)
                *reinterpret_cast<float2*>(p.part_acc + (th * p.S + split) * R + col) = make_float2(o[nt][2 * i], o[nt][2 * i + 1]);
            else
                *reinterpret_cast<uint32_t*>(static_cast<__nv_bfloat16*>(p.out) + th * R + col) = pack_bf16(o[nt][2 * i] * f, o[nt][2 * i + 1] * f);
        }
        if (p.S > 1 && hf == 0 && q4 == 0) {
            p.part_ml[(th * p.S + split) * 2] = m_run[i];
            p.part_ml[(th * p.S + split) * 2 + 1] = l_run[i];
        }
    }
}

static size_t lt_smem_bytes(int RS) {
    return ((size_t)kLtRows + (size_t)kLtStages * kLtKeys) * (RS + 8) * 2 + (size_t)kLtRows * kLtSp * 4;
}
template <int NK>
static cudaError_t lt_launch(const LaTileP& pp, dim3 grid, bool pdl, cudaStream_t st) {
    const size_t smem = lt_smem_bytes(pp.a.RS);
    static size_t set_for = 0;
    if (smem > 48 * 1024 && smem > set_for) {
        const cudaError_t e = cudaFuncSetAttribute(k_latent_tile_mma<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        set_for = smem;
    }
    return launch(k_latent_tile_mma<NK>, grid, dim3(256), smem, st, pdl, pp);
}

static bool lm_eligible(int dtype, int R) {
    static const bool off = getenv("ZL_LATENT_ATTN_NO_MMA") != nullptr;
    return !off && dtype == ZL_BF16 && R % 64 == 0 && R >= 64 && R <= 512;
}
template <bool EX>
static size_t lm_smem_bytes(int RS) { return (size_t)lm_stages<EX>() * kLmKeys * (RS + 8) * 2 + (size_t)4 * kLmRows * 34 * 4; }
// the general form needs its score-only columns in whole 16-column steps, at most one per warp
static bool lm_eligible_ex(int dtype, int R, int RS) {
    return lm_eligible(dtype, R) && (RS - R) % 16 == 0 && RS - R <= 64 && lm_smem_bytes<true>(RS) <= 200 * 1024;
}

template <int NK, bool EX>
static cudaError_t lm_attr(int bytes) {   // the largest request stands: models of several sizes may live side by side
    static int set_for = 0;
    if (bytes <= 48 * 1024 || bytes <= set_for) return cudaSuccess;
    const cudaError_t e = cudaFuncSetAttribute(k_latent_attn_mma<NK, EX>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e == cudaSuccess) set_for = bytes;
    return e;
}
template <bool EX>
static cudaError_t lm_prepare(int R, int RS) {
    const int b = (int)lm_smem_bytes<EX>(RS);
    switch (R / 64) {
        case 1: return lm_attr<1, EX>(b);
        case 2: return lm_attr<2, EX>(b);
        case 3: return lm_attr<3, EX>(b);
        case 4: return lm_attr<4, EX>(b);
        case 5: return lm_attr<5, EX>(b);
        case 6: return lm_attr<6, EX>(b);
        case 7: return lm_attr<7, EX>(b);
        default: return lm_attr<8, EX>(b);
    }
}

template <bool EX>
static int lm_launch(const LaParams<__nv_bfloat16>& p, int T, bool pdl, cudaStream_t st) {
    const size_t smem = lm_smem_bytes<EX>(p.RS);
    const dim3 grid(cdiv(p.H, kLmRows), T, p.S), block(128);
    switch (p.R / 64) {
        case 1: ZL_CHECK_CUDA(launch(k_latent_attn_mma<1, EX>, grid, block, smem, st, pdl, p)); break;
        case 2: ZL_CHECK_CUDA(launch(k_latent_attn_mma<2, EX>, grid, block, smem, st, pdl, p)); break;
        case 3: ZL_CHECK_CUDA(launch(k_latent_attn_mma<3, EX>, grid, block, smem, st, pdl, p)); break;
        case 4: ZL_CHECK_CUDA(launch(k_latent_attn_mma<4, EX>, grid, block, smem, st, pdl, p)); break;
        case 5: ZL_CHECK_CUDA(launch(k_latent_attn_mma<5, EX>, grid, block, smem, st, pdl, p)); break;
        case 6: ZL_CHECK_CUDA(launch(k_latent_attn_mma<6, EX>, grid, block, smem, st, pdl, p)); break;
        case 7: ZL_CHECK_CUDA(launch(k_latent_attn_mma<7, EX>, grid, block, smem, st, pdl, p)); break;
        default: ZL_CHECK_CUDA(launch(k_latent_attn_mma<8, EX>, grid, block, smem, st, pdl, p)); break;
    }
    if (p.S > 1)
        ZL_CHECK_CUDA(launch(k_latent_attn_merge<__nv_bfloat16>, dim3(p.H, T), dim3(128), 0, st, pdl, (const float*)p.part_acc,
                             (const float*)p.part_ml, p.sink, p.gate, p.ldg, static_cast<__nv_bfloat16*>(p.out), p.H, p.R, p.S));
    return ZL_OK;
}

// the prompt form: tiles of 64 rows over the runs of the step
static int lt_run(const LaParams<__nv_bfloat16>& p, const int32_t* run_row0, const int32_t* run_len, int runs, int max_run_len, int T,
                  bool pdl, cudaStream_t st) {
    const int hb = p.H < kLtRows ? p.H : kLtRows, nq = kLtRows / hb;
    const LaTileP pp{p, run_row0, run_len, hb, nq};
    const dim3 grid(cdiv(p.H, hb), cdiv(max_run_len, nq), runs * p.S);
    switch (p.R / 64) {
        case 1: ZL_CHECK_CUDA(lt_launch<1>(pp, grid, pdl, st)); break;
        case 2: ZL_CHECK_CUDA(lt_launch<2>(pp, grid, pdl, st)); break;
        case 3: ZL_CHECK_CUDA(lt_launch<3>(pp, grid, pdl, st)); break;
        case 4: ZL_CHECK_CUDA(lt_launch<4>(pp, grid, pdl, st)); break;
        case 5: ZL_CHECK_CUDA(lt_launch<5>(pp, grid, pdl, st)); break;
        case 6: ZL_CHECK_CUDA(lt_launch<6>(pp, grid, pdl, st)); break;
        case 7: ZL_CHECK_CUDA(lt_launch<7>(pp, grid, pdl, st)); break;
        default: ZL_CHECK_CUDA(lt_launch<8>(pp, grid, pdl, st)); break;
    }
    if (p.S > 1)
        ZL_CHECK_CUDA(launch(k_latent_attn_merge<__nv_bfloat16>, dim3(p.H, T), dim3(128), 0, st, pdl, (const float*)p.part_acc,
                             (const float*)p.part_ml, p.sink, p.gate, p.ldg, static_cast<__nv_bfloat16*>(p.out), p.H, p.R, p.S));
    return ZL_OK;
}

static int la_heads_per_cta(int H, int R) {
    int hg = kLaMaxElems / R;
    if (hg < 1) hg = 1;
    return hg < H ? hg : H;
}
static size_t la_smem_bytes(int HG, int RS) {
    return sizeof(float) * ((size_t)HG * RS + (size_t)kLaKeys * (RS + 1) + (size_t)HG * kLaKeys + 3 * (size_t)HG);
}

template <typename TC>
static int la_launch(LaParams<TC> p, int T, bool pdl, cudaStream_t st) {
    const size_t smem = la_smem_bytes(p.HG, p.RS);
    const int ept = cdiv(p.HG * p.R, kLaThreads);
    const dim3 grid(T, cdiv(p.H, p.HG), p.S), block(kLaThreads);
#define ZL_LA_CASE(E)                                                                                        \
    {                                                                                                        \
        ZL_CHECK_CUDA(launch(k_latent_attn<TC, E>, grid, block, smem, st, pdl, p));                           \
    }
    if (ept <= 4) ZL_LA_CASE(4)
    else if (ept <= 8) ZL_LA_CASE(8)
    else if (ept <= 16) ZL_LA_CASE(16)
    else ZL_LA_CASE(32)
#undef ZL_LA_CASE
    if (p.S > 1)
        ZL_CHECK_CUDA(launch(k_latent_attn_merge<TC>, dim3(p.H, T), dim3(128), 0, st, pdl, (const float*)p.part_acc,
                             (const float*)p.part_ml, p.sink, p.gate, p.ldg, static_cast<TC*>(p.out), p.H, p.R, p.S));
    return ZL_OK;
}

// one warp per (token, unit): the H query heads, then the rotated key part, then the latent (norm and append)
struct LaPrepP {
    const float* proj;         // the queries' matrix
    long long ldp;
    const float* kv;           // the latents' matrix (the same one, or its own)
    long long ldkv;
    int q_off, H, d, rd;
    const float2* table;       // (T, rd / 2)
    void* q_out;
    float* qa;
    int c_off, R;
    const float* kv_w;
    int rank_cols, row_cols;
    void* const* slot_addrs;
    const int32_t *slot, *pos;
    float eps;
};
template <typename TO>
__global__ void __launch_bounds__(256) k_latent_rope_append(LaPrepP p) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.y, unit = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit > p.H + 1) return;
    const float* row = p.proj + (size_t)t * p.ldp;
    const float2* tab = p.table + (size_t)t * (p.rd >> 1);
    if (unit < p.H) {
        const float* src = row + p.q_off + (size_t)unit * (p.d + p.rd);
        TO* dst = static_cast<TO*>(p.q_out) + ((size_t)t * p.H + unit) * p.d;
#pragma unroll 4
        for (int c = lane; c < p.d; c += 32) dst[c] = from_f32<TO>(__ldg(src + c));
        float* qr = p.qa + ((size_t)t * p.H + unit) * p.row_cols + p.rank_cols;
        for (int i = lane; i < (p.rd >> 1); i += 32) {
            const float u = __ldg(src + p.d + 2 * i), v = __ldg(src + p.d + 2 * i + 1);
            const float2 cs = __ldg(tab + i);
            qr[2 * i] = u * cs.x - v * cs.y;
            qr[2 * i + 1] = v * cs.x + u * cs.y;
        }
        return;
    }
    TO* dst = static_cast<TO*>(p.slot_addrs[p.slot[t]]) + (size_t)p.pos[t] * p.row_cols;
    const float* src = p.kv + (size_t)t * p.ldkv + p.c_off;
    if (unit == p.H) {
        for (int i = lane; i < (p.rd >> 1); i += 32) {
            const float u = src[p.R + 2 * i], v = src[p.R + 2 * i + 1];
            const float2 cs = tab[i];
            dst[p.rank_cols + 2 * i] = from_f32<TO>(u * cs.x - v * cs.y);
            dst[p.rank_cols + 2 * i + 1] = from_f32<TO>(v * cs.x + u * cs.y);
        }
        return;
    }
    float keep[16], ss = 0.f;   // the first 512 columns in registers, every load in flight at once
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int c = lane + 32 * i;
        keep[i] = c < p.R ? __ldg(src + c) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < 16; ++i) ss = fmaf(keep[i], keep[i], ss);
    for (int c = lane + 512; c < p.R; c += 32) ss = fmaf(src[c], src[c], ss);
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)p.R + p.eps);
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int c = lane + 32 * i;
        if (c < p.R) dst[c] = from_f32<TO>(keep[i] * r * __ldg(p.kv_w + c));
    }
    for (int c = lane + 512; c < p.R; c += 32) dst[c] = from_f32<TO>(src[c] * r * p.kv_w[c]);
}

}  // namespace zl

using namespace zl;

extern "C" size_t zl_latent_attention_workspace_bytes(int T, int heads, int kv_rank, int splits) {
    if (splits <= 1) return 0;
    return sizeof(float) * (size_t)T * heads * splits * ((size_t)kv_rank + 2);
}

template <typename TC>
static int la_prepare(size_t smem) {
    static size_t set_for = 0;
    if (smem <= 48 * 1024 || smem <= set_for) return ZL_OK;
    ZL_CHECK_CUDA(cudaFuncSetAttribute(k_latent_attn<TC, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    ZL_CHECK_CUDA(cudaFuncSetAttribute(k_latent_attn<TC, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    ZL_CHECK_CUDA(cudaFuncSetAttribute(k_latent_attn<TC, 16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    ZL_CHECK_CUDA(cudaFuncSetAttribute(k_latent_attn<TC, 32>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    set_for = smem;
    return ZL_OK;
}

// how many CTAs share one token's keys: enough to fill the GPU when the step has few (token, head group) pairs
extern "C" int zl_latent_attention_splits(int T, int heads, int kv_rank, int max_len) {
    if (T <= 0 || heads <= 0 || kv_rank <= 0 || kv_rank > kLaMaxElems) return 1;
    const int ctas = T * cdiv(heads, lm_eligible(ZL_BF16, kv_rank) ? kLmRows : la_heads_per_cta(heads, kv_rank));
    const int want = 2 * device_sm_count();
    if (ctas >= want || max_len <= 4 * kLaKeys) return 1;
    int s = want / ctas;   // rounded down: one wave of CTAs, no tail
    const int by_len = cdiv(max_len, 4 * kLaKeys);
    if (s > by_len) s = by_len;
    return s < 1 ? 1 : (s > 64 ? 64 : s);
}

// opt-in shared memory of the kernel for this shape; call once outside any stream capture
extern "C" int zl_latent_attention_prepare(int heads, int kv_rank, int dtype) {
    if (lm_eligible(dtype, kv_rank)) ZL_CHECK_CUDA(lm_prepare<false>(kv_rank, kv_rank));
    return zl_latent_attention_prepare_ex(heads, kv_rank, kv_rank, dtype);
}

extern "C" int zl_latent_attention_prepare_ex(int heads, int rank_cols, int row_cols, int dtype) {
    ZL_CHECK_ARG(heads > 0 && rank_cols > 0 && row_cols >= rank_cols);
    ZL_CHECK_ARG(dtype == ZL_F16 || dtype == ZL_BF16 || dtype == ZL_F32);
    ZL_CHECK_SUPPORTED(rank_cols <= kLaMaxElems);
    const size_t smem = la_smem_bytes(la_heads_per_cta(heads, rank_cols), row_cols);
    ZL_CHECK_SUPPORTED(smem <= 200 * 1024);
    if (lm_eligible_ex(dtype, rank_cols, row_cols)) ZL_CHECK_CUDA(lm_prepare<true>(rank_cols, row_cols));
    if (dtype == ZL_F32) return la_prepare<float>(smem);
    if (dtype == ZL_BF16) return la_prepare<__nv_bfloat16>(smem);
    return la_prepare<__half>(smem);
}

template <typename TC>
static LaParams<TC> la_params(const float* qa, void* const* slot_addrs, const int32_t* slot, const int32_t* pos, const float* sink,
                              float scale, void* out, int T, int heads, int R, int RS, int splits, void* workspace,
                              const float* gate, long long ldg, int window = 0) {
    float* part_acc = static_cast<float*>(workspace);
    float* part_ml = splits > 1 ? part_acc + (size_t)T * heads * splits * R : nullptr;
    return LaParams<TC>{qa, slot_addrs, slot, pos, sink, out, part_acc, part_ml, scale, heads, R, la_heads_per_cta(heads, R), splits,
                        RS, gate, ldg, window};
}

extern "C" int zl_latent_attention(const float* q_absorbed, void* const* slot_addrs, const int32_t* slot, const int32_t* pos,
                                   const float* sink, float scale, void* out, int T, int heads, int kv_rank, int splits,
                                   void* workspace, size_t workspace_bytes, int dtype, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(q_absorbed && slot_addrs && slot && pos && sink && out && T > 0 && heads > 0 && kv_rank > 0);
    ZL_CHECK_ARG(splits >= 1 && splits <= 65535 && heads <= 65535);
    ZL_CHECK_SUPPORTED(kv_rank <= kLaMaxElems);
    ZL_CHECK_ARG(workspace_bytes >= zl_latent_attention_workspace_bytes(T, heads, kv_rank, splits) && (splits == 1 || workspace));
    if (lm_eligible(dtype, kv_rank) && (reinterpret_cast<uintptr_t>(q_absorbed) & 7) == 0)
        return lm_launch<false>(la_params<__nv_bfloat16>(q_absorbed, slot_addrs, slot, pos, sink, scale, out, T, heads, kv_rank, kv_rank,
                                                         splits, workspace, nullptr, 0), T, pdl != 0, stream);
    return zl_latent_attention_ex(q_absorbed, slot_addrs, slot, pos, sink, nullptr, 0, scale, out, T, heads, kv_rank, kv_rank, splits,
                                  workspace, workspace_bytes, nullptr, nullptr, 0, 0, dtype, pdl, stream);
}

extern "C" int zl_latent_attention_ex(const float* q_absorbed, void* const* slot_addrs, const int32_t* slot, const int32_t* pos,
                                      const float* sink, const float* gate, long long ldg, float scale, void* out, int T,
                                      int heads, int rank_cols, int row_cols, int splits, void* workspace, size_t workspace_bytes,
                                      const int32_t* run_row0, const int32_t* run_len, int runs, int max_run_len, int dtype, int pdl,
                                      zl_stream_t stream) {
    return zl_latent_window_attention(q_absorbed, slot_addrs, slot, pos, sink, gate, ldg, scale, 0, out, T, heads, rank_cols, row_cols,
                                      splits, workspace, workspace_bytes, run_row0, run_len, runs, max_run_len, dtype, pdl, stream);
}

extern "C" int zl_latent_window_attention(const float* q_absorbed, void* const* slot_addrs, const int32_t* slot, const int32_t* pos,
                                          const float* sink, const float* gate, long long ldg, float scale, int window, void* out,
                                          int T, int heads, int rank_cols, int row_cols, int splits, void* workspace,
                                          size_t workspace_bytes, const int32_t* run_row0, const int32_t* run_len, int runs,
                                          int max_run_len, int dtype, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(window >= 0);
    ZL_CHECK_ARG(q_absorbed && slot_addrs && slot && pos && out && T > 0 && T <= 65535 && heads > 0 && rank_cols > 0);
    ZL_CHECK_ARG(row_cols >= rank_cols && (dtype == ZL_F16 || dtype == ZL_BF16 || dtype == ZL_F32));
    ZL_CHECK_ARG(splits >= 1 && splits <= 64 && heads <= 65535);
    ZL_CHECK_SUPPORTED(rank_cols <= kLaMaxElems);
    ZL_CHECK_ARG(workspace_bytes >= zl_latent_attention_workspace_bytes(T, heads, rank_cols, splits) && (splits == 1 || workspace));
    ZL_CHECK_SUPPORTED(la_smem_bytes(la_heads_per_cta(heads, rank_cols), row_cols) <= 200 * 1024);
#define ZL_LA_P(TC) \
    la_params<TC>(q_absorbed, slot_addrs, slot, pos, sink, scale, out, T, heads, rank_cols, row_cols, splits, workspace, gate, ldg, window)
    if (dtype == ZL_F32) return la_launch<float>(ZL_LA_P(float), T, pdl != 0, stream);
    if (dtype == ZL_F16) return la_launch<__half>(ZL_LA_P(__half), T, pdl != 0, stream);
    const bool mma = lm_eligible_ex(dtype, rank_cols, row_cols) && row_cols % 8 == 0 && (reinterpret_cast<uintptr_t>(q_absorbed) & 15) == 0;
    // runs whose rows fill more than one 16-row tile per key tile: a prompt
    static const bool no_tile = getenv("ZL_LATENT_ATTN_NO_TILE") != nullptr;
    if (mma && !no_tile && run_row0 && run_len && runs > 0 && (long long)max_run_len * heads >= 2 * kLmRows && max_run_len > 1 &&
        (long long)runs * splits <= 65535 && lt_smem_bytes(row_cols) <= 225 * 1024)
        return lt_run(ZL_LA_P(__nv_bfloat16), run_row0, run_len, runs, max_run_len, T, pdl != 0, stream);
    if (mma)
        return lm_launch<true>(ZL_LA_P(__nv_bfloat16), T, pdl != 0, stream);
    return la_launch<__nv_bfloat16>(ZL_LA_P(__nv_bfloat16), T, pdl != 0, stream);
#undef ZL_LA_P
}

static int latent_append(const float* q_proj, long long ldq, int q_off, int heads, int dim, int rot_dim, const float* table, void* q_out,
                         float* qa, const float* kv_proj, long long ldkv, int c_off, int kv_rank, const float* kv_weight,
                         int rank_cols, int row_cols, void* const* slot_addrs, const int32_t* slot, const int32_t* pos, int T,
                         float eps, int dtype, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(q_proj && kv_proj && q_out && qa && kv_weight && slot_addrs && slot && pos && T > 0 && T <= 65535 && heads > 0 && dim > 0);
    ZL_CHECK_ARG(kv_rank > 0 && rank_cols >= kv_rank && rot_dim >= 0 && rot_dim % 2 == 0 && row_cols >= rank_cols + rot_dim);
    ZL_CHECK_ARG((rot_dim == 0 || table) && (dtype == ZL_F16 || dtype == ZL_BF16 || dtype == ZL_F32));
    const LaPrepP p{q_proj, ldq, kv_proj, ldkv, q_off, heads, dim, rot_dim, reinterpret_cast<const float2*>(table), q_out, qa, c_off, kv_rank, kv_weight,
                    rank_cols, row_cols, slot_addrs, slot, pos, eps};
    const dim3 grid(cdiv(heads + 2, 8), T), block(256);
    cudaError_t e;
    if (dtype == ZL_F32) e = launch(k_latent_rope_append<float>, grid, block, 0, stream, pdl != 0, p);
    else if (dtype == ZL_BF16) e = launch(k_latent_rope_append<__nv_bfloat16>, grid, block, 0, stream, pdl != 0, p);
    else e = launch(k_latent_rope_append<__half>, grid, block, 0, stream, pdl != 0, p);
    ZL_CHECK_CUDA(e);
    return ZL_OK;
}

extern "C" int zl_latent_rope_append(const float* proj, long long ldp, int q_off, int heads, int dim, int rot_dim,
                                     const float* table, void* q_out, float* qa, int c_off, int kv_rank, const float* kv_weight,
                                     int rank_cols, int row_cols, void* const* slot_addrs, const int32_t* slot, const int32_t* pos,
                                     int T, float eps, int dtype, int pdl, zl_stream_t stream) {
    return latent_append(proj, ldp, q_off, heads, dim, rot_dim, table, q_out, qa, proj, ldp, c_off, kv_rank, kv_weight, rank_cols,
                         row_cols, slot_addrs, slot, pos, T, eps, dtype, pdl, stream);
}

extern "C" int zl_latent_rope_append_split(const float* q_proj, long long ldq, int heads, int dim, int rot_dim, const float* table,
                                           void* q_out, float* qa, const float* kv_proj, long long ldkv, int c_off, int kv_rank,
                                           const float* kv_weight, int rank_cols, int row_cols, void* const* slot_addrs,
                                           const int32_t* slot, const int32_t* pos, int T, float eps, int dtype, int pdl,
                                           zl_stream_t stream) {
    return latent_append(q_proj, ldq, 0, heads, dim, rot_dim, table, q_out, qa, kv_proj, ldkv, c_off, kv_rank, kv_weight, rank_cols,
                         row_cols, slot_addrs, slot, pos, T, eps, dtype, pdl, stream);
}
