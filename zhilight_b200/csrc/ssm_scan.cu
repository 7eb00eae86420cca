// Selective state space (the state-space duality form): a recurrent mixer whose state per head is a (vdim, state) fp32 matrix,
//   S_t = exp(-exp(a_log) dt_t) S_(t-1) + (dt_t x_t) B_t^T,      o_t = S_t C_t + d_skip x_t,
// one scalar decay per head and token, B and C shared by the heads of a group, dt_t = softplus(logit + bias).  x, B and C come
// out of a causal convolution per channel (the last taps - 1 inputs of a sequence are kept per slot) and silu.
//
// k_ssm_prep: convolution, silu, step sizes and decays of all rows of the step at once.  k_ssm_scan: a row of S (one value
// channel) depends on its own past and the token's vectors only; it is walked through the tokens of its sequence in order, so a
// token's result does not depend on how the sequence was cut into steps or on the rest of the step.  A CTA owns 32 channels of
// one head of one run; a channel's state lives in the registers of four adjacent lanes, in 4-element pieces f = 4 i + q of the
// state dimension (their 16-byte reads of a staged vector fall into different banks), updated and read out with packed fp32
// pairs.  The token vectors fly into shared memory chunk by chunk ahead of use.  State sizes above 256 take k_ssm_scan_any
// (state in shared memory, one thread per channel).  A run that starts at position 0 starts from a zero state (a slot given to
// a new sequence needs no clearing); the final state and the convolution's last inputs go back to the slot.
#include "common.cuh"

namespace zl {

struct SsmP {
    const float* proj;          // (T, ld): x | B | C at col_x (C channels), step-size logits (H) at col_dt
    long long ld;
    int col_x, col_dt;
    const float *conv_w, *conv_b;   // (taps, C), (C)
    int taps;
    const float *dt_bias, *a_log, *d_skip;   // (H)
    void* const* ring_addrs;    // slot -> (taps - 1, C): input at position p sits in entry p % (taps - 1)
    const int32_t *run_row0, *run_len, *slot, *pos;
    void* const* state_addrs;   // slot -> (H, dv, N)
    float* o;
    long long ld_o;
    int H, dv, N, G, C;
    float* xbc;                 // (T, C) after convolution and silu
    float2* dtd;                // (T, H): dt, decay
    int vec;                    // staged pieces of 16 bytes
};

constexpr int kSsChunk = 16, kSsCols = 32, kSsLanes = 4, kSsThreads = kSsCols * kSsLanes;

__device__ __forceinline__ float ss_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// grid (channel blocks + 1, T); the last block computes the heads' step sizes.  V channels per thread (4: 16-byte rows).
template <int V>
__global__ void __launch_bounds__(256) k_ssm_prep(SsmP p) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.y, sl = p.slot[t], pos = p.pos[t], nr = p.taps - 1, C = p.C;
    if (blockIdx.x == gridDim.x - 1) {
        for (int h = threadIdx.x; h < p.H; h += blockDim.x) {
            const float dt = ss_softplus(p.proj[(size_t)t * p.ld + p.col_dt + h] + p.dt_bias[h]);
            p.dtd[(size_t)t * p.H + h] = make_float2(dt, expf(-expf(p.a_log[h]) * dt));
        }
        return;
    }
    const int c = (blockIdx.x * 256 + threadIdx.x) * V;
    if (c >= C) return;
    const float* row = p.proj + (size_t)t * p.ld + p.col_x + c;
    const float* ring = nr > 0 ? static_cast<const float*>(p.ring_addrs[sl]) + c : nullptr;
    // how many earlier rows of this step belong to the same sequence (at most taps - 1 matter)
    int back = 0;
    while (back < nr && t - back - 1 >= 0 && p.slot[t - back - 1] == sl) ++back;
    float acc[V];
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = p.conv_b[c + i];
    auto add = [&](const float* w, const float* x) {
        if constexpr (V == 4) {
            const float4 a = *reinterpret_cast<const float4*>(w), b = *reinterpret_cast<const float4*>(x);
            acc[0] = fmaf(a.x, b.x, acc[0]), acc[1] = fmaf(a.y, b.y, acc[1]), acc[2] = fmaf(a.z, b.z, acc[2]), acc[3] = fmaf(a.w, b.w, acc[3]);
        } else {
            acc[0] = fmaf(w[0], x[0], acc[0]);
        }
    };
    add(p.conv_w + (size_t)nr * C + c, row);
#pragma unroll 3
    for (int j = 1; j <= nr; ++j) {   // the input j positions back
        const int pj = pos - j;
        if (pj < 0) break;
        add(p.conv_w + (size_t)(nr - j) * C + c, j <= back ? row - (long long)j * p.ld : ring + (size_t)(pj % nr) * C);
    }
    float* dst = p.xbc + (size_t)t * C + c;
    if constexpr (V == 4) *reinterpret_cast<float4*>(dst) = make_float4(silu_f(acc[0]), silu_f(acc[1]), silu_f(acc[2]), silu_f(acc[3]));
    else dst[0] = silu_f(acc[0]);
}

// packed pairs of fp32
using f2 = unsigned long long;
__device__ __forceinline__ f2 f2_pack(float a, float b) {
    f2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 f2_unpack(f2 v) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f2 f2_fma(f2 a, f2 b, f2 c) {
    f2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
__device__ __forceinline__ f2 f2_mul(f2 a, f2 b) {
    f2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
template <int BYTES>
__device__ __forceinline__ void ss_cp_async(void* smem_dst, const void* gsrc) {
    if constexpr (BYTES == 16)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(smem_dst)), "l"(gsrc), "n"(BYTES) : "memory");
}

// the run's last taps - 1 inputs go into the slot's ring, by all CTAs of the run together (nobody reads it in this kernel)
__device__ __forceinline__ void ss_store_tails(const SsmP& p, int row0, int len, float* ring) {
    const int nr = p.taps - 1, n = min(nr, len);
    const int stride = gridDim.x * gridDim.y * blockDim.x;
    for (int i = (blockIdx.y * gridDim.x + blockIdx.x) * blockDim.x + threadIdx.x; i < n * p.C; i += stride) {
        const int j = i / p.C, c = i - j * p.C, row = row0 + len - 1 - j;
        ring[(size_t)(p.pos[row] % nr) * p.C + c] = p.proj[(size_t)row * p.ld + p.col_x + c];
    }
}

// grid (ceil(dv / 32), H, runs).  P: pieces per lane, the state is at most 16 P long.
template <int P>
__global__ void __launch_bounds__(kSsThreads) k_ssm_scan(SsmP p) {
    constexpr int NP = P * kSsLanes * 4, PER = 2 * NP + kSsCols + 4;   // staged per token: B | C | x | dt, decay
    extern __shared__ __align__(16) float ssm[];   // [2][kSsChunk][PER]
    pdl_trigger();
    pdl_wait();
    const int run = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, N = p.N;
    const int row0 = p.run_row0[run], len = p.run_len[run];
    if (len <= 0) return;
    const int q = tid & (kSsLanes - 1), col = tid / kSsLanes, j0 = blockIdx.x * kSsCols, j = j0 + col;
    const bool mine = j < p.dv;   // the lanes of a channel agree
    const int sl = p.slot[row0];
    const int inner = p.H * p.dv, g = h / (p.H / p.G), ncol = min(kSsCols, p.dv - j0);
    const float* sB = p.xbc + (size_t)row0 * p.C + inner + (size_t)g * N;
    const float* sX = p.xbc + (size_t)row0 * p.C + (size_t)h * p.dv + j0;
    const size_t c_off = (size_t)p.G * N;   // from a group's B to its C
    if (NP > N) {   // padding of the staged vectors: zero, never written again
        const int pad = NP - N;
        for (int i = tid; i < 2 * kSsChunk * 2 * pad; i += kSsThreads) {
            const int v = i / pad, e = i - v * pad;   // v: (buffer, token, B or C)
            ssm[(size_t)(v >> 1) * PER + (v & 1) * NP + N + e] = 0.f;
        }
    }
    auto stage = [&](int buf, int c0) {
        const int cn = min(kSsChunk, len - c0);
        float* dst0 = ssm + (size_t)buf * kSsChunk * PER;
        const int unit = p.vec ? 4 : 1, nb = N / unit, nx = ncol / unit, items = 2 * nb + nx + 1;
        for (int i = tid; i < cn * items; i += kSsThreads) {
            const int tt = i / items, e = i - tt * items;
            float* dst = dst0 + (size_t)tt * PER;
            const size_t tok = (size_t)(c0 + tt) * p.C;
            if (e == items - 1) {
                ss_cp_async<8>(dst + 2 * NP + kSsCols, p.dtd + (size_t)(row0 + c0 + tt) * p.H + h);
                continue;
            }
            const float* src;
            if (e < nb) src = sB + tok + e * unit, dst += e * unit;
            else if (e < 2 * nb) src = sB + c_off + tok + (e - nb) * unit, dst += NP + (e - nb) * unit;
            else src = sX + tok + (e - 2 * nb) * unit, dst += 2 * NP + (e - 2 * nb) * unit;
            if (p.vec) ss_cp_async<16>(dst, src);
            else ss_cp_async<4>(dst, src);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float* sg = static_cast<float*>(p.state_addrs[sl]) + ((size_t)h * p.dv + (mine ? j : 0)) * N;
    const bool fresh = p.pos[row0] == 0, n4 = (N & 3) == 0;
    f2 S[2 * P];
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int k = (kSsLanes * i + q) * 4;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (mine && !fresh) {
            if (n4) {
                if (k < N) v = *reinterpret_cast<const float4*>(sg + k);
            } else {
                if (k < N) v.x = sg[k];
                if (k + 1 < N) v.y = sg[k + 1];
                if (k + 2 < N) v.z = sg[k + 2];
                if (k + 3 < N) v.w = sg[k + 3];
            }
        }
        S[2 * i] = f2_pack(v.x, v.y), S[2 * i + 1] = f2_pack(v.z, v.w);
    }
    if (p.taps > 1) ss_store_tails(p, row0, len, static_cast<float*>(p.ring_addrs[sl]));
    const float skip = p.d_skip[h];
    float* optr = p.o + (size_t)row0 * p.ld_o + (size_t)h * p.dv + j;
    int buf = 0;
    for (int c0 = 0; c0 < len; c0 += kSsChunk, buf ^= 1) {
        const int cn = min(kSsChunk, len - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // this chunk has landed for every thread; the other half is no longer read
        if (c0 + kSsChunk < len) stage(buf ^ 1, c0 + kSsChunk);
        const float* tv = ssm + (size_t)buf * kSsChunk * PER;
#pragma unroll 2
        for (int tt = 0; tt < cn; ++tt, tv += PER, optr += p.ld_o) {
            const float x = mine ? tv[2 * NP + col] : 0.f;
            const float2 dd = *reinterpret_cast<const float2*>(tv + 2 * NP + kSsCols);
            const f2 v2 = f2_pack(dd.x * x, dd.x * x), d2 = f2_pack(dd.y, dd.y);
            const ulonglong2* mB = reinterpret_cast<const ulonglong2*>(tv) + q;
            const ulonglong2* mC = reinterpret_cast<const ulonglong2*>(tv + NP) + q;
            f2 o0 = 0ull, o1 = 0ull;
#pragma unroll
            for (int i = 0; i < P; ++i) {
                const ulonglong2 b = mB[kSsLanes * i], c = mC[kSsLanes * i];
                S[2 * i] = f2_fma(b.x, v2, f2_mul(d2, S[2 * i]));
                S[2 * i + 1] = f2_fma(b.y, v2, f2_mul(d2, S[2 * i + 1]));
                o0 = f2_fma(c.x, S[2 * i], o0);
                o1 = f2_fma(c.y, S[2 * i + 1], o1);
            }
            const float2 a = f2_unpack(o0), b = f2_unpack(o1);
            float out = (a.x + a.y) + (b.x + b.y);
#pragma unroll
            for (int m = 1; m < kSsLanes; m <<= 1) out += __shfl_xor_sync(0xffffffffu, out, m);
            if (mine && q == 0) *optr = fmaf(skip, x, out);
        }
    }
    if (!mine) return;
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int k = (kSsLanes * i + q) * 4;
        const float2 a = f2_unpack(S[2 * i]), b = f2_unpack(S[2 * i + 1]);
        if (n4) {
            if (k < N) *reinterpret_cast<float4*>(sg + k) = make_float4(a.x, a.y, b.x, b.y);
        } else {
            if (k < N) sg[k] = a.x;
            if (k + 1 < N) sg[k + 1] = a.y;
            if (k + 2 < N) sg[k + 2] = b.x;
            if (k + 3 < N) sg[k + 3] = b.y;
        }
    }
}

// any state size: one thread per channel, grid (ceil(dv / 32), H, runs), 32 threads
__global__ void __launch_bounds__(32) k_ssm_scan_any(SsmP p) {
    extern __shared__ float st[];   // [N][32]
    pdl_trigger();
    pdl_wait();
    const int run = blockIdx.z, h = blockIdx.y, lane = threadIdx.x, j = blockIdx.x * 32 + lane, N = p.N;
    const int row0 = p.run_row0[run], len = p.run_len[run];
    if (len <= 0) return;
    const int sl = p.slot[row0], inner = p.H * p.dv, g = h / (p.H / p.G);
    const bool mine = j < p.dv, fresh = p.pos[row0] == 0;
    float* sg = static_cast<float*>(p.state_addrs[sl]) + ((size_t)h * p.dv + (mine ? j : 0)) * N;
    for (int k = 0; k < N; ++k) st[k * 32 + lane] = mine && !fresh ? sg[k] : 0.f;
    if (p.taps > 1) ss_store_tails(p, row0, len, static_cast<float*>(p.ring_addrs[sl]));
    for (int i = 0; i < len; ++i) {
        const float* row = p.xbc + (size_t)(row0 + i) * p.C;
        const float* B = row + inner + (size_t)g * N;
        const float* Cv = B + (size_t)p.G * N;
        const float2 dd = p.dtd[(size_t)(row0 + i) * p.H + h];
        const float x = mine ? row[(size_t)h * p.dv + j] : 0.f, v = dd.x * x;
        float out = 0.f;
        for (int k = 0; k < N; ++k) {
            const float s = fmaf(B[k], v, dd.y * st[k * 32 + lane]);
            st[k * 32 + lane] = s;
            out = fmaf(Cv[k], s, out);
        }
        if (mine) p.o[(size_t)(row0 + i) * p.ld_o + (size_t)h * p.dv + j] = fmaf(p.d_skip[h], x, out);
    }
    if (mine)
        for (int k = 0; k < N; ++k) sg[k] = st[k * 32 + lane];
}

template <int P>
static int ssm_launch(const SsmP& p, int runs, bool pdl, cudaStream_t st) {
    constexpr size_t smem = (size_t)2 * kSsChunk * (2 * P * kSsLanes * 4 + kSsCols + 4) * sizeof(float);
    if (smem > 48 * 1024) {
        static bool set = false;
        if (!set) {
            ZL_CHECK_CUDA(cudaFuncSetAttribute(k_ssm_scan<P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            set = true;
        }
    }
    ZL_CHECK_CUDA(launch(k_ssm_scan<P>, dim3(cdiv(p.dv, kSsCols), p.H, runs), dim3(kSsThreads), smem, st, pdl, p));
    return ZL_OK;
}

// y[t] = w * v / sqrt(mean(v^2) + eps) in equal parts, v = o silu(z).  grid (groups, T); the first 8 values of a thread stay in
// registers between the passes.
template <typename TO>
__global__ void __launch_bounds__(512) k_silu_gate_group_rmsnorm(const float* __restrict__ o, long long ldo,
                                                                 const float* __restrict__ z, long long ldz,
                                                                 const float* __restrict__ w, TO* __restrict__ y, long long ldy,
                                                                 int gs, float eps) {
    __shared__ float red[16];
    pdl_trigger();
    pdl_wait();
    const int c0 = blockIdx.x * gs, n = blockDim.x;
    const float *orow = o + (size_t)blockIdx.y * ldo + c0, *zr = z + (size_t)blockIdx.y * ldz + c0;
    float keep[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = threadIdx.x + i * n;
        keep[i] = c < gs ? orow[c] * silu_f(zr[c]) : 0.f;
        ss = fmaf(keep[i], keep[i], ss);
    }
    for (int c = threadIdx.x + 8 * n; c < gs; c += n) {
        const float v = orow[c] * silu_f(zr[c]);
        ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < n >> 5; ++i) tot += red[i];
    const float r = 1.0f / sqrtf(tot / (float)gs + eps);
    TO* yr = y + (size_t)blockIdx.y * ldy + c0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = threadIdx.x + i * n;
        if (c < gs) yr[c] = from_f32<TO>(keep[i] * r * w[c0 + c]);
    }
    for (int c = threadIdx.x + 8 * n; c < gs; c += n) yr[c] = from_f32<TO>(orow[c] * silu_f(zr[c]) * r * w[c0 + c]);
}

}  // namespace zl

using namespace zl;

extern "C" size_t zl_ssm_workspace_bytes(int T, int heads, int vdim, int state, int groups) {
    const size_t c = (size_t)heads * vdim + 2 * (size_t)groups * state;
    return (((size_t)T * c + 3) / 4 * 4 + (size_t)T * heads * 2) * sizeof(float);
}

extern "C" int zl_ssm_prepare(int vdim, int state) {
    ZL_CHECK_ARG(vdim > 0 && state > 0);
    ZL_CHECK_SUPPORTED(state <= 256 || (size_t)state * 32 * sizeof(float) <= 200 * 1024);
    return ZL_OK;
}

extern "C" int zl_ssm_scan(const float* proj, long long ld, int col_x, int col_dt, const float* conv_weight, const float* conv_bias,
                           int taps, const float* dt_bias, const float* a_log, const float* d_skip, void* const* ring_addrs,
                           const int32_t* run_row0, const int32_t* run_len, int runs, const int32_t* slot, const int32_t* pos,
                           void* const* state_addrs, float* o, long long ld_o, int heads, int vdim, int state, int groups, int T,
                           void* workspace, size_t workspace_bytes, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(proj && conv_weight && conv_bias && dt_bias && a_log && d_skip && run_row0 && run_len && slot && pos && state_addrs && o);
    ZL_CHECK_ARG(taps >= 1 && (taps == 1 || ring_addrs) && heads > 0 && groups > 0 && heads % groups == 0 && vdim > 0 && state > 0);
    ZL_CHECK_ARG(runs > 0 && runs <= 65535 && heads <= 65535 && T > 0 && T <= 65535 && col_x >= 0 && col_dt >= 0);
    ZL_CHECK_ARG(workspace && workspace_bytes >= zl_ssm_workspace_bytes(T, heads, vdim, state, groups));
    if (int rc = zl_ssm_prepare(vdim, state)) return rc;
    const int inner = heads * vdim, C = inner + 2 * groups * state;
    ZL_CHECK_ARG(ld >= col_x + C && ld >= col_dt + heads && ld_o >= inner);
    float* xbc = static_cast<float*>(workspace);
    SsmP p{proj, ld, col_x, col_dt, conv_weight, conv_bias, taps, dt_bias, a_log, d_skip, ring_addrs, run_row0, run_len, slot, pos,
           state_addrs, o, ld_o, heads, vdim, state, groups, C, xbc, reinterpret_cast<float2*>(xbc + ((size_t)T * C + 3) / 4 * 4), 0};
    auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
    ZL_CHECK_ARG(al16(workspace));
    p.vec = C % 4 == 0 && inner % 4 == 0 && vdim % 4 == 0 && state % 4 == 0;
    const bool v4 = C % 4 == 0 && ld % 4 == 0 && col_x % 4 == 0 && al16(proj) && al16(conv_weight);
    const dim3 grid(cdiv(C, 256 * (v4 ? 4 : 1)) + 1, T);
    if (v4) ZL_CHECK_CUDA(launch(k_ssm_prep<4>, grid, dim3(256), 0, stream, pdl != 0, p));
    else ZL_CHECK_CUDA(launch(k_ssm_prep<1>, grid, dim3(256), 0, stream, pdl != 0, p));
    switch (state <= 128 ? (state + 15) / 16 : (state <= 192 ? 12 : (state <= 256 ? 16 : 0))) {
        case 1: return ssm_launch<1>(p, runs, pdl != 0, stream);
        case 2: return ssm_launch<2>(p, runs, pdl != 0, stream);
        case 3: return ssm_launch<3>(p, runs, pdl != 0, stream);
        case 4: return ssm_launch<4>(p, runs, pdl != 0, stream);
        case 5: return ssm_launch<5>(p, runs, pdl != 0, stream);
        case 6: return ssm_launch<6>(p, runs, pdl != 0, stream);
        case 7: return ssm_launch<7>(p, runs, pdl != 0, stream);
        case 8: return ssm_launch<8>(p, runs, pdl != 0, stream);
        case 12: return ssm_launch<12>(p, runs, pdl != 0, stream);
        case 16: return ssm_launch<16>(p, runs, pdl != 0, stream);
        default: break;
    }
    const size_t smem = (size_t)state * 32 * sizeof(float);
    static size_t set_for = 0;
    if (smem > 48 * 1024 && smem > set_for) {
        ZL_CHECK_CUDA(cudaFuncSetAttribute(k_ssm_scan_any, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set_for = smem;
    }
    ZL_CHECK_CUDA(launch(k_ssm_scan_any, dim3(cdiv(vdim, 32), heads, runs), dim3(32), smem, stream, pdl != 0, p));
    return ZL_OK;
}

extern "C" int zl_silu_gate_group_rmsnorm(const float* o, long long ldo, const float* z, long long ldz, const float* weight, void* y,
                                          long long ldy, int T, int D, int groups, float eps, int out_dtype, int pdl,
                                          zl_stream_t stream) {
    ZL_CHECK_ARG(o && z && weight && y && T > 0 && T <= 65535 && D > 0 && groups > 0 && D % groups == 0);
    ZL_CHECK_ARG(ldo >= D && ldz >= D && ldy >= D && (out_dtype == ZL_F16 || out_dtype == ZL_BF16 || out_dtype == ZL_F32));
    const int gs = D / groups;
    const dim3 grid(groups, T), block(gs >= 2048 ? 512 : (gs >= 512 ? 256 : 128));
    cudaError_t e;
    if (out_dtype == ZL_F32)
        e = launch(k_silu_gate_group_rmsnorm<float>, grid, block, 0, stream, pdl != 0, o, ldo, z, ldz, weight, (float*)y, ldy, gs, eps);
    else if (out_dtype == ZL_BF16)
        e = launch(k_silu_gate_group_rmsnorm<__nv_bfloat16>, grid, block, 0, stream, pdl != 0, o, ldo, z, ldz, weight, (__nv_bfloat16*)y,
                   ldy, gs, eps);
    else
        e = launch(k_silu_gate_group_rmsnorm<__half>, grid, block, 0, stream, pdl != 0, o, ldo, z, ldz, weight, (__half*)y, ldy, gs, eps);
    ZL_CHECK_CUDA(e);
    return ZL_OK;
}
