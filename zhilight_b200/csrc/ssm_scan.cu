// Selective state space (the state-space duality form): a recurrent mixer whose state per head is a (vdim, state) fp32 matrix,
//   S_t = exp(-exp(a_log) dt_t) S_(t-1) + (dt_t x_t) B_t^T,      o_t = S_t C_t + d_skip x_t,
// one scalar decay per head and token, B and C shared by the heads of a group, dt_t = softplus(logit + bias).  x, B and C come
// out of a causal convolution per channel (the last taps - 1 inputs of a sequence are kept per slot) and silu.
//
// k_ssm_prep: convolution, silu, step sizes and decays of all rows of the step at once.  k_ssm_scan: a row of S (one value
// channel) depends on its own past and the token's vectors only; it is walked through the tokens of its sequence in order, so a
// token's result does not depend on how the sequence was cut into steps or on the rest of the step.  A CTA owns 32 channels of
// one head of one run; two channels' states live in the registers of eight adjacent lanes, in 4-element pieces f = 8 i + q of the
// state dimension, updated and read out with packed fp32 pairs.  The token vectors fly into shared memory chunk by chunk ahead
// of use.  k_ssm_step: the same for one token per sequence, straight from and to the states.  State sizes above 256 take
// k_ssm_scan_any (state in shared memory, one thread per channel).  A run that starts at position 0 starts from a zero state (a
// slot given to a new sequence needs no clearing); the final state and the convolution's last inputs go back to the slot.
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

constexpr int kSsChunk = 16, kSsCols = 32, kSsThreads = 128;

__device__ __forceinline__ float ss_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

template <int V>
struct SsVec {
    float v[V];
};
template <int V>
__device__ __forceinline__ SsVec<V> ss_load(const float* p) {
    SsVec<V> r;
    if constexpr (V == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        r.v[0] = a.x, r.v[1] = a.y, r.v[2] = a.z, r.v[3] = a.w;
    } else {
        r.v[0] = p[0];
    }
    return r;
}

// grid (channel blocks + 1, ceil(T / ROWS)); the last block computes the heads' step sizes.  V channels per thread (4: 16-byte
// rows).  TAPS > 0: that many taps, a thread's rows and the ones before them are loaded once, all in flight; 0: any number, read
// back row by row.  An earlier input is a row of this step if that belongs to the same sequence, else the slot's ring, else
// (before the start) zero.
template <int V, int TAPS, int ROWS>
__global__ void __launch_bounds__(256) k_ssm_prep(SsmP p, int T) {
    pdl_trigger();
    pdl_wait();
    constexpr int NR = TAPS > 0 ? TAPS - 1 : 0;
    const int t0 = blockIdx.y * ROWS, rows = min(ROWS, T - t0), nr = TAPS > 0 ? NR : p.taps - 1, C = p.C;
    if (blockIdx.x == gridDim.x - 1) {
        for (int i = threadIdx.x; i < rows * p.H; i += blockDim.x) {
            const int t = t0 + i / p.H, h = i % p.H;
            const float dt = ss_softplus(p.proj[(size_t)t * p.ld + p.col_dt + h] + p.dt_bias[h]);
            p.dtd[(size_t)t * p.H + h] = make_float2(dt, expf(-expf(p.a_log[h]) * dt));
        }
        return;
    }
    const int c = (blockIdx.x * 256 + threadIdx.x) * V;
    if (c >= C) return;
    const float* src = p.proj + p.col_x + c;
    const SsVec<V> bias = ss_load<V>(p.conv_b + c);
    SsVec<V> w[TAPS > 0 ? TAPS : 1], x[NR + ROWS];   // x[NR + i]: row t0 + i
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = ss_load<V>(p.conv_w + (size_t)j * C + c);
#pragma unroll
    for (int i = 0; i < NR + ROWS; ++i) {
        const int t = t0 + i - NR;
#pragma unroll
        for (int e = 0; e < V; ++e) x[i].v[e] = 0.f;
        if (t >= 0 && t < T) x[i] = ss_load<V>(src + (size_t)t * p.ld);
    }
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
        if (i >= rows) break;
        const int t = t0 + i, sl = p.slot[t], pos = p.pos[t];
        int back = 0;   // how many earlier rows of this step belong to the same sequence (at most taps - 1 matter)
        while (back < nr && t - back - 1 >= 0 && p.slot[t - back - 1] == sl) ++back;
        SsVec<V> acc = bias;
        auto add = [&](const SsVec<V>& a, const SsVec<V>& v) {
#pragma unroll
            for (int e = 0; e < V; ++e) acc.v[e] = fmaf(a.v[e], v.v[e], acc.v[e]);
        };
        auto stored = [&](int j) { return ss_load<V>(static_cast<const float*>(p.ring_addrs[sl]) + (size_t)((pos - j) % nr) * C + c); };
        if constexpr (TAPS > 0) {
            add(w[NR], x[NR + i]);
#pragma unroll
            for (int j = 1; j <= NR; ++j) {
                if (j <= back) add(w[NR - j], x[NR + i - j]);
                else if (pos >= j) add(w[NR - j], stored(j));
            }
        } else {
            add(ss_load<V>(p.conv_w + (size_t)nr * C + c), x[i]);
            for (int j = 1; j <= nr && j <= pos; ++j)
                add(ss_load<V>(p.conv_w + (size_t)(nr - j) * C + c), j <= back ? ss_load<V>(src + (size_t)(t - j) * p.ld) : stored(j));
        }
        float* dst = p.xbc + (size_t)t * C + c;
        if constexpr (V == 4)
            *reinterpret_cast<float4*>(dst) = make_float4(silu_f(acc.v[0]), silu_f(acc.v[1]), silu_f(acc.v[2]), silu_f(acc.v[3]));
        else
            dst[0] = silu_f(acc.v[0]);
    }
}

template <int V, int ROWS>
static cudaError_t ssm_prep_launch(const SsmP& p, int T, bool pdl, cudaStream_t st) {
    const dim3 grid(cdiv(p.C, 256 * V) + 1, cdiv(T, ROWS)), block(256);
    switch (p.taps) {
        case 2: return launch(k_ssm_prep<V, 2, ROWS>, grid, block, 0, st, pdl, p, T);
        case 3: return launch(k_ssm_prep<V, 3, ROWS>, grid, block, 0, st, pdl, p, T);
        case 4: return launch(k_ssm_prep<V, 4, ROWS>, grid, block, 0, st, pdl, p, T);
        default: return launch(k_ssm_prep<V, 0, ROWS>, grid, block, 0, st, pdl, p, T);
    }
}
template <int V>
static cudaError_t ssm_prep_launch(const SsmP& p, int T, bool pdl, cudaStream_t st) {
    return T > 64 ? ssm_prep_launch<V, 4>(p, T, pdl, st) : ssm_prep_launch<V, 1>(p, T, pdl, st);
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

// grid (ceil(dv / 32), H, runs).  LANES adjacent lanes share CE channels: a lane holds P pieces of each of them (the state is at
// most 4 P LANES long), so that a staged piece of B or C serves CE channels.
template <int P, int LANES, int CE>
__global__ void __launch_bounds__(kSsThreads) k_ssm_scan(SsmP p) {
    static_assert(kSsThreads / LANES * CE == kSsCols && 4 * CE == LANES, "a lane per (token, channel) of a group of four tokens");
    constexpr int NP = P * LANES * 4, PER = 2 * NP + kSsCols + 4;   // staged per token: B | C | x | dt, decay
    extern __shared__ __align__(16) float ssm[];   // [2][kSsChunk][PER]
    pdl_trigger();
    pdl_wait();
    const int run = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, N = p.N;
    const int row0 = p.run_row0[run], len = p.run_len[run];
    if (len <= 0) return;
    const int q = tid & (LANES - 1), col = tid / LANES * CE, j0 = blockIdx.x * kSsCols, j = j0 + col;
    const int sl = p.slot[row0];
    const int inner = p.H * p.dv, g = h / (p.H / p.G), ncol = min(kSsCols, p.dv - j0);
    const float* sB = p.xbc + (size_t)row0 * p.C + inner + (size_t)g * N;
    const float* sX = p.xbc + (size_t)row0 * p.C + (size_t)h * p.dv + j0;
    const size_t c_off = (size_t)p.G * N;   // from a group's B to its C
    // padding of the staged vectors: zero, never written again
    if (NP > N) {
        const int pad = NP - N;
        for (int i = tid; i < 2 * kSsChunk * 2 * pad; i += kSsThreads) {
            const int v = i / pad, e = i - v * pad;   // v: (buffer, token, B or C)
            ssm[(size_t)(v >> 1) * PER + (v & 1) * NP + N + e] = 0.f;
        }
    }
    if (ncol < kSsCols) {
        const int pad = kSsCols - ncol;
        for (int i = tid; i < 2 * kSsChunk * pad; i += kSsThreads) {
            const int v = i / pad, e = i - v * pad;
            ssm[(size_t)v * PER + 2 * NP + ncol + e] = 0.f;
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
    float* sg = static_cast<float*>(p.state_addrs[sl]) + ((size_t)h * p.dv + j) * N;
    const bool fresh = p.pos[row0] == 0, n4 = (N & 3) == 0;
    f2 S[CE][2 * P];
#pragma unroll
    for (int c = 0; c < CE; ++c)
#pragma unroll
        for (int i = 0; i < P; ++i) {
            const int k = (LANES * i + q) * 4;
            const float* src = sg + (size_t)c * N + k;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (j + c < p.dv && !fresh) {
                if (n4) {
                    if (k < N) v = *reinterpret_cast<const float4*>(src);
                } else {
                    if (k < N) v.x = src[0];
                    if (k + 1 < N) v.y = src[1];
                    if (k + 2 < N) v.z = src[2];
                    if (k + 3 < N) v.w = src[3];
                }
            }
            S[c][2 * i] = f2_pack(v.x, v.y), S[c][2 * i + 1] = f2_pack(v.z, v.w);
        }
    if (p.taps > 1) ss_store_tails(p, row0, len, static_cast<float*>(p.ring_addrs[sl]));
    const float skip = p.d_skip[h];
    float* optr = p.o + (size_t)row0 * p.ld_o + (size_t)h * p.dv + j;
    // a token's update of the state and this lane's share of the read-outs
    auto token = [&](const float* tk, float* out) {
        const float2 dd = *reinterpret_cast<const float2*>(tk + 2 * NP + kSsCols);
        const f2 d2 = f2_pack(dd.y, dd.y);
        f2 v2[CE], o0[CE], o1[CE];
#pragma unroll
        for (int c = 0; c < CE; ++c) {
            const float v = dd.x * tk[2 * NP + col + c];
            v2[c] = f2_pack(v, v);
            o0[c] = o1[c] = 0ull;
        }
        const ulonglong2* mB = reinterpret_cast<const ulonglong2*>(tk) + q;
        const ulonglong2* mC = reinterpret_cast<const ulonglong2*>(tk + NP) + q;
#pragma unroll
        for (int i = 0; i < P; ++i) {
            const ulonglong2 b = mB[LANES * i], r = mC[LANES * i];
#pragma unroll
            for (int c = 0; c < CE; ++c) {
                S[c][2 * i] = f2_fma(b.x, v2[c], f2_mul(d2, S[c][2 * i]));
                S[c][2 * i + 1] = f2_fma(b.y, v2[c], f2_mul(d2, S[c][2 * i + 1]));
                o0[c] = f2_fma(r.x, S[c][2 * i], o0[c]);
                o1[c] = f2_fma(r.y, S[c][2 * i + 1], o1[c]);
            }
        }
#pragma unroll
        for (int c = 0; c < CE; ++c) {
            const float2 a = f2_unpack(o0[c]), b = f2_unpack(o1[c]);
            out[c] = (a.x + a.y) + (b.x + b.y);
        }
    };
    int buf = 0;
    for (int c0 = 0; c0 < len; c0 += kSsChunk, buf ^= 1) {
        const int cn = min(kSsChunk, len - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // this chunk has landed for every thread; the other half is no longer read
        if (c0 + kSsChunk < len) stage(buf ^ 1, c0 + kSsChunk);
        const float* tv = ssm + (size_t)buf * kSsChunk * PER;
        int tt = 0;
        // four tokens at a time: the sums over the lanes are finished together, each round of shuffles halving the values a lane
        // carries, until lane q holds the one of token q / CE and channel q % CE.  A sum's order is that of the single-token form.
        for (; tt + 4 <= cn; tt += 4, tv += 4 * PER, optr += 4 * p.ld_o) {
            float val[LANES];
#pragma unroll
            for (int k = 0; k < 4; ++k) token(tv + k * PER, val + k * CE);
#pragma unroll
            for (int m = 1; m < LANES; m <<= 1) {
                const bool up = q & m;
#pragma unroll
                for (int i = 0; i < LANES / (2 * m); ++i) {
                    const float keep = up ? val[2 * i + 1] : val[2 * i], send = up ? val[2 * i] : val[2 * i + 1];
                    val[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                }
            }
            const int k = q / CE, c = q % CE;
            if (j + c < p.dv) optr[k * p.ld_o + c] = fmaf(skip, tv[k * PER + 2 * NP + col + c], val[0]);
        }
        for (; tt < cn; ++tt, tv += PER, optr += p.ld_o) {
            float val[CE];
            token(tv, val);
#pragma unroll
            for (int c = 0; c < CE; ++c) {
#pragma unroll
                for (int m = 1; m < LANES; m <<= 1) val[c] += __shfl_xor_sync(0xffffffffu, val[c], m);
                if (q == c && j + c < p.dv) optr[c] = fmaf(skip, tv[2 * NP + col + c], val[c]);
            }
        }
    }
#pragma unroll
    for (int c = 0; c < CE; ++c) {
        if (j + c >= p.dv) continue;
#pragma unroll
        for (int i = 0; i < P; ++i) {
            const int k = (LANES * i + q) * 4;
            float* dst = sg + (size_t)c * N + k;
            const float2 a = f2_unpack(S[c][2 * i]), b = f2_unpack(S[c][2 * i + 1]);
            if (n4) {
                if (k < N) *reinterpret_cast<float4*>(dst) = make_float4(a.x, a.y, b.x, b.y);
            } else {
                if (k < N) dst[0] = a.x;
                if (k + 1 < N) dst[1] = a.y;
                if (k + 2 < N) dst[2] = b.x;
                if (k + 3 < N) dst[3] = b.y;
            }
        }
    }
}

// One token per sequence (decode steps): the state is read, updated, read out and written once, every load independent.  Eight
// lanes per channel in the pieces and the order of sums of k_ssm_scan.  grid (ceil(dv / 16), H, runs)
template <int P>
__global__ void __launch_bounds__(128) k_ssm_step(SsmP p) {
    constexpr int LANES = 8;
    pdl_trigger();
    pdl_wait();
    const int run = blockIdx.z, h = blockIdx.y, N = p.N, q = threadIdx.x & (LANES - 1), j = blockIdx.x * 16 + (threadIdx.x >> 3);
    if (p.run_len[run] <= 0) return;
    const int row = p.run_row0[run], sl = p.slot[row], inner = p.H * p.dv, g = h / (p.H / p.G);
    const bool mine = j < p.dv, fresh = p.pos[row] == 0;
    const float* xr = p.xbc + (size_t)row * p.C;
    const float *B = xr + inner + (size_t)g * N, *Cv = B + (size_t)p.G * N;
    float* sg = static_cast<float*>(p.state_addrs[sl]) + ((size_t)h * p.dv + (mine ? j : 0)) * N;
    float S[P][4], b[P][4], r[P][4];
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int k = (LANES * i + q) * 4;
        if (p.vec) {   // whole pieces
            const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 s4 = k < N && mine && !fresh ? *reinterpret_cast<const float4*>(sg + k) : z;
            const float4 b4 = k < N ? *reinterpret_cast<const float4*>(B + k) : z, r4 = k < N ? *reinterpret_cast<const float4*>(Cv + k) : z;
            S[i][0] = s4.x, S[i][1] = s4.y, S[i][2] = s4.z, S[i][3] = s4.w;
            b[i][0] = b4.x, b[i][1] = b4.y, b[i][2] = b4.z, b[i][3] = b4.w;
            r[i][0] = r4.x, r[i][1] = r4.y, r[i][2] = r4.z, r[i][3] = r4.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const bool in = k + e < N;
                S[i][e] = in && mine && !fresh ? sg[k + e] : 0.f;
                b[i][e] = in ? B[k + e] : 0.f;
                r[i][e] = in ? Cv[k + e] : 0.f;
            }
        }
    }
    if (p.taps > 1) ss_store_tails(p, row, 1, static_cast<float*>(p.ring_addrs[sl]));
    const float2 dd = p.dtd[(size_t)row * p.H + h];
    const float x = mine ? xr[(size_t)h * p.dv + j] : 0.f, v = dd.x * x;
    float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int i = 0; i < P; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            S[i][e] = fmaf(b[i][e], v, dd.y * S[i][e]);
            o[e] = fmaf(r[i][e], S[i][e], o[e]);
        }
    float out = (o[0] + o[1]) + (o[2] + o[3]);
#pragma unroll
    for (int m = 1; m < LANES; m <<= 1) out += __shfl_xor_sync(0xffffffffu, out, m);
    if (!mine) return;
    if (q == 0) p.o[(size_t)row * p.ld_o + (size_t)h * p.dv + j] = fmaf(p.d_skip[h], x, out);
#pragma unroll
    for (int i = 0; i < P; ++i) {
        const int k = (LANES * i + q) * 4;
        if (p.vec) {
            if (k < N) *reinterpret_cast<float4*>(sg + k) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (k + e < N) sg[k + e] = S[i][e];
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

template <int P, int LANES, int CE>
static int ssm_launch(const SsmP& p, int runs, bool pdl, cudaStream_t st) {
    constexpr size_t smem = (size_t)2 * kSsChunk * (2 * P * LANES * 4 + kSsCols + 4) * sizeof(float);
    if (smem > 48 * 1024) {
        static bool set = false;
        if (!set) {
            ZL_CHECK_CUDA(cudaFuncSetAttribute(k_ssm_scan<P, LANES, CE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            set = true;
        }
    }
    ZL_CHECK_CUDA(launch(k_ssm_scan<P, LANES, CE>, dim3(cdiv(p.dv, kSsCols), p.H, runs), dim3(kSsThreads), smem, st, pdl, p));
    return ZL_OK;
}

// y[t] = w * v / sqrt(mean(v^2) + eps) in equal parts, v = o silu(z).  One CTA per (token, part): grid (groups, T); the first 8
// values of a thread stay in registers between the passes.
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

// The same with a warp per (token, part) for parts of at most 1024 values in 16-byte pieces: no barrier, every load in flight.
// grid (ceil(groups / 8), T), 8 warps
template <typename TO, int PIECES>
__global__ void __launch_bounds__(256) k_silu_gate_group_rmsnorm_warp(const float* __restrict__ o, long long ldo,
                                                                      const float* __restrict__ z, long long ldz,
                                                                      const float* __restrict__ w, TO* __restrict__ y, long long ldy,
                                                                      int groups, int gs, float eps) {
    pdl_trigger();
    pdl_wait();
    const int g = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, c0 = g * gs;
    if (g >= groups) return;
    const float *orow = o + (size_t)blockIdx.y * ldo + c0, *zr = z + (size_t)blockIdx.y * ldz + c0;
    float4 keep[PIECES];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
        const int c = (lane + 32 * i) * 4;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
        if (c < gs) a = *reinterpret_cast<const float4*>(orow + c), b = *reinterpret_cast<const float4*>(zr + c);
        keep[i] = make_float4(a.x * silu_f(b.x), a.y * silu_f(b.y), a.z * silu_f(b.z), a.w * silu_f(b.w));
        ss = fmaf(keep[i].x, keep[i].x, fmaf(keep[i].y, keep[i].y, fmaf(keep[i].z, keep[i].z, fmaf(keep[i].w, keep[i].w, ss))));
    }
    const float r = 1.0f / sqrtf(warp_sum(ss) / (float)gs + eps);
    TO* yr = y + (size_t)blockIdx.y * ldy + c0;
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
        const int c = (lane + 32 * i) * 4;
        if (c >= gs) continue;
        const float4 wv = *reinterpret_cast<const float4*>(w + c0 + c);
        TO v[4] = {from_f32<TO>(keep[i].x * r * wv.x), from_f32<TO>(keep[i].y * r * wv.y), from_f32<TO>(keep[i].z * r * wv.z),
                   from_f32<TO>(keep[i].w * r * wv.w)};
        if constexpr (sizeof(TO) == 4) *reinterpret_cast<float4*>(yr + c) = *reinterpret_cast<const float4*>(v);
        else *reinterpret_cast<uint2*>(yr + c) = *reinterpret_cast<const uint2*>(v);
    }
}

template <typename TO>
static cudaError_t silu_gate_launch(const float* o, long long ldo, const float* z, long long ldz, const float* w, TO* y, long long ldy,
                                    int T, int groups, int gs, float eps, bool pdl, cudaStream_t st) {
    auto al = [](const void* q, int b) { return (reinterpret_cast<uintptr_t>(q) & (b - 1)) == 0; };
    // (few tokens have no warps to spare: a CTA per part)
    if (T > 64 && gs % 4 == 0 && gs <= 1024 && ldo % 4 == 0 && ldz % 4 == 0 && ldy % 4 == 0 && al(o, 16) && al(z, 16) && al(w, 16) &&
        al(y, 4 * (int)sizeof(TO))) {
        const dim3 grid(cdiv(groups, 8), T), block(256);
        if (gs <= 256) return launch(k_silu_gate_group_rmsnorm_warp<TO, 2>, grid, block, 0, st, pdl, o, ldo, z, ldz, w, y, ldy, groups, gs, eps);
        if (gs <= 512) return launch(k_silu_gate_group_rmsnorm_warp<TO, 4>, grid, block, 0, st, pdl, o, ldo, z, ldz, w, y, ldy, groups, gs, eps);
        return launch(k_silu_gate_group_rmsnorm_warp<TO, 8>, grid, block, 0, st, pdl, o, ldo, z, ldz, w, y, ldy, groups, gs, eps);
    }
    return launch(k_silu_gate_group_rmsnorm<TO>, dim3(groups, T), dim3(gs >= 2048 ? 512 : (gs >= 512 ? 256 : 128)), 0, st, pdl, o, ldo, z,
                  ldz, w, y, ldy, gs, eps);
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
    ZL_CHECK_CUDA(v4 ? ssm_prep_launch<4>(p, T, pdl != 0, stream) : ssm_prep_launch<1>(p, T, pdl != 0, stream));
    if (runs == T && state <= 256) {   // a token per sequence
        const dim3 grid(cdiv(vdim, 16), heads, runs), block(128);
        if (state <= 32) ZL_CHECK_CUDA(launch(k_ssm_step<1>, grid, block, 0, stream, pdl != 0, p));
        else if (state <= 64) ZL_CHECK_CUDA(launch(k_ssm_step<2>, grid, block, 0, stream, pdl != 0, p));
        else if (state <= 128) ZL_CHECK_CUDA(launch(k_ssm_step<4>, grid, block, 0, stream, pdl != 0, p));
        else ZL_CHECK_CUDA(launch(k_ssm_step<8>, grid, block, 0, stream, pdl != 0, p));
        return ZL_OK;
    }
    switch (state <= 128 ? (state + 31) / 32 : (state <= 192 ? 6 : (state <= 256 ? 8 : 0))) {
        case 1: return ssm_launch<1, 8, 2>(p, runs, pdl != 0, stream);
        case 2: return ssm_launch<2, 8, 2>(p, runs, pdl != 0, stream);
        case 3: return ssm_launch<3, 8, 2>(p, runs, pdl != 0, stream);
        case 4: return ssm_launch<4, 8, 2>(p, runs, pdl != 0, stream);
        case 6: return ssm_launch<6, 8, 2>(p, runs, pdl != 0, stream);
        case 8: return ssm_launch<8, 8, 2>(p, runs, pdl != 0, stream);
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
    cudaError_t e;
    if (out_dtype == ZL_F32) e = silu_gate_launch(o, ldo, z, ldz, weight, (float*)y, ldy, T, groups, gs, eps, pdl != 0, stream);
    else if (out_dtype == ZL_BF16)
        e = silu_gate_launch(o, ldo, z, ldz, weight, (__nv_bfloat16*)y, ldy, T, groups, gs, eps, pdl != 0, stream);
    else e = silu_gate_launch(o, ldo, z, ldz, weight, (__half*)y, ldy, T, groups, gs, eps, pdl != 0, stream);
    ZL_CHECK_CUDA(e);
    return ZL_OK;
}
