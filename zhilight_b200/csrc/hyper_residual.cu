// Residual of several copies of a token's vector ("streams") joined by hyper-connections, all in fp32.  One kernel takes a
// sublayer's result into every stream and reads the next sublayer's input:
//   y     = sum_p coef_p part_p + dense           (parts in the order of p: a token's experts, then the shared one)
//   x_s'  = sum_s mix[s, s'] x_s + out[s'] y      (all new streams from the old ones)
//   u     = sum_s in[s] x_s,   h = w * u / sqrt(mean(u^2) + eps)
// The embedding is the same kernel with every stream set to the scaled row.  One CTA per token; a thread owns 4-channel pieces
// (16-byte loads) when the rows allow it, so that every stream's load of a piece is independent of the others, and keeps its
// pieces of u in registers between the two passes.
#include "common.cuh"

namespace zl {

struct HyperP {
    float* x;                  // (T, S, D)
    const float* parts;        // n_parts rows per token, or null: no update
    long long ldp;
    const float* coef;         // (T, n_parts) or null: ones
    int n_parts;
    const float* dense;        // one more row per token, or null
    long long ldd;
    const float *mix, *out, *in;
    const int32_t* ids;        // embedding form: x_s[t] = scale * table[ids[t]]
    const void* table;
    int vocab;
    float scale;
    const float* next_w;
    void* h;
    float* u_out;
    int S, D;
    float eps;
};

constexpr int kHyMaxStreams = 16, kHyPieces = 4;

__device__ __forceinline__ float hy_block_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += red[i];
    return tot;
}
__device__ __forceinline__ float4 hy_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 hy_fma(float a, float4 v, float4 s) {
    return make_float4(fmaf(a, v.x, s.x), fmaf(a, v.y, s.y), fmaf(a, v.z, s.z), fmaf(a, v.w, s.w));
}
template <typename TO>
__device__ __forceinline__ void hy_store4(TO* dst, float a, float b, float c, float d) {
    if constexpr (sizeof(TO) == 4) {
        *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
    } else {
        TO v[4] = {from_f32<TO>(a), from_f32<TO>(b), from_f32<TO>(c), from_f32<TO>(d)};
        *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<const uint2*>(v);
    }
}

// SC: the number of streams when it is compiled, at most 4 (the 16-byte path)
template <typename TO, int SC>
__global__ void __launch_bounds__(512) k_hyper_vec(HyperP p) {
    __shared__ float red[16];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, D = p.D;
    float* xr = p.x + (size_t)t * SC * D;
    const float* pr = p.parts ? p.parts + (size_t)t * p.n_parts * p.ldp : nullptr;
    const float* dr = p.dense ? p.dense + (size_t)t * p.ldd : nullptr;
    const float* cf = p.coef ? p.coef + (size_t)t * p.n_parts : nullptr;
    const TO* er = nullptr;
    if (p.ids) {
        const int id = p.ids[t];
        er = static_cast<const TO*>(p.table) + (size_t)(id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id)) * D;
    }
    float in[SC];
#pragma unroll
    for (int s = 0; s < SC; ++s) in[s] = p.in ? __ldg(p.in + s) : 1.0f;
    float mix[SC][SC], out[SC];
    if (pr) {
#pragma unroll
        for (int s = 0; s < SC; ++s) {
            out[s] = __ldg(p.out + s);
#pragma unroll
            for (int q = 0; q < SC; ++q) mix[s][q] = __ldg(p.mix + s * SC + q);
        }
    }
    float4 u[kHyPieces];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kHyPieces; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= D) continue;
        float4 nx[SC];
        if (er) {
            const float4 e = make_float4(to_f32<TO>(er[c]) * p.scale, to_f32<TO>(er[c + 1]) * p.scale, to_f32<TO>(er[c + 2]) * p.scale,
                                         to_f32<TO>(er[c + 3]) * p.scale);
#pragma unroll
            for (int s = 0; s < SC; ++s) nx[s] = e;
        } else {
            float4 old[SC];
#pragma unroll
            for (int s = 0; s < SC; ++s) old[s] = hy_ld4(xr + (size_t)s * D + c);
            float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
            if (pr) {
#pragma unroll 4
                for (int q = 0; q < p.n_parts; ++q) y = hy_fma(cf ? cf[q] : 1.0f, hy_ld4(pr + (size_t)q * p.ldp + c), y);
                if (dr) y = hy_fma(1.0f, hy_ld4(dr + c), y);
#pragma unroll
                for (int q = 0; q < SC; ++q) {
                    float4 a = make_float4(out[q] * y.x, out[q] * y.y, out[q] * y.z, out[q] * y.w);
#pragma unroll
                    for (int s = 0; s < SC; ++s) a = hy_fma(mix[s][q], old[s], a);
                    nx[q] = a;
                }
            } else {
#pragma unroll
                for (int s = 0; s < SC; ++s) nx[s] = old[s];
            }
        }
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int s = 0; s < SC; ++s) {
            if (pr || er) *reinterpret_cast<float4*>(xr + (size_t)s * D + c) = nx[s];
            v = hy_fma(in[s], nx[s], v);
        }
        if (p.u_out) *reinterpret_cast<float4*>(p.u_out + (size_t)t * D + c) = v;
        u[i] = v;
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    if (!p.next_w) return;
    const float r = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)D + p.eps);
    TO* h = static_cast<TO*>(p.h) + (size_t)t * D;
#pragma unroll
    for (int i = 0; i < kHyPieces; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        if (c >= D) continue;
        const float4 w = hy_ld4(p.next_w + c);
        hy_store4<TO>(h + c, u[i].x * r * w.x, u[i].y * r * w.y, u[i].z * r * w.z, u[i].w * r * w.w);
    }
}

// any width and up to 16 streams, channel by channel; u waits in shared memory (D floats)
template <typename TO>
__global__ void __launch_bounds__(512) k_hyper_any(HyperP p) {
    extern __shared__ float su[];
    __shared__ float red[16];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, D = p.D, S = p.S;
    float* xr = p.x + (size_t)t * S * D;
    const float* pr = p.parts ? p.parts + (size_t)t * p.n_parts * p.ldp : nullptr;
    const float* cf = p.coef ? p.coef + (size_t)t * p.n_parts : nullptr;
    const TO* er = nullptr;
    if (p.ids) {
        const int id = p.ids[t];
        er = static_cast<const TO*>(p.table) + (size_t)(id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id)) * D;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < D; c += blockDim.x) {
        float v = 0.f, old[kHyMaxStreams];
        if (er) {
            const float e = to_f32<TO>(er[c]) * p.scale;
            for (int s = 0; s < S; ++s) {
                xr[(size_t)s * D + c] = e;
                v = fmaf(p.in ? p.in[s] : 1.0f, e, v);
            }
        } else {
#pragma unroll
            for (int s = 0; s < kHyMaxStreams; ++s) old[s] = s < S ? xr[(size_t)s * D + c] : 0.f;
            float y = 0.f;
            if (pr) {
                for (int q = 0; q < p.n_parts; ++q) y = fmaf(cf ? cf[q] : 1.0f, pr[(size_t)q * p.ldp + c], y);
                if (p.dense) y += p.dense[(size_t)t * p.ldd + c];
            }
            for (int q = 0; q < S; ++q) {
                float a = 0.f;
                if (pr) {
                    a = p.out[q] * y;
#pragma unroll
                    for (int s = 0; s < kHyMaxStreams; ++s)
                        if (s < S) a = fmaf(p.mix[s * S + q], old[s], a);
                    xr[(size_t)q * D + c] = a;
                } else {
                    a = xr[(size_t)q * D + c];
                }
                v = fmaf(p.in ? p.in[q] : 1.0f, a, v);
            }
        }
        if (p.u_out) p.u_out[(size_t)t * D + c] = v;
        su[c] = v;
        ss = fmaf(v, v, ss);
    }
    if (!p.next_w) return;
    const float r = 1.0f / sqrtf(hy_block_sum(ss, red) / (float)D + p.eps);
    TO* h = static_cast<TO*>(p.h) + (size_t)t * D;
    for (int c = threadIdx.x; c < D; c += blockDim.x) h[c] = from_f32<TO>(su[c] * r * p.next_w[c]);   // a thread reads what it wrote
}

template <typename TO>
static int hyper_launch_t(const HyperP& p, int T, bool pdl, cudaStream_t st) {
    auto al = [](const void* q, int b) { return (reinterpret_cast<uintptr_t>(q) & (b - 1)) == 0; };
    const int ab = 4 * (int)sizeof(TO);   // hy_store4 of the activation dtype
    const int D = p.D;
    const bool vec = p.S <= 4 && D % 4 == 0 && D <= 4 * 512 * kHyPieces && al(p.x, 16) &&
                     (!p.parts || (p.ldp % 4 == 0 && al(p.parts, 16))) && (!p.dense || (p.ldd % 4 == 0 && al(p.dense, 16))) &&
                     (!p.next_w || (al(p.next_w, 16) && al(p.h, ab))) && (!p.u_out || al(p.u_out, 16));
    if (vec) {
        const int per = D / 4, block = per >= 512 ? 512 : (per <= 128 ? 128 : (per + 31) / 32 * 32);
        switch (p.S) {
            case 1: ZL_CHECK_CUDA(launch(k_hyper_vec<TO, 1>, dim3(T), dim3(block), 0, st, pdl, p)); break;
            case 2: ZL_CHECK_CUDA(launch(k_hyper_vec<TO, 2>, dim3(T), dim3(block), 0, st, pdl, p)); break;
            case 3: ZL_CHECK_CUDA(launch(k_hyper_vec<TO, 3>, dim3(T), dim3(block), 0, st, pdl, p)); break;
            default: ZL_CHECK_CUDA(launch(k_hyper_vec<TO, 4>, dim3(T), dim3(block), 0, st, pdl, p)); break;
        }
        return ZL_OK;
    }
    const size_t smem = (size_t)D * sizeof(float);
    ZL_CHECK_SUPPORTED(smem <= 200 * 1024);
    static size_t set_for = 0;
    if (smem > 48 * 1024 && smem > set_for) {
        ZL_CHECK_CUDA(cudaFuncSetAttribute(k_hyper_any<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        set_for = smem;
    }
    ZL_CHECK_CUDA(launch(k_hyper_any<TO>, dim3(T), dim3(256), smem, st, pdl, p));
    return ZL_OK;
}

static int hyper_launch(const HyperP& p, int act_dtype, int T, int pdl, cudaStream_t st) {
    if (act_dtype == ZL_F32) return hyper_launch_t<float>(p, T, pdl != 0, st);
    if (act_dtype == ZL_BF16) return hyper_launch_t<__nv_bfloat16>(p, T, pdl != 0, st);
    return hyper_launch_t<__half>(p, T, pdl != 0, st);
}

}  // namespace zl

using namespace zl;

extern "C" int zl_hyper_update(float* x, int streams, const float* parts, long long ldp, const float* coef, int n_parts,
                               const float* dense, long long ldd, const float* mix, const float* out, const float* in,
                               const float* next_w, void* h, float* u_out, int act_dtype, int T, int D, float eps, int pdl,
                               zl_stream_t stream) {
    ZL_CHECK_ARG(x && streams >= 1 && streams <= kHyMaxStreams && T > 0 && D > 0 && eps >= 0.f);
    ZL_CHECK_ARG(!parts || (n_parts > 0 && ldp >= D && mix && out));
    ZL_CHECK_ARG((!dense || (parts && ldd >= D)) && (!next_w || h));
    ZL_CHECK_ARG(act_dtype == ZL_F16 || act_dtype == ZL_BF16 || act_dtype == ZL_F32);
    return hyper_launch(HyperP{x, parts, ldp, coef, n_parts, dense, ldd, mix, out, in, nullptr, nullptr, 0, 1.f, next_w, h, u_out,
                               streams, D, eps}, act_dtype, T, pdl, stream);
}

extern "C" int zl_hyper_embed(const int32_t* ids, const void* table, int vocab, float scale, float* x, int streams, const float* in,
                              const float* next_w, void* h, float* u_out, int act_dtype, int T, int D, float eps, int pdl,
                              zl_stream_t stream) {
    ZL_CHECK_ARG(ids && table && vocab > 0 && x && streams >= 1 && streams <= kHyMaxStreams && T > 0 && D > 0 && eps >= 0.f);
    ZL_CHECK_ARG(!next_w || h);
    ZL_CHECK_ARG(act_dtype == ZL_F16 || act_dtype == ZL_BF16 || act_dtype == ZL_F32);
    return hyper_launch(HyperP{x, nullptr, 0, nullptr, 0, nullptr, 0, nullptr, nullptr, in, ids, table, vocab, scale, next_w, h, u_out,
                               streams, D, eps}, act_dtype, T, pdl, stream);
}
