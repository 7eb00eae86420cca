// Routing of a mixture of experts, on the device from the router's input to the index lists of the grouped GEMMs:
//   * k_moe_route: logits z = W_router x in fp32 (x is the fp32 residual stream), a score per expert (sigmoid or
//     softmax over the experts), the `top` experts with the largest score + correction (ties: the lower index), their
//     weights = the scores without the correction, optionally renormalised to sum 1.  The logits may also arrive ready
//     (columns of a fused projection), or come from a 16-bit input and router.  Restricted choice: the experts form equal
//     groups of neighbours, a group ranks by its largest score + correction or the sum of its two largest, and only
//     experts of the `keep` best groups can be chosen; the weights may carry a constant factor;
//   * k_moe_plan: the (token, choice) pairs sorted by expert: group offsets, and for every list entry the token row it
//     reads and the pair row it writes.  The order inside a group is arbitrary (no row's result depends on it).
// Nothing returns to the host, so a step with routing can be captured in a CUDA graph.
#include "common.cuh"

namespace zl {

constexpr int kRouteWarps = 16;

// row . row with independent 16-byte loads in flight (both rows 16-byte aligned, D % 4 == 0), else element by element
__device__ __forceinline__ float route_dot(const float* __restrict__ a, const float* __restrict__ b, int D, int lane, bool vec) {
    float acc0 = 0.f, acc1 = 0.f;
    if (vec) {
        const float4* a4 = reinterpret_cast<const float4*>(a);
        const float4* b4 = reinterpret_cast<const float4*>(b);
        const int n4 = D >> 2;
        int c = lane;
        for (; c + 32 < n4; c += 64) {
            const float4 x0 = a4[c], y0 = b4[c], x1 = a4[c + 32], y1 = b4[c + 32];
            acc0 = fmaf(x0.x, y0.x, fmaf(x0.y, y0.y, fmaf(x0.z, y0.z, fmaf(x0.w, y0.w, acc0))));
            acc1 = fmaf(x1.x, y1.x, fmaf(x1.y, y1.y, fmaf(x1.z, y1.z, fmaf(x1.w, y1.w, acc1))));
        }
        for (; c < n4; c += 32) {
            const float4 x0 = a4[c], y0 = b4[c];
            acc0 = fmaf(x0.x, y0.x, fmaf(x0.y, y0.y, fmaf(x0.z, y0.z, fmaf(x0.w, y0.w, acc0))));
        }
    } else {
        for (int c = lane; c < D; c += 32) acc0 = fmaf(a[c], b[c], acc0);
    }
    return warp_sum(acc0 + acc1);
}

// 16-bit rows: 16-byte loads of eight elements when both rows allow it
template <typename T>
__device__ __forceinline__ float route_dot16(const T* __restrict__ a, const T* __restrict__ b, int D, int lane, bool vec) {
    float acc0 = 0.f, acc1 = 0.f;
    if (vec) {
        const uint4 *a8 = reinterpret_cast<const uint4*>(a), *b8 = reinterpret_cast<const uint4*>(b);
        const int n8 = D >> 3;
        for (int c0 = lane; c0 < n8; c0 += 128) {   // four pieces of both rows in flight
            uint4 u[4], v[4];
#pragma unroll
            for (int k = 0; k < 4; ++k)
                if (c0 + 32 * k < n8) u[k] = a8[c0 + 32 * k], v[k] = b8[c0 + 32 * k];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (c0 + 32 * k >= n8) break;
                float x[8], y[8];
                unpack8<T>(u[k], x);
                unpack8<T>(v[k], y);
#pragma unroll
                for (int i = 0; i < 8; i += 2) acc0 = fmaf(x[i], y[i], acc0), acc1 = fmaf(x[i + 1], y[i + 1], acc1);
            }
        }
    } else {
        for (int c = lane; c < D; c += 32) acc0 = fmaf(to_f32<T>(a[c]), to_f32<T>(b[c]), acc0);
    }
    return warp_sum(acc0 + acc1);
}

// grid (T), 16 warps; dynamic shared memory (2 * E + groups) floats.  w_router null: x[t] holds the E logits (fp32).
template <typename T>
__global__ void __launch_bounds__(kRouteWarps * 32) k_moe_route(const T* __restrict__ x, long long ldx,
                                                   const T* __restrict__ w_router, const float* __restrict__ correction,
                                                   int32_t* __restrict__ top_e, float* __restrict__ top_w, int D, int E,
                                                   int top, int score_fn, int renorm, int groups, int keep, int group_rank,
                                                   float renorm_eps, float weight_scale) {
    extern __shared__ float sm[];
    float* score = sm;        // s_e
    float* choice = sm + E;   // s_e + correction_e; taken experts drop to -inf
    float* gbest = sm + 2 * E;   // rank of every group; a kept group is marked +inf
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* xr = x + (size_t)t * ldx;
    if (w_router) {
        constexpr int kVec = 16 / (int)sizeof(T);
        const bool vec = D % kVec == 0 && ldx % kVec == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w_router)) & 15) == 0;
        for (int e = warp; e < E; e += kRouteWarps) {
            float acc;
            if constexpr (sizeof(T) == 4) acc = route_dot(xr, w_router + (size_t)e * D, D, lane, vec);
            else acc = route_dot16<T>(xr, w_router + (size_t)e * D, D, lane, vec);
            if (lane == 0) score[e] = acc;
        }
    } else {
        for (int e = threadIdx.x; e < E; e += blockDim.x) score[e] = to_f32<T>(xr[e]);
    }
    __syncthreads();
    if (warp != 0) return;
    if (score_fn == ZL_MOE_SCORE_SOFTMAX) {
        float mx = -INFINITY;
        for (int e = lane; e < E; e += 32) mx = fmaxf(mx, score[e]);
        mx = warp_max(mx);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) sum += expf(score[e] - mx);
        sum = warp_sum(sum);
        for (int e = lane; e < E; e += 32) score[e] = expf(score[e] - mx) / sum;
    } else {
        for (int e = lane; e < E; e += 32) score[e] = 1.0f / (1.0f + expf(-score[e]));
    }
    for (int e = lane; e < E; e += 32) choice[e] = score[e] + (correction ? correction[e] : 0.f);
    __syncwarp();
    if (groups > 1 && keep < groups) {
        // the `keep` groups of the highest rank survive (ties: the lower group); the others' members drop to -inf
        const int per = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float b = -INFINITY, b2 = -INFINITY;   // the two largest
            for (int i = 0; i < per; ++i) {
                const float v = choice[g * per + i];
                if (v > b) b2 = b, b = v;
                else b2 = fmaxf(b2, v);
            }
            gbest[g] = group_rank == ZL_MOE_GROUP_TOP2 && per > 1 ? b + b2 : b;
        }
        __syncwarp();
        for (int k = 0; k < keep; ++k) {
            float bv = -INFINITY;
            int bi = 0x7fffffff;
            for (int g = lane; g < groups; g += 32) {
                const float v = gbest[g];
                if (v != INFINITY && (v > bv || bi == 0x7fffffff)) bv = v, bi = g;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
                const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                if (oi != 0x7fffffff && (bi == 0x7fffffff || ov > bv || (ov == bv && oi < bi))) bv = ov, bi = oi;
            }
            if (lane == 0 && bi < groups) gbest[bi] = INFINITY;
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (gbest[e / per] != INFINITY) choice[e] = -INFINITY;
        __syncwarp();
    }
    float wsum = 0.f;
    for (int k = 0; k < top; ++k) {
        float bv = -INFINITY;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float v = choice[e];
            if (v > bv) bv = v, bi = e;   // ascending e: the lower index wins a tie inside a lane
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) bv = ov, bi = oi;
        }
        if (bi >= E) bi = k < E ? k : 0;   // only when every score is NaN / -inf
        if (lane == 0) {
            top_e[(size_t)t * top + k] = bi;
            top_w[(size_t)t * top + k] = score[bi];
            choice[bi] = -INFINITY;
        }
        wsum += score[bi];
        __syncwarp();
    }
    if (lane == 0 && (renorm || weight_scale != 1.0f)) {
        const float div = renorm ? wsum + renorm_eps : 1.0f;
        for (int k = 0; k < top; ++k) top_w[(size_t)t * top + k] = top_w[(size_t)t * top + k] / div * weight_scale;
    }
}

// one CTA; dynamic shared memory 2 * (E + 1) ints
__global__ void __launch_bounds__(1024) k_moe_plan(const int32_t* __restrict__ top_e, int pairs, int E, int top,
                                                   int32_t* __restrict__ grp_off, int32_t* __restrict__ list_token,
                                                   int32_t* __restrict__ list_pair) {
    extern __shared__ int ism[];
    int* cnt = ism;            // E + 1
    int* cur = ism + E + 1;    // E + 1
    pdl_trigger();
    pdl_wait();
    for (int e = threadIdx.x; e <= E; e += blockDim.x) cnt[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) atomicAdd(&cnt[top_e[i]], 1);
    __syncthreads();
    if (threadIdx.x == 0) {
        int run = 0;
        for (int e = 0; e < E; ++e) {
            const int c = cnt[e];
            cur[e] = run;
            grp_off[e] = run;
            run += c;
        }
        grp_off[E] = run;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
        const int at = atomicAdd(&cur[top_e[i]], 1);
        list_token[at] = i / top;
        list_pair[at] = i;
    }
}

}  // namespace zl

using namespace zl;

extern "C" int zl_moe_route(const float* x, long long ldx, const float* w_router, const float* correction, int32_t* top_experts,
                            float* top_weights, int32_t* group_offsets, int32_t* list_token, int32_t* list_pair, int T, int D,
                            int experts, int top, int score_fn, int renormalize, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(x && w_router && top_experts && top_weights && group_offsets && list_token && list_pair);
    ZL_CHECK_ARG(T > 0 && D > 0 && experts > 0 && top > 0 && top <= experts && experts <= 4096);
    ZL_CHECK_ARG(score_fn == ZL_MOE_SCORE_SIGMOID || score_fn == ZL_MOE_SCORE_SOFTMAX);
    return zl_moe_route_grouped(x, ldx, w_router, correction, top_experts, top_weights, group_offsets, list_token, list_pair, T, D,
                                experts, top, 1, 1, score_fn, renormalize, 0.f, pdl, stream);
}

extern "C" int zl_moe_route_grouped(const float* x, long long ldx, const float* w_router, const float* correction,
                                    int32_t* top_experts, float* top_weights, int32_t* group_offsets, int32_t* list_token,
                                    int32_t* list_pair, int T, int D, int slots, int top, int groups, int keep, int score_fn,
                                    int renormalize, float renorm_eps, int pdl, zl_stream_t stream) {
    return zl_moe_route_ex(x, ldx, w_router, ZL_F32, correction, top_experts, top_weights, group_offsets, list_token, list_pair, T,
                           D, slots, top, groups, keep, ZL_MOE_GROUP_MAX, score_fn, renormalize, renorm_eps, 1.0f, pdl, stream);
}

extern "C" int zl_moe_route_ex(const void* x, long long ldx, const void* w_router, int in_dtype, const float* correction,
                               int32_t* top_experts, float* top_weights, int32_t* group_offsets, int32_t* list_token,
                               int32_t* list_pair, int T, int D, int slots, int top, int groups, int keep, int group_rank,
                               int score_fn, int renormalize, float renorm_eps, float weight_scale, int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(x && top_experts && top_weights && group_offsets && list_token && list_pair);
    ZL_CHECK_ARG(T > 0 && (D > 0 || !w_router) && slots > 0 && top > 0 && top <= slots && slots <= 4096);
    ZL_CHECK_ARG(w_router || (ldx >= slots && in_dtype == ZL_F32));
    ZL_CHECK_ARG(groups >= 1 && slots % groups == 0 && keep >= 1 && keep <= groups && keep * (slots / groups) >= top);
    ZL_CHECK_ARG(score_fn == ZL_MOE_SCORE_SIGMOID || score_fn == ZL_MOE_SCORE_SOFTMAX);
    ZL_CHECK_ARG(group_rank == ZL_MOE_GROUP_MAX || group_rank == ZL_MOE_GROUP_TOP2);
    ZL_CHECK_ARG(in_dtype == ZL_F32 || in_dtype == ZL_BF16 || in_dtype == ZL_F16);
    // with ready logits only the choosing warp has work
    const dim3 grid(T), block(w_router ? kRouteWarps * 32 : 32);
    const size_t smem = (size_t)(2 * slots + groups) * sizeof(float);
    cudaError_t e;
#define ZL_ROUTE(TX)                                                                                                          \
    launch(k_moe_route<TX>, grid, block, smem, stream, pdl != 0, static_cast<const TX*>(x), ldx, static_cast<const TX*>(w_router), \
           correction, top_experts, top_weights, D, slots, top, score_fn, renormalize, groups, keep, group_rank, renorm_eps, weight_scale)
    if (in_dtype == ZL_F32) e = ZL_ROUTE(float);
    else if (in_dtype == ZL_BF16) e = ZL_ROUTE(__nv_bfloat16);
    else e = ZL_ROUTE(__half);
#undef ZL_ROUTE
    ZL_CHECK_CUDA(e);
    ZL_CHECK_CUDA(launch(k_moe_plan, dim3(1), dim3(1024), (size_t)2 * (slots + 1) * sizeof(int), stream, pdl != 0,
                         (const int32_t*)top_experts, T * top, slots, top, group_offsets, list_token, list_pair));
    return ZL_OK;
}
