// Attention whose heads' scores are mixed before the softmax: s'_h = sum_g mix[h][g] (q_g . k_{kv(g)}), over per-slot key
// and value caches with grouped key/value heads, causal, in a sliding window, an ordinary softmax.  A key's mixed score
// needs the scores of every head, so a CTA holds all heads of its tokens; the mixing is fp32 FMAs on fp32 scores in
// shared memory between the two products.  Token t of the step sees keys of slot[t] up to pos[t]; the step's own keys and
// values are appended before this runs.  Key splits leave partial results of the layout of sink_attn.cu and its merge.
//
// k_mixed_head_mma (bfloat16, head sizes that are multiples of 16, values up to 128 wide, at most 16 query heads per
// key/value head and 64 in all, whose tiles fit shared memory): a warp owns 16 rows = (tokens) x (the query heads of one key/value
// head); G warps cover the heads of a token block, and a CTA takes as many token blocks as make up eight warps.  Per key
// tile: S = Q K^T on mma.sync into shared memory; every thread then owns (token, key) columns of all heads and replaces
// them by the mixed scores in place; the warps read their rows back for mask, online softmax and O += P V, the
// probabilities as a bfloat16 pair hi + lo.  The next tile's keys fly during mixing and the second product, its values
// during the next first product.
// k_mixed_head: any sizes and dtype, fp32 FMAs; one CTA per token and group of value heads.
#include "sink_attn.cuh"

#include <cmath>
#include <cstdlib>

namespace zl {

struct MixedP {
    SinkAttnP a;
    const float* mix;          // (H, H)
    const int32_t *run_row0, *run_len;
    int blocks;                // tensor-core kernel: token blocks per CTA
    int kt;                    // its keys per tile
    int hg;                    // general kernel: heads whose values a CTA sums
};

// ---- general kernel ----------------------------------------------------------------------------------------------------
constexpr int kMhWarps = 8, kMhKeys = 32, kMhElems = 32;   // accumulators per thread: hg * vd <= 256 * kMhElems

template <typename T>
__global__ void __launch_bounds__(kMhWarps * 32) k_mixed_head(MixedP pp) {
    extern __shared__ float mh[];
    const SinkAttnP& p = pp.a;
    const int H = p.H, R = H / p.G, d = p.d, vd = p.vd;
    float* sq = mh;                          // [H][d]
    float* ss = sq + (size_t)H * d;          // [H][kMhKeys] scores
    float* sp = ss + H * kMhKeys;            // [hg][kMhKeys] mixed scores, then probabilities
    float* sm = sp + pp.hg * kMhKeys;        // [hg] running max, sum, correction
    float* sl = sm + pp.hg;
    float* sc = sl + pp.hg;
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, h0 = blockIdx.y * pp.hg, hg = min(pp.hg, H - h0), split = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pos = p.pos[t], sl_ = p.slot[t];
    const T* q = static_cast<const T*>(p.q) + (size_t)t * H * d;
    const T* kc = static_cast<const T*>(p.k_addrs[sl_]);
    const T* vc = static_cast<const T*>(p.v_addrs[sl_]);
    const size_t kst = (size_t)p.G * d, vst = (size_t)p.G * vd;
    for (int i = tid; i < H * d; i += blockDim.x) sq[i] = to_f32<T>(q[i]);
    for (int i = tid; i < hg; i += blockDim.x) sm[i] = -INFINITY, sl[i] = 0.f;
    float acc[kMhElems];
#pragma unroll
    for (int e = 0; e < kMhElems; ++e) acc[e] = 0.f;
    int lo = sa_first_key(p, pos), hi = pos + 1;
    if (p.splits > 1) {
        const int per = cdiv(cdiv(hi - lo, p.splits), kMhKeys) * kMhKeys;
        lo += split * per;
        hi = min(hi, lo + per);
    }
    for (int j0 = lo; j0 < hi; j0 += kMhKeys) {
        const int n = min(kMhKeys, hi - j0);
        __syncthreads();   // the previous tile's probabilities are no longer read; the query is in place
        for (int j = warp; j < n; j += kMhWarps)
            for (int g = 0; g < p.G; ++g) {
                const T* kr = kc + (size_t)(j0 + j) * kst + (size_t)g * d;
                for (int r = 0; r < R; ++r) {
                    const float* qh = sq + (size_t)(g * R + r) * d;
                    float s = 0.f;
                    for (int c = lane; c < d; c += 32) s = fmaf(qh[c], to_f32<T>(kr[c]), s);
                    s = warp_sum(s);
                    if (lane == 0) ss[(g * R + r) * kMhKeys + j] = s;
                }
            }
        __syncthreads();
        for (int i = tid; i < hg * kMhKeys; i += blockDim.x) {
            const int h = i / kMhKeys, j = i - h * kMhKeys;
            float s = -INFINITY;
            if (j < n) {
                const float* mrow = pp.mix + (size_t)(h0 + h) * H;
                s = 0.f;
                for (int g = 0; g < H; ++g) s = fmaf(mrow[g], ss[g * kMhKeys + j], s);
            }
            sp[i] = s;
        }
        __syncthreads();
        for (int h = warp; h < hg; h += kMhWarps) {   // a key per lane
            const float s = sp[h * kMhKeys + lane], m_old = sm[h], m_new = fmaxf(m_old, warp_max(s));
            const float e = lane < n ? expf(s - m_new) : 0.f, sum = warp_sum(e);
            sp[h * kMhKeys + lane] = e;
            __syncwarp();
            if (lane == 0) {
                sc[h] = m_old == -INFINITY ? 0.f : expf(m_old - m_new);
                sl[h] = sl[h] * sc[h] + sum;
                sm[h] = m_new;
            }
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < kMhElems; ++e) {
            const int i = tid + e * kMhWarps * 32;
            if (i < hg * vd) {
                const int h = i / vd, c = i - h * vd;
                const T* vr = vc + (size_t)j0 * vst + (size_t)((h0 + h) / R) * vd + c;
                float o = acc[e] * sc[h];
                for (int j = 0; j < n; ++j) o = fmaf(sp[h * kMhKeys + j], to_f32<T>(vr[(size_t)j * vst]), o);
                acc[e] = o;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < kMhElems; ++e) {
        const int i = tid + e * kMhWarps * 32;
        if (i < hg * vd) {
            const int h = i / vd, c = i - h * vd;
            const size_t th = (size_t)t * H + h0 + h;
            if (p.splits > 1) p.ws[(th * p.splits + split) * (2 + vd) + 2 + c] = acc[e];
            else static_cast<T*>(p.out)[th * vd + c] = from_f32<T>(acc[e] / sl[h]);
        }
    }
    if (p.splits > 1)
        for (int h = tid; h < hg; h += blockDim.x) {
            float* part = p.ws + (((size_t)t * H + h0 + h) * p.splits + split) * (2 + vd);
            part[0] = sm[h], part[1] = sl[h];
        }
}

// ---- tensor-core kernel --------------------------------------------------------------------------------------------------
// HM: head count rounded up to the registers of the mixing (8, 16, 32, 64).  NV: 8-column value tiles per warp.  NT: most threads.
template <int NV, int HM, int NT>
__global__ void __launch_bounds__(NT) k_mixed_head_mma(MixedP pp) {
    using T = __nv_bfloat16;
    extern __shared__ __align__(16) unsigned char mh_raw[];
    const SinkAttnP& p = pp.a;
    const int H = p.H, G = p.G, R = H / G, d = p.d, vd = p.vd, KT = pp.kt;
    const int mma_warps = G * pp.blocks, rows = mma_warps * 16;
    const int DP = d + 8, KP = G * d + 8, VP = G * vd + 8, SP = KT + 8;
    T* sQ = reinterpret_cast<T*>(mh_raw);               // [rows][DP]
    T* sK = sQ + (size_t)rows * DP;                     // [KT][KP]
    T* sV = sK + (size_t)KT * KP;                       // [KT][VP]
    float* sS = reinterpret_cast<float*>(sV + (size_t)KT * VP);   // [rows][SP]
    float* sM = sS + (size_t)rows * SP;                 // [H][HM]: mix transposed, zero beyond H
    pdl_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    for (int i = tid; i < H * HM; i += blockDim.x) {
        const int g = i / HM, h = i - g * HM;
        sM[i] = h < H ? pp.mix[(size_t)h * H + g] : 0.f;   // weights: not written by a predecessor in the stream
    }
    pdl_wait();
    const int run = blockIdx.z / p.splits, split = blockIdx.z % p.splits;
    const int nb = 16 / R, nq = nb * pp.blocks;         // tokens per block and per CTA
    const int len = pp.run_len[run], t0 = blockIdx.x * nq;
    if (t0 >= len) return;
    const int ntok = min(nq, len - t0), row0 = pp.run_row0[run] + t0;
    const int sl = p.slot[row0], pos0 = p.pos[row0], n_keys = pos0 + ntok;
    // key tiles start at multiples of KT from key 0 whatever the step
    int k_lo = (sa_first_key(p, pos0) / KT) * KT, k_hi = n_keys;
    if (p.splits > 1) {
        const int per = cdiv(cdiv(n_keys - k_lo, p.splits), KT) * KT;
        k_lo += split * per;
        k_hi = min(n_keys, k_lo + per);
    }
    const T* kc = static_cast<const T*>(p.k_addrs[sl]);
    const T* vc = static_cast<const T*>(p.v_addrs[sl]);
    const int k8 = G * d / 8, v8 = G * vd / 8, d8 = d / 8;
    auto load = [&](T* dst, const T* src, int n8, int ld, int k0) {   // KT rows of n8 16-byte pieces; rows past k_hi are zeros
        for (int i = tid; i < KT * n8; i += blockDim.x) {
            const int r = i / n8, c = i - r * n8;
            if (k0 + r < k_hi) sa_cp_async16(dst + (size_t)r * ld + c * 8, src + ((size_t)(k0 + r) * n8 + c) * 8);
            else *reinterpret_cast<uint4*>(dst + (size_t)r * ld + c * 8) = make_uint4(0, 0, 0, 0);
        }
    };
    // row of the shared-memory tiles that holds (token, head): the warp of (token block, key/value head), then (token in the
    // block, head in the group)
    auto row_of = [&](int tok, int h) {
        const int b = tok / nb, g = h / R;
        return (b * G + g) * 16 + (tok - b * nb) * R + (h - g * R);
    };
    const bool work = warp < mma_warps;
    const int blk = warp / G, g = warp - blk * G;
    int pos_of[2], first_of[2], t_of[2], h_of[2];
    bool row_ok[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        const int r = gq + hh * 8, tk = r / R;
        t_of[hh] = blk * nb + tk;
        h_of[hh] = g * R + (r - tk * R);
        row_ok[hh] = work && tk < nb && t_of[hh] < ntok;
        pos_of[hh] = pos0 + t_of[hh];
        first_of[hh] = sa_first_key(p, pos_of[hh]);
    }
    float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.f, 0.f}, O[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) O[j][c] = 0.f;

    if (k_lo < k_hi) {
        for (int i = tid; i < rows * d8; i += blockDim.x) {
            const int r = i / d8, c = i - r * d8, w = r >> 4, ri = r & 15, b = w / G, tk = ri / R, tok = b * nb + tk;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (tk < nb && tok < ntok)
                v = *reinterpret_cast<const uint4*>(static_cast<const T*>(p.q) +
                                                    ((size_t)(row0 + tok) * H + (w - b * G) * R + (ri - tk * R)) * d + c * 8);
            *reinterpret_cast<uint4*>(sQ + (size_t)r * DP + c * 8) = v;
        }
        load(sK, kc, k8, KP, k_lo);
        sa_cp_commit();
        load(sV, vc, v8, VP, k_lo);
        sa_cp_commit();
        for (int k0 = k_lo; k0 < k_hi; k0 += KT) {
            sa_cp_wait<1>();   // the keys of this tile; its values may still fly
            __syncthreads();
            if (work) {
                const T* qw = sQ + (size_t)warp * 16 * DP;
                float* sw = sS + (size_t)warp * 16 * SP;
                for (int j = 0; j < KT; j += 16) {
                    float S0[4] = {0.f, 0.f, 0.f, 0.f}, S1[4] = {0.f, 0.f, 0.f, 0.f};
                    for (int kk = 0; kk < d; kk += 16) {
                        uint32_t a[4], b[4];
                        sa_ldmatrix_x4(a, qw + (size_t)(lane & 15) * DP + kk + (lane >> 4) * 8);
                        sa_ldmatrix_x4(b, sK + (size_t)(j + (lane & 7) + (lane >> 4) * 8) * KP + g * d + kk + ((lane >> 3) & 1) * 8);
                        mma_16816_bf16(S0, a, b[0], b[1], S0);
                        mma_16816_bf16(S1, a, b[2], b[3], S1);
                    }
                    *reinterpret_cast<float2*>(sw + (size_t)gq * SP + j + 2 * tq) = make_float2(S0[0], S0[1]);
                    *reinterpret_cast<float2*>(sw + (size_t)(gq + 8) * SP + j + 2 * tq) = make_float2(S0[2], S0[3]);
                    *reinterpret_cast<float2*>(sw + (size_t)gq * SP + j + 8 + 2 * tq) = make_float2(S1[0], S1[1]);
                    *reinterpret_cast<float2*>(sw + (size_t)(gq + 8) * SP + j + 8 + 2 * tq) = make_float2(S1[2], S1[3]);
                }
            }
            __syncthreads();   // all scores are in place; the key tile is free
            if (k0 + KT < k_hi) load(sK, kc, k8, KP, k0 + KT);
            sa_cp_commit();
            // mixing: a thread owns the column (token, key) of every head
            for (int i = tid; i < ntok * KT; i += blockDim.x) {
                const int tok = i / KT, key = i - tok * KT;
                float* col = sS + (size_t)row_of(tok, 0) * SP + key;   // head h: row (h / R) * 16 + h % R from here
                float y[HM];
#pragma unroll
                for (int h = 0; h < HM; ++h) y[h] = 0.f;
                for (int gh = 0, rg = 0, rr = 0; gh < H; ++gh) {
                    const float s = col[(size_t)(rg + rr) * SP];
                    const float* mrow = sM + gh * HM;
#pragma unroll
                    for (int h = 0; h < HM; h += 4) {
                        const float4 mv = *reinterpret_cast<const float4*>(mrow + h);
                        y[h] = fmaf(mv.x, s, y[h]), y[h + 1] = fmaf(mv.y, s, y[h + 1]);
                        y[h + 2] = fmaf(mv.z, s, y[h + 2]), y[h + 3] = fmaf(mv.w, s, y[h + 3]);
                    }
                    if (++rr == R) rr = 0, rg += 16;
                }
                int rg = 0, rr = 0;
#pragma unroll
                for (int h = 0; h < HM; ++h) {
                    if (h < H) col[(size_t)(rg + rr) * SP] = y[h];
                    if (++rr == R) rr = 0, rg += 16;
                }
            }
            sa_cp_wait<1>();   // the values of this tile; the next keys may still fly
            __syncthreads();
            if (work) {
                const float* sw = sS + (size_t)warp * 16 * SP;
                auto score = [&](int hh, int key, float s) {   // mask
                    return row_ok[hh] && key < k_hi && key <= pos_of[hh] && key >= first_of[hh] ? s : -1e30f;
                };
                float mx[2] = {-1e30f, -1e30f}, corr[2];
                for (int j = 0; j < KT; j += 8)
#pragma unroll
                    for (int hh = 0; hh < 2; ++hh) {
                        const float2 s = *reinterpret_cast<const float2*>(sw + (size_t)(gq + hh * 8) * SP + j + 2 * tq);
                        mx[hh] = fmaxf(mx[hh], fmaxf(score(hh, k0 + j + 2 * tq, s.x), score(hh, k0 + j + 2 * tq + 1, s.y)));
                    }
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
                    mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
                    const float mn = fmaxf(m_run[hh], mx[hh]);
                    corr[hh] = expf(m_run[hh] - mn);
                    m_run[hh] = mn;
                    l_run[hh] *= corr[hh];
                }
#pragma unroll
                for (int j = 0; j < NV; ++j) {
                    O[j][0] *= corr[0], O[j][1] *= corr[0];
                    O[j][2] *= corr[1], O[j][3] *= corr[1];
                }
                for (int j = 0; j < KT; j += 16) {
                    uint32_t ah[4], al[4];
#pragma unroll
                    for (int r = 0; r < 4; ++r) {   // rows gq / gq + 8 (r & 1), columns + 8 (r >> 1)
                        const int hh = r & 1, col = j + (r >> 1) * 8 + 2 * tq;
                        const float2 s = *reinterpret_cast<const float2*>(sw + (size_t)(gq + hh * 8) * SP + col);
                        const float sx = score(hh, k0 + col, s.x), sy = score(hh, k0 + col + 1, s.y);
                        const float x = sx > -1e29f ? expf(sx - m_run[hh]) : 0.f, y = sy > -1e29f ? expf(sy - m_run[hh]) : 0.f;
                        l_run[hh] += x + y;
                        ah[r] = sa_pack<T>(x, y);
                        al[r] = sa_pack<T>(x - round_to<T>(x), y - round_to<T>(y));
                    }
#pragma unroll
                    for (int nn = 0; nn < NV / 2; ++nn) {
                        if (nn * 16 >= vd) break;
                        uint32_t b[4];
                        sa_ldmatrix_x4_trans(b, sV + (size_t)(j + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + g * vd + nn * 16 + (lane >> 4) * 8);
                        mma_16816_bf16(O[2 * nn], ah, b[0], b[1], O[2 * nn]);
                        mma_16816_bf16(O[2 * nn + 1], ah, b[2], b[3], O[2 * nn + 1]);
                        mma_16816_bf16(O[2 * nn], al, b[0], b[1], O[2 * nn]);
                        mma_16816_bf16(O[2 * nn + 1], al, b[2], b[3], O[2 * nn + 1]);
                    }
                }
            }
            __syncthreads();   // the scores and the value tile are free
            if (k0 + KT < k_hi) load(sV, vc, v8, VP, k0 + KT);
            sa_cp_commit();
        }
    }
    if (!work) return;
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
        l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        if (!row_ok[hh]) continue;
        const size_t th = (size_t)(row0 + t_of[hh]) * H + h_of[hh];
        if (p.splits > 1) {
            float* part = p.ws + (th * p.splits + split) * (2 + vd);
            const bool empty = l_run[hh] <= 0.f;
            if (tq == 0) part[0] = empty ? -INFINITY : m_run[hh], part[1] = empty ? 0.f : l_run[hh];
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int c = 8 * j + 2 * tq;
                if (c < vd) part[2 + c] = O[j][hh * 2], part[2 + c + 1] = O[j][hh * 2 + 1];
            }
        } else {
            const float inv = 1.0f / l_run[hh];
            T* out = static_cast<T*>(p.out) + th * vd;
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                const int c = 8 * j + 2 * tq;
                if (c < vd) *reinterpret_cast<uint32_t*>(out + c) = sa_pack<T>(O[j][hh * 2] * inv, O[j][hh * 2 + 1] * inv);
            }
        }
    }
}

constexpr int kMhSmemMax = 225 * 1024;

static size_t mixed_smem(int H, int G, int d, int vd, int blocks, int kt, int hm) {
    const size_t rows = (size_t)G * blocks * 16;
    return 2 * (rows * (d + 8) + (size_t)kt * (G * d + 8) + (size_t)kt * (G * vd + 8)) + 4 * (rows * (kt + 8) + (size_t)H * hm);
}

// token blocks per CTA and keys per tile of the tensor-core kernel; false: the sizes do not suit it.  max_tokens: the
// longest run (0: unknown) -- a decode step needs one block.
static bool mixed_shape(int H, int G, int d, int vd, int max_tokens, int& blocks, int& kt, int& hm) {
    const int R = H / G;
    if (d % 16 || vd % 16 || vd > 128 || d > 256 || R > 16 || G > 16 || H > 64) return false;
    hm = H <= 8 ? 8 : (H <= 16 ? 16 : (H <= 32 ? 32 : 64));
    const int nb = 16 / R;
    blocks = G >= 8 ? 1 : 8 / G;
    const int need = max_tokens > 0 ? cdiv(max_tokens, nb) : blocks;
    if (blocks > need) blocks = need;
    for (kt = 64; kt >= 16; kt >>= 1)
        if (mixed_smem(H, G, d, vd, blocks, kt, hm) <= (size_t)kMhSmemMax) return true;
    blocks = 1;
    kt = 16;
    return mixed_smem(H, G, d, vd, 1, 16, hm) <= (size_t)kMhSmemMax;
}

template <int NV, int HM, int NT>
static cudaError_t launch_mixed(const MixedP& pp, dim3 grid, size_t smem, bool pdl, cudaStream_t st) {
    static size_t set_for = 0;
    if (smem > 48 * 1024 && smem > set_for) {
        const cudaError_t e = cudaFuncSetAttribute(k_mixed_head_mma<NV, HM, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        set_for = smem;
    }
    const int warps = pp.a.G * pp.blocks;   // at least four warps: spare ones help to load and mix
    return launch(k_mixed_head_mma<NV, HM, NT>, grid, dim3(32 * (warps < 4 ? 4 : warps)), smem, st, pdl, pp);
}
template <int NV>
static cudaError_t launch_mixed_h(const MixedP& pp, int hm, dim3 grid, size_t smem, bool pdl, cudaStream_t st) {
    if (pp.a.G * pp.blocks > 8) {   // more than eight key/value heads
        if (hm == 16) return launch_mixed<NV, 16, 512>(pp, grid, smem, pdl, st);
        if (hm == 32) return launch_mixed<NV, 32, 512>(pp, grid, smem, pdl, st);
        return launch_mixed<NV, 64, 512>(pp, grid, smem, pdl, st);
    }
    if (hm == 8) return launch_mixed<NV, 8, 256>(pp, grid, smem, pdl, st);
    if (hm == 16) return launch_mixed<NV, 16, 256>(pp, grid, smem, pdl, st);
    if (hm == 32) return launch_mixed<NV, 32, 256>(pp, grid, smem, pdl, st);
    return launch_mixed<NV, 64, 256>(pp, grid, smem, pdl, st);
}

template <typename T>
static cudaError_t launch_mixed_general(const MixedP& pp, int T_, bool pdl, cudaStream_t st) {
    const SinkAttnP& p = pp.a;
    const size_t smem = ((size_t)p.H * p.d + (size_t)(p.H + pp.hg) * kMhKeys + 3 * (size_t)pp.hg) * sizeof(float);
    static size_t set_for = 0;
    if (smem > 48 * 1024 && smem > set_for) {
        const cudaError_t e = cudaFuncSetAttribute(k_mixed_head<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        set_for = smem;
    }
    return launch(k_mixed_head<T>, dim3(T_, cdiv(p.H, pp.hg), p.splits), dim3(kMhWarps * 32), smem, st, pdl, pp);
}

}  // namespace zl

using namespace zl;

// a CTA holds every head of its token: one wave of CTAs, no split shorter than 32 keys, at most 32
extern "C" int zl_mixed_head_attention_splits(int T, int heads, int max_len) {
    (void)heads;
    const int want = cdiv(device_sm_count(), T > 0 ? T : 1), cap = max_len / 32 > 0 ? max_len / 32 : 1;
    int s = want < cap ? want : cap;
    if (s > 32) s = 32;
    return s < 1 ? 1 : s;
}

extern "C" int zl_mixed_head_attention(const void* q, void* const* k_addrs, void* const* v_addrs, const int32_t* slot,
                                       const int32_t* pos, const float* mix, int window, void* out, int T, int heads, int kv_heads,
                                       int dim, int vdim, int splits, void* workspace, size_t workspace_bytes,
                                       const int32_t* run_row0, const int32_t* run_len, int runs, int max_run_len, int dtype,
                                       int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(q && k_addrs && v_addrs && slot && pos && mix && out && T > 0 && T <= 65535 && heads > 0 && kv_heads > 0);
    ZL_CHECK_ARG(heads % kv_heads == 0 && dim > 0 && vdim > 0 && window >= 0);
    ZL_CHECK_ARG(dtype == ZL_F16 || dtype == ZL_BF16 || dtype == ZL_F32);
    ZL_CHECK_ARG(splits >= 1 && splits <= 32);
    ZL_CHECK_ARG(splits == 1 || (workspace && workspace_bytes >= zl_sink_attention_workspace_bytes(T, heads, vdim, splits)));
    MixedP pp{};
    pp.a = SinkAttnP{q, k_addrs, v_addrs, slot, pos, nullptr, nullptr, 0, out, heads, kv_heads, dim, vdim, 1.0f, splits,
                     static_cast<float*>(workspace)};
    pp.a.no_sink = 1;
    pp.a.window = window;
    pp.mix = mix;
    pp.run_row0 = run_row0;
    pp.run_len = run_len;
    static const bool no_mma = getenv("ZL_MIXED_HEAD_NO_MMA") != nullptr;
    int hm = 0;
    if (!no_mma && dtype == ZL_BF16 && run_row0 && run_len && runs > 0 && max_run_len > 0 &&
        mixed_shape(heads, kv_heads, dim, vdim, max_run_len, pp.blocks, pp.kt, hm)) {
        ZL_CHECK_ARG((long long)runs * splits <= 65535);
        const dim3 grid(cdiv(max_run_len, 16 / (heads / kv_heads) * pp.blocks), 1, runs * splits);
        const size_t smem = mixed_smem(heads, kv_heads, dim, vdim, pp.blocks, pp.kt, hm);
        ZL_CHECK_CUDA(vdim <= 64 ? launch_mixed_h<8>(pp, hm, grid, smem, pdl != 0, stream)
                                 : launch_mixed_h<16>(pp, hm, grid, smem, pdl != 0, stream));
    } else {
        ZL_CHECK_SUPPORTED(vdim <= kMhWarps * 32 * kMhElems);
        pp.hg = kMhWarps * 32 * kMhElems / vdim;
        if (pp.hg > heads) pp.hg = heads;
        ZL_CHECK_SUPPORTED(((size_t)heads * dim + (size_t)2 * heads * (kMhKeys + 2)) * sizeof(float) <= (size_t)kMhSmemMax);
        cudaError_t e;
        if (dtype == ZL_F32) e = launch_mixed_general<float>(pp, T, pdl != 0, stream);
        else if (dtype == ZL_BF16) e = launch_mixed_general<__nv_bfloat16>(pp, T, pdl != 0, stream);
        else e = launch_mixed_general<__half>(pp, T, pdl != 0, stream);
        ZL_CHECK_CUDA(e);
    }
    return splits > 1 ? sink_attn_merge(pp.a, 1, T, dtype, pdl != 0, stream) : ZL_OK;
}
