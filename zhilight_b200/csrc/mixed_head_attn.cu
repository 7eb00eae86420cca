// Attention whose heads' scores are mixed before the softmax: s'_h = sum_g mix[h][g] factor[g] (q_g . k_{kv(g)}), over
// per-slot key and value caches with grouped key/value heads, causal, in a sliding window, an ordinary softmax.  A key's
// mixed score needs the scores of every head, so a CTA holds all heads of its tokens.  Token t of the step sees keys of
// slot[t] up to pos[t]; the step's own keys and values are appended before this runs.  Key splits leave partial results of
// the layout of sink_attn.cu and its merge.
//
// k_mixed_head_mma (bfloat16, head sizes that are multiples of 16, values up to 128 wide, at most 16 key/value heads, 16
// query heads per key/value head and 64 in all): a warp owns 16 rows = (tokens) x (the query heads of one key/value head),
// its queries in registers; G warps cover the heads of a token block, and a CTA takes as many token blocks as make up
// eight warps.  Per key tile: S = Q K^T on mma.sync; the fp32 scores go to shared memory as the sum of three bfloat16
// numbers (24 bits: nothing of the fp32 score is lost), token by token with the heads as rows; mixing is then a product of
// the (H, H) matrix, whose weights are 16-bit in this mode anyway, with those parts on the tensor cores, fp32 accumulators
// to a second array; the warps read their rows back for mask, online softmax and O += P V, the probabilities as a pair
// hi + lo.  (Mixing on the FMA pipes cost two thirds of the kernel's instructions.)  The next tile's keys fly during mixing
// and the second product, a tile's values during its first product and mixing; two CTAs share an SM where the tiles allow.
// k_mixed_head: any sizes and dtype, fp32 FMAs; one CTA per token and group of value heads.
#include "sink_attn.cuh"

#include <cmath>
#include <cstdlib>

namespace zl {

struct MixedP {
    SinkAttnP a;
    const float* mix;          // (H, H)
    const float* factor;       // (H): of a head's scores before the mixing
    const int32_t *run_row0, *run_len;
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
                    if (lane == 0) ss[(g * R + r) * kMhKeys + j] = s * pp.factor[g * R + r];
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
constexpr float kLog2E = 1.44269504f, kLn2 = 0.693147181f;

// Byte offsets of the dynamic shared memory: the key tile and the value tile (before the first tile: the queries on their
// way to registers), three arrays of the scores' bfloat16 parts, the mixed scores, the mixing matrix, the heads'
// rows.
struct MixedShape {
    int blocks, h16;
    size_t v_off, s_off, y_off, a_off, t_off, bytes;
};

// NV: 8-column value tiles per warp.  ND: 16-column contraction steps held in registers.  KT keys per tile.  NT threads at
// most, NB CTAs per SM.
template <int NV, int ND, int KT, int NT, int NB>
__global__ void __launch_bounds__(NT, NB) k_mixed_head_mma(MixedP pp, MixedShape sh) {
    using T = __nv_bfloat16;
    constexpr int SB = KT + 8, NS = KT / 8;
    extern __shared__ __align__(16) unsigned char mh_raw[];
    const SinkAttnP& p = pp.a;
    const int H = p.H, G = p.G, R = H / G, d = p.d, vd = p.vd, H16 = sh.h16;
    const int mma_warps = G * sh.blocks, rows = mma_warps * 16;
    const int nb = 16 / R, nq = nb * sh.blocks;                  // tokens per block and per CTA
    const int DP = d + 8, KP = G * d + 8, VP = G * vd + 8, AP = H16 + 8;
    T* sK = reinterpret_cast<T*>(mh_raw);                        // [KT][KP]
    T* sV = reinterpret_cast<T*>(mh_raw + sh.v_off);             // [KT][VP]
    T* sQ = reinterpret_cast<T*>(mh_raw);                        // [rows][DP], before the tiles
    T* sS = reinterpret_cast<T*>(mh_raw + sh.s_off);             // [3][nq * H16][SB]: row (token, head), zero rows beyond H
    float* sY = reinterpret_cast<float*>(mh_raw + sh.y_off);     // [rows][SB] mixed scores, row as in the queries' tiles
    T* sA = reinterpret_cast<T*>(mh_raw + sh.a_off);             // [H16][AP] mixing matrix
    int* sR = reinterpret_cast<int*>(mh_raw + sh.t_off);         // [H16] row of a head from its token's first row, or -1
    const int part = nq * H16 * SB;
    pdl_trigger();
    const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    for (int i = tid; i < H16 * H16; i += nthr) {                // weights: not written by a predecessor in the stream
        const int h = i / H16, g = i - h * H16;
        sA[h * AP + g] = from_f32<T>(h < H && g < H ? pp.mix[(size_t)h * H + g] : 0.f);
    }
    for (int h = tid; h < H16; h += nthr) sR[h] = h < H ? (h / R) * 16 + h % R : -1;
    pdl_wait();
    const int run = blockIdx.z / p.splits, split = blockIdx.z - run * p.splits;
    const int len = pp.run_len[run], t0 = (int)(gridDim.x - 1 - blockIdx.x) * nq;   // the tiles with the most keys start first
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
    // KT rows of n8 16-byte pieces (contiguous in the cache), rows past k_hi are zeros
    const int kr0 = tid / k8, kdr = nthr / k8, vr0 = tid / v8, vdr = nthr / v8;
    const bool k_even = kdr * k8 == nthr, v_even = vdr * v8 == nthr;   // every round of loads covers whole rows
    auto load = [&](T* dst, const T* src, int n8, int ld, int k0, int r, int dr, bool even) {
        const T* s = src + ((size_t)k0 * n8 + tid) * 8;
        const int rows_in = k_hi - k0;
        if (even) {
            uint32_t o = smem_u32(dst + r * ld + (tid - r * n8) * 8);
            const uint32_t step = 2 * dr * ld;
#pragma unroll 4
            for (; r < KT; r += dr, o += step, s += (size_t)nthr * 8) {
                if (r < rows_in) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(o), "l"(s) : "memory");
                else asm volatile("st.shared.v4.u32 [%0], {%1, %1, %1, %1};" ::"r"(o), "r"(0) : "memory");
            }
            return;
        }
        for (int i = tid; i < KT * n8; i += nthr, s += (size_t)nthr * 8) {
            const int rr = i / n8;
            T* o = dst + rr * ld + (i - rr * n8) * 8;
            if (rr < rows_in) sa_cp_async16(o, s);
            else *reinterpret_cast<uint4*>(o) = make_uint4(0, 0, 0, 0);
        }
    };
    const bool work = warp < mma_warps;
    const int blk = warp / G, g = warp - blk * G;
    int pos_of[2], first_of[2], t_of[2], h_of[2];
    bool row_ok[2], in_tile[2];
    float f_of[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        const int r = gq + hh * 8, tk = r / R;
        t_of[hh] = blk * nb + tk;
        h_of[hh] = g * R + (r - tk * R);
        in_tile[hh] = work && tk < nb;
        row_ok[hh] = in_tile[hh] && t_of[hh] < ntok;
        pos_of[hh] = row_ok[hh] ? pos0 + t_of[hh] : -1;   // a row without a token sees nothing
        first_of[hh] = row_ok[hh] ? sa_first_key(p, pos_of[hh]) : 0;
        f_of[hh] = in_tile[hh] ? pp.factor[h_of[hh]] * kLog2E : 0.f;   // scores in units of ln 2: weights are powers of two
    }
    // every row of this warp has a token and sees all keys from all_lo to all_hi
    const bool full_rows = __all_sync(0xffffffffu, row_ok[0] && row_ok[1]);
    const int all_lo = sa_first_key(p, pos0 + ntok - 1), all_hi = pos0;
    float m_run[2] = {-1e30f, -1e30f}, l_run[2] = {0.f, 0.f}, O[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j)
#pragma unroll
        for (int c = 0; c < 4; ++c) O[j][c] = 0.f;

    if (k_lo < k_hi) {
        for (int i = tid; i < rows * d8; i += nthr) {
            const int r = i / d8, c = i - r * d8, w = r >> 4, ri = r & 15, b = w / G, tk = ri / R, tok = b * nb + tk;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (tk < nb && tok < ntok)
                v = *reinterpret_cast<const uint4*>(static_cast<const T*>(p.q) +
                                                    ((size_t)(row0 + tok) * H + (w - b * G) * R + (ri - tk * R)) * d + c * 8);
            *reinterpret_cast<uint4*>(sQ + (size_t)r * DP + c * 8) = v;
        }
        __syncthreads();
        uint32_t qf[ND][4];
        if (work) {
#pragma unroll
            for (int kk = 0; kk < ND; ++kk)
                if (kk * 16 < d) sa_ldmatrix_x4(qf[kk], sQ + (size_t)(warp * 16 + (lane & 15)) * DP + kk * 16 + (lane >> 4) * 8);
        }
        __syncthreads();   // the queries are in registers: the tiles may be written
        load(sK, kc, k8, KP, k_lo, kr0, kdr, k_even);
        sa_cp_commit();
        if (H16 > H)
            for (int i = tid; i < 3 * part; i += nthr) sS[i] = from_f32<T>(0.f);   // heads that do not exist score zero
        const int units = ntok * (H16 / 16) * (KT / 16), n_warps = nthr >> 5;
        for (int k0 = k_lo; k0 < k_hi; k0 += KT) {
            sa_cp_wait<0>();
            __syncthreads();   // the keys of this tile; every warp is done with the previous values and mixed scores
            load(sV, vc, v8, VP, k0, vr0, vdr, v_even);
            sa_cp_commit();
            if (work) {
#pragma unroll
                for (int j = 0; j < KT; j += 16) {
                    float S[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
                    const T* kb = sK + (j + (lane & 7) + (lane >> 4) * 8) * KP + g * d + ((lane >> 3) & 1) * 8;
#pragma unroll
                    for (int kk = 0; kk < ND; ++kk)
                        if (kk * 16 < d) {
                            uint32_t b[4];
                            sa_ldmatrix_x4(b, kb + kk * 16);
                            mma_16816_bf16(S[0], qf[kk], b[0], b[1], S[0]);
                            mma_16816_bf16(S[1], qf[kk], b[2], b[3], S[1]);
                        }
                    // fp32 scores as the sum of three bfloat16 numbers
#pragma unroll
                    for (int hh = 0; hh < 2; ++hh) {
                        if (!in_tile[hh]) continue;
                        T* dst = sS + (t_of[hh] * H16 + h_of[hh]) * SB + j + 2 * tq;
#pragma unroll
                        for (int n = 0; n < 2; ++n) {
                            float x = S[n][2 * hh] * f_of[hh], y = S[n][2 * hh + 1] * f_of[hh];
#pragma unroll
                            for (int q = 0; q < 3; ++q) {
                                const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
                                *reinterpret_cast<__nv_bfloat162*>(dst + q * part + n * 8) = v;
                                x -= __low2float(v), y -= __high2float(v);
                            }
                        }
                    }
                }
            }
            __syncthreads();   // all scores are in place; the key tile is free
            if (k0 + KT < k_hi) load(sK, kc, k8, KP, k0 + KT, kr0, kdr, k_even);
            sa_cp_commit();
            // mixing: a warp takes 16 output heads of one token and 16 keys, (16 x H) by (H x 16)
            for (int u = warp; u < units; u += n_warps) {
                const int n16 = u % (KT / 16), rest = u / (KT / 16), mt = rest / ntok, tok = rest - mt * ntok, b = tok / nb;
                float y[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
                const T* arow = sA + (mt * 16 + (lane & 15)) * AP + (lane >> 4) * 8;
                const T* brow = sS + (tok * H16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SB + n16 * 16 + (lane >> 4) * 8;
                for (int kg = 0; kg < H16; kg += 16) {
                    uint32_t a[4];
                    sa_ldmatrix_x4(a, arow + kg);
#pragma unroll
                    for (int q = 2; q >= 0; --q) {   // the small parts first
                        uint32_t bv[4];
                        sa_ldmatrix_x4_trans(bv, brow + kg * SB + q * part);
                        mma_16816_bf16(y[0], a, bv[0], bv[1], y[0]);
                        mma_16816_bf16(y[1], a, bv[2], bv[3], y[1]);
                    }
                }
                float* yb = sY + (b * G * 16 + (tok - b * nb) * R) * SB + n16 * 16 + 2 * tq;
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    const int ro = sR[mt * 16 + gq + hh * 8];
                    if (ro < 0) continue;
                    *reinterpret_cast<float2*>(yb + ro * SB) = make_float2(y[0][2 * hh], y[0][2 * hh + 1]);
                    *reinterpret_cast<float2*>(yb + ro * SB + 8) = make_float2(y[1][2 * hh], y[1][2 * hh + 1]);
                }
            }
            sa_cp_wait<1>();   // the values of this tile; the next keys may still fly
            __syncthreads();
            if (!work) continue;
            const float* sw = sY + warp * 16 * SB + 2 * tq;
            float v[NS][4], mx[2] = {-1e30f, -1e30f}, corr[2];
#pragma unroll
            for (int j = 0; j < NS; ++j)
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    const float2 s = *reinterpret_cast<const float2*>(sw + (gq + hh * 8) * SB + j * 8);
                    v[j][2 * hh] = s.x, v[j][2 * hh + 1] = s.y;
                }
            if (!(full_rows && k0 >= all_lo && k0 + KT - 1 <= all_hi)) {   // a tile at an edge: mask
#pragma unroll
                for (int j = 0; j < NS; ++j)
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        const int key = k0 + j * 8 + 2 * tq + (c & 1);
                        if (key > pos_of[c >> 1] || key < first_of[c >> 1]) v[j][c] = -1e30f;
                    }
            }
#pragma unroll
            for (int j = 0; j < NS; ++j)
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) mx[hh] = fmaxf(mx[hh], fmaxf(v[j][2 * hh], v[j][2 * hh + 1]));
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
                mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
                const float mn = fmaxf(m_run[hh], mx[hh]);
                corr[hh] = exp2f(m_run[hh] - mn);
                m_run[hh] = mn;
                l_run[hh] *= corr[hh];
            }
            if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
                for (int j = 0; j < NV; ++j) {
                    O[j][0] *= corr[0], O[j][1] *= corr[0];
                    O[j][2] *= corr[1], O[j][3] *= corr[1];
                }
            }
#pragma unroll
            for (int j = 0; j < NS; j += 2) {
                uint32_t ah[4], al[4];
#pragma unroll
                for (int r = 0; r < 4; ++r) {   // rows gq / gq + 8 (r & 1), columns + 8 (r >> 1)
                    const int hh = r & 1;
                    const float sx = v[j + (r >> 1)][2 * hh], sy = v[j + (r >> 1)][2 * hh + 1];
                    const float x = sx > -1e29f ? exp2f(sx - m_run[hh]) : 0.f, y = sy > -1e29f ? exp2f(sy - m_run[hh]) : 0.f;
                    l_run[hh] += x + y;
                    ah[r] = sa_pack<T>(x, y);
                    al[r] = sa_pack<T>(x - round_to<T>(x), y - round_to<T>(y));
                }
                const T* vb = sV + (j * 8 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + g * vd + (lane >> 4) * 8;
#pragma unroll
                for (int nn = 0; nn < NV / 2; ++nn)
                    if (nn * 16 < vd) {
                        uint32_t b[4];
                        sa_ldmatrix_x4_trans(b, vb + nn * 16);
                        mma_16816_bf16(O[2 * nn], ah, b[0], b[1], O[2 * nn]);
                        mma_16816_bf16(O[2 * nn + 1], ah, b[2], b[3], O[2 * nn + 1]);
                        mma_16816_bf16(O[2 * nn], al, b[0], b[1], O[2 * nn]);
                        mma_16816_bf16(O[2 * nn + 1], al, b[2], b[3], O[2 * nn + 1]);
                    }
            }
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
            if (tq == 0) part[0] = empty ? -INFINITY : m_run[hh] * kLn2, part[1] = empty ? 0.f : l_run[hh];
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

constexpr int kMhSmemMax = 225 * 1024, kMhSmemTwo = 112 * 1024;   // one CTA per SM, two CTAs per SM

static MixedShape mixed_layout(int H, int G, int d, int vd, int blocks, int kt) {
    MixedShape s{};
    const size_t rows = (size_t)G * blocks * 16, nq = (size_t)16 / (H / G) * blocks;
    s.blocks = blocks, s.h16 = (H + 15) / 16 * 16;
    s.v_off = (size_t)2 * kt * (G * d + 8);
    s.s_off = s.v_off + (size_t)2 * kt * (G * vd + 8);
    s.y_off = s.s_off + (size_t)2 * 3 * nq * s.h16 * (kt + 8);
    s.a_off = s.y_off + 4 * rows * (kt + 8);
    if (s.a_off < 2 * rows * (d + 8)) s.a_off = 2 * rows * (d + 8);   // the queries pass through the front
    s.t_off = s.a_off + (size_t)2 * s.h16 * (s.h16 + 8);
    s.bytes = s.t_off + (size_t)4 * s.h16;
    return s;
}

// token blocks per CTA: as many as make up eight warps, no more than the longest run needs (max_tokens 0: unknown)
static int mixed_blocks(int H, int G, int max_tokens) {
    const int nb = 16 / (H / G), full = G >= 8 ? 1 : 8 / G, need = max_tokens > 0 ? cdiv(max_tokens, nb) : full;
    return full < need ? full : need;
}
static bool mixed_sizes_ok(int H, int G, int d, int vd) {
    return d % 16 == 0 && vd % 16 == 0 && vd <= 128 && d <= 256 && H / G <= 16 && G <= 16 && H <= 64;
}
// keys per tile (16 or 32) and CTAs per SM; false: the sizes do not suit the tensor-core kernel
static bool mixed_shape(int H, int G, int d, int vd, int max_tokens, MixedShape& s, int& kt, int& ctas) {
    if (!mixed_sizes_ok(H, G, d, vd)) return false;
    const int blocks = mixed_blocks(H, G, max_tokens);
    if (G * blocks <= 8 && d <= 128)
        for (kt = 32; kt >= 16; kt >>= 1) {
            s = mixed_layout(H, G, d, vd, blocks, kt);
            ctas = 2;
            if (s.bytes <= (size_t)kMhSmemTwo) return true;
        }
    kt = 16, ctas = 1;
    s = mixed_layout(H, G, d, vd, blocks, kt);
    if (s.bytes > (size_t)kMhSmemMax) s = mixed_layout(H, G, d, vd, 1, kt);
    return s.bytes <= (size_t)kMhSmemMax;
}

template <int NV, int ND, int KT, int NT, int NB>
static cudaError_t launch_mixed(const MixedP& pp, const MixedShape& s, dim3 grid, bool pdl, cudaStream_t st) {
    static size_t set_for = 0;
    if (s.bytes > 48 * 1024 && s.bytes > set_for) {
        const cudaError_t e = cudaFuncSetAttribute(k_mixed_head_mma<NV, ND, KT, NT, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s.bytes);
        if (e != cudaSuccess) return e;
        set_for = s.bytes;
    }
    const int warps = pp.a.G * s.blocks;   // at least eight warps: spare ones help to load and mix
    return launch(k_mixed_head_mma<NV, ND, KT, NT, NB>, grid, dim3(32 * (warps < 8 ? 8 : warps)), s.bytes, st, pdl, pp, s);
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

// a CTA holds every head of its tokens: at most two CTAs per SM in one wave, no split shorter than 32 keys, at most 32
extern "C" int zl_mixed_head_attention_splits(int T, int runs, int heads, int kv_heads, int dim, int vdim, int max_len) {
    if (T <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads) return 1;
    int ctas = T;
    if (runs > 0 && mixed_sizes_ok(heads, kv_heads, dim, vdim)) {
        const int per = 16 / (heads / kv_heads) * mixed_blocks(heads, kv_heads, T - runs + 1);
        ctas = cdiv(T, per) > runs ? cdiv(T, per) : runs;
    }
    const int want = 2 * device_sm_count() / ctas, cap = max_len / 32 > 0 ? max_len / 32 : 1;
    int s = want < cap ? want : cap;
    if (s > 32) s = 32;
    return s < 1 ? 1 : s;
}

extern "C" int zl_mixed_head_attention(const void* q, void* const* k_addrs, void* const* v_addrs, const int32_t* slot,
                                       const int32_t* pos, const float* mix, const float* factor, int window, void* out, int T, int heads, int kv_heads,
                                       int dim, int vdim, int splits, void* workspace, size_t workspace_bytes,
                                       const int32_t* run_row0, const int32_t* run_len, int runs, int max_run_len, int dtype,
                                       int pdl, zl_stream_t stream) {
    ZL_CHECK_ARG(q && k_addrs && v_addrs && slot && pos && mix && factor && out && T > 0 && T <= 65535 && heads > 0 && kv_heads > 0);
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
    pp.factor = factor;
    pp.run_row0 = run_row0;
    pp.run_len = run_len;
    static const bool no_mma = getenv("ZL_MIXED_HEAD_NO_MMA") != nullptr;
    MixedShape sh;
    int kt = 0, ctas = 0;
    if (!no_mma && dtype == ZL_BF16 && run_row0 && run_len && runs > 0 && max_run_len > 0 &&
        mixed_shape(heads, kv_heads, dim, vdim, max_run_len, sh, kt, ctas)) {
        ZL_CHECK_ARG((long long)runs * splits <= 65535);
        const dim3 grid(cdiv(max_run_len, 16 / (heads / kv_heads) * sh.blocks), 1, runs * splits);
        cudaError_t e;
        if (ctas == 2 && kt == 32) {
            e = vdim <= 64 && dim <= 64 ? launch_mixed<8, 4, 32, 256, 2>(pp, sh, grid, pdl != 0, stream)
                                        : launch_mixed<16, 8, 32, 256, 2>(pp, sh, grid, pdl != 0, stream);
        } else if (ctas == 2) e = launch_mixed<16, 8, 16, 256, 2>(pp, sh, grid, pdl != 0, stream);
        else if (kv_heads * sh.blocks > 8) e = launch_mixed<16, 16, 16, 512, 1>(pp, sh, grid, pdl != 0, stream);
        else e = launch_mixed<16, 16, 16, 256, 1>(pp, sh, grid, pdl != 0, stream);
        ZL_CHECK_CUDA(e);
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
