// Host-side driver of the Dekalorn model family: weights, slot caches, the per-step kernel chain and its CUDA graph.
// Same driver shape as dizizen_runner.cu (task slots, host (token, slot, position) rows in, logits / greedy picks out),
// built from the shared pieces of runner_common.cuh.
//
// Pre-norm layers on an fp32 stream x: x += mixer(w rms(x)), x += ff(w rms(x)).  The layers of a step are a list of *runs*: a
// looped range of layers appears once per pass, with the same weights and caches of its own.  Before a pass
// x <- W_in [x; x0]: the concatenation's second half is written once per step by the embedding kernel, its first half by
// whatever kernel updated x last.  Everything that is a Linear of the mixer's input is ONE projection with fp32 output.
//   latent:        [W_q; W_dkv; W_g] -> rotation of the queries' and the shared key part, norm of the latent, append
//                  (latent_attn.cu) -> queries absorbed through W_uk per head -> attention over the cached latents with the
//                  rotated part as extra score columns and the sigmoid gate per head on its output -> W_uv per head -> W_o.
//   differential:  [W_q; W_k; W_v; W_g] -> append -> two softmax maps per head in a sliding window, their difference, norm and
//                  gate in one kernel (sink_attn.cu) -> W_o.
//   mixed heads:   [W_q; W_k; W_v] -> rotation, append -> attention with the heads' scores mixed before the softmax
//                  (mixed_head_attn.cu) -> W_o.
//   residual:      one kernel adds a sublayer's result (for experts: the weighted sum of a token's choices, in their order)
//                  and writes the next sublayer's normed input.
//   dense ff:      [W_gate; W_up] with rows interleaved and relu(gate) * up as the epilogue, then W_down.
//   experts:       routing on the device (moe_route.cu) -> two grouped GEMMs over the (token, choice) pairs, the silu-gated
//                  unit as the first one's epilogue.
// One step takes T rows in any mix of prompt portions and single decode tokens; every kernel indexes caches by
// (slot, position).
#include "runner_common.cuh"

#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

namespace {

using namespace zl;

struct KLayer {
    zl_dekalorn_layer_t c{};
    float *norm1 = nullptr, *norm2 = nullptr;
    void* w_in = nullptr;                        // fused projection (n_in, width)
    int n_in = 0, k_off = 0, v_off = 0, g_off = 0, c_off = 0;   // columns of the projection (queries at 0)
    void* o = nullptr;                           // (width, heads * vdim)
    // latent
    int rank_cols = 0, row_cols = 0;             // padded latent columns, columns of a cached row
    float* dkv_norm = nullptr;
    void *uk_t = nullptr, *uv = nullptr;         // (heads, rank_cols, dim), (heads * vdim, rank_cols)
    // differential / mixed heads
    float lambda = 0.f;
    float *mix = nullptr, *factor = nullptr;     // (heads, heads), (heads): temperature times scale
    int rot = -1;                                // index into the model's rotation tables
    // feed-forward
    void* w_gu = nullptr;                        // dense (2 * ff, width), experts (experts, 2 * ff, width): rows 2j / 2j+1 = gate_j / up_j
    void* w_down = nullptr;                      // dense (width, ff), experts (experts, width, ff)
    void* router = nullptr;                      // (experts, width)
    bool ready = false;
};

// one layer in the order of a step, with the caches of this pass
struct KRun {
    int layer = 0;
    bool enters = false;                         // first layer of a pass of the loop
    SlotCache a, b;                              // latent: rows in a; otherwise keys in a, values in b
};

// one (cos, sin) table per distinct (base, size, scaling): filled once per step from the rows' positions
struct RotTable {
    double base = 0, factor = 0, low = 0, high = 0, original = 0;
    int dims = 0;
    double* inv_freq = nullptr;   // device (dims / 2)
    float* table = nullptr;       // device (tcap, dims / 2) float pairs
};

}  // namespace

struct zl_dekalorn {
    zl_dekalorn_config_t cfg{};
    cudaStream_t stream = nullptr;
    StagedMap staged;
    std::vector<KLayer> layers;
    std::vector<KRun> runs;
    std::vector<RotTable> rots;
    void *embed = nullptr, *head = nullptr, *loop_in = nullptr;
    float* final_norm = nullptr;
    bool finalized = false;
    int esz = 2;
    int tcap = 0;
    float *x = nullptr, *proj = nullptr, *y = nullptr, *qa = nullptr, *xw = nullptr, *logits = nullptr, *top_w = nullptr;
    void *h = nullptr, *xcat = nullptr, *q = nullptr, *olat = nullptr, *att = nullptr, *act = nullptr, *xn = nullptr;
    int32_t *d_tokens = nullptr, *d_slots = nullptr, *d_pos = nullptr, *d_want = nullptr, *d_next = nullptr;
    int32_t *d_run0 = nullptr, *d_runlen = nullptr, *top_e = nullptr, *grp_off = nullptr, *list_token = nullptr,
            *list_pair = nullptr;
    int32_t* h_stage = nullptr;   // pinned: tokens | slots | pos | want | next | run0 | runlen
    void* attn_ws = nullptr;
    size_t attn_ws_bytes = 0;
    void* argmax_ws = nullptr;
    float* layer_dump = nullptr;
    bool capture = false;
    std::map<long long, cudaGraphExec_t> graphs;
    int cur_max_len = 0;
    double weight_bytes = 0;
    int kernels_per_step = 0;
};

namespace {

int fail(int line, const std::string& msg, int code = ZL_ERR_STATE) {
    zl_set_last_error(__FILE__, line, msg.c_str());
    return code;
}

int rot_index(zl_dekalorn* m, const zl_dekalorn_layer_t& c) {
    for (size_t i = 0; i < m->rots.size(); ++i) {
        const RotTable& r = m->rots[i];
        if (r.base == c.rot_base && r.dims == c.rot_dims && r.factor == c.rot_factor && r.low == c.rot_low && r.high == c.rot_high &&
            r.original == c.rot_original)
            return (int)i;
    }
    RotTable r;
    r.base = c.rot_base, r.dims = c.rot_dims;
    r.factor = c.rot_factor, r.low = c.rot_low, r.high = c.rot_high, r.original = c.rot_original;
    m->rots.push_back(r);
    return (int)m->rots.size() - 1;
}

int finalize_ff(zl_dekalorn* m, int l) {
    KLayer& L = m->layers[l];
    const auto& lc = L.c;
    const int D = m->cfg.width, F = lc.ff;
    const std::string p = "l" + std::to_string(l) + ".mlp.";
    RCHECK(take_f32(m, "l" + std::to_string(l) + ".norm2", 1, D, &L.norm2));
    if (lc.ff_kind == ZL_FF_DENSE) {
        RCHECK(dmalloc(&L.w_gu, (size_t)2 * F * D * m->esz));
        RCHECK(put_interleaved(m, p + "gate", p + "up", F, D, L.w_gu, 0, false));
        return take_weight(m, p + "down", D, F, &L.w_down);
    }
    const int E = lc.experts;
    RCHECK(take_weight(m, p + "router", E, D, &L.router));
    RCHECK(dmalloc(&L.w_gu, (size_t)E * 2 * F * D * m->esz));
    RCHECK(dmalloc(&L.w_down, (size_t)E * D * F * m->esz));
    for (int e = 0; e < E; ++e) {
        const std::string pe = p + "e" + std::to_string(e) + ".";
        RCHECK(put_interleaved(m, pe + "gate", pe + "up", F, D, L.w_gu, (size_t)e * 2 * F * D, false));
        RCHECK(put_weight(m, pe + "down", D, F, L.w_down, (size_t)e * D * F));
    }
    return ZL_OK;
}

int finalize_layer(zl_dekalorn* m, int l) {
    KLayer& L = m->layers[l];
    const auto& lc = L.c;
    const std::string p = "l" + std::to_string(l) + ".", mx = p + "mix.";
    const int D = m->cfg.width, H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
    RCHECK(take_f32(m, p + "norm1", 1, D, &L.norm1));
    // (name, rows) of the fused projection's segments in order
    std::vector<std::pair<std::string, int>> seg;
    if (lc.type == ZL_DEKALORN_LATENT) {
        seg = {{"q", H * (d + lc.rot_dim)}, {"dkv", lc.kv_rank + lc.rot_dim}, {"g", H}};
        L.c_off = seg[0].second;
        L.g_off = L.c_off + seg[1].second;
    } else if (lc.type == ZL_DEKALORN_DIFF) {
        seg = {{"q", H * 2 * d}, {"k", G * 2 * d}, {"v", G * vd}, {"g", H * vd}};
        L.k_off = seg[0].second;
        L.v_off = L.k_off + seg[1].second;
        L.g_off = L.v_off + seg[2].second;
    } else {
        seg = {{"q", H * d}, {"k", G * d}, {"v", G * vd}};
        L.k_off = seg[0].second;
        L.v_off = L.k_off + seg[1].second;
    }
    for (auto& s : seg) L.n_in += s.second;
    L.n_in = round_up(L.n_in, 8);   // rows of zeros behind the last segment
    RCHECK(dmalloc(&L.w_in, (size_t)L.n_in * D * m->esz));
    ZL_CHECK_CUDA(cudaMemsetAsync(L.w_in, 0, (size_t)L.n_in * D * m->esz, m->stream));
    int at = 0;
    for (auto& s : seg) {
        RCHECK(put_weight(m, mx + s.first, s.second, D, L.w_in, (size_t)at * D));
        at += s.second;
    }
    if (lc.type == ZL_DEKALORN_LATENT) {
        // 16-bit runs pad the latent to the tensor-core kernel's column step and the rotated part to its contraction step (zero
        // weights and never-written cache columns)
        const bool f32 = m->cfg.dtype == ZL_F32;
        L.rank_cols = f32 ? lc.kv_rank : round_up(lc.kv_rank, lc.kv_rank <= 512 ? 64 : 8);
        L.row_cols = L.rank_cols + (f32 ? lc.rot_dim : round_up(lc.rot_dim, 16));
        RCHECK(take_f32(m, mx + "dkv.norm", 1, lc.kv_rank, &L.dkv_norm));
        RCHECK(take_latent(m, mx + "uk", true, H, d, lc.kv_rank, L.rank_cols, &L.uk_t));
        RCHECK(take_latent(m, mx + "uv", false, H, vd, lc.kv_rank, L.rank_cols, &L.uv));
    } else if (lc.type == ZL_DEKALORN_DIFF) {
        std::vector<double> v[4];
        const char* names[4] = {"lq1", "lk1", "lq2", "lk2"};
        for (int i = 0; i < 4; ++i) RCHECK(take_host(m, mx + names[i], 1, d, v[i]));
        double s1 = 0, s2 = 0;
        for (int i = 0; i < d; ++i) s1 += v[0][i] * v[1][i], s2 += v[2][i] * v[3][i];
        L.lambda = (float)(exp(s1) - exp(s2) + (double)lc.diff);
    } else {
        std::vector<double> temp, talk;
        RCHECK(take_host(m, mx + "temp", 1, H, temp));
        RCHECK(take_host(m, mx + "talk", H, H, talk));
        std::vector<float> mix(talk.begin(), talk.end()), factor(H);
        for (int h = 0; h < H; ++h) factor[h] = (float)(temp[h] * (double)lc.scale);
        RCHECK(dmalloc((void**)&L.mix, mix.size() * 4));
        ZL_CHECK_CUDA(cudaMemcpy(L.mix, mix.data(), mix.size() * 4, cudaMemcpyHostToDevice));
        RCHECK(dmalloc((void**)&L.factor, factor.size() * 4));
        ZL_CHECK_CUDA(cudaMemcpy(L.factor, factor.data(), factor.size() * 4, cudaMemcpyHostToDevice));
    }
    RCHECK(take_weight(m, mx + "o", D, H * vd, &L.o));
    if (lc.ff_kind != ZL_FF_NONE) RCHECK(finalize_ff(m, l));
    if (lc.rot_dims > 0) L.rot = rot_index(m, lc);
    L.ready = true;
    return ZL_OK;
}

int len_bucket(const zl_dekalorn* m, int max_len) {
    int b = 256;
    while (b < max_len) b <<= 1;
    return b < m->cfg.max_seq ? b : (m->cfg.max_seq > 256 ? m->cfg.max_seq : 256);
}

int attn_splits(const zl_dekalorn_layer_t& lc, int rank_cols, int T, int n_runs, int max_len) {
    const int len = lc.window > 0 && lc.window < max_len ? lc.window : max_len;
    if (lc.type == ZL_DEKALORN_LATENT) return zl_latent_attention_splits(T, lc.heads, rank_cols, max_len);
    if (lc.type == ZL_DEKALORN_DIFF) return zl_sink_attention_splits(T, lc.heads, lc.kv_heads, len);
    return zl_mixed_head_attention_splits(T, n_runs, lc.heads, lc.kv_heads, lc.dim, lc.vdim, len);
}

int alloc_runtime(zl_dekalorn* m) {
    const auto& c = m->cfg;
    const int D = c.width, T = m->tcap, B = c.max_batch;
    size_t n_in = 1, hd = 1, hv = 1, hr = 1, ha = 1, ffw = 1, top = 1, experts = 1;
    for (auto& L : m->layers) {
        const auto& lc = L.c;
        const bool latent = lc.type == ZL_DEKALORN_LATENT;
        const int maps = lc.type == ZL_DEKALORN_DIFF ? 2 : 1;
        if (latent) RCHECK(zl_latent_attention_prepare_ex(lc.heads, L.rank_cols, L.row_cols, c.dtype));
        // the split count falls as the rows grow and depends on how they form runs: size for the worst product
        const int len = len_bucket(m, c.max_seq);
        for (int b = 1; b <= T; ++b) {
            const int s = std::max(attn_splits(lc, L.rank_cols, b, 1, len), attn_splits(lc, L.rank_cols, b, b, len));
            m->attn_ws_bytes = std::max(m->attn_ws_bytes, latent ? zl_latent_attention_workspace_bytes(b, lc.heads, L.rank_cols, s)
                                                                 : zl_sink_attention_workspace_bytes(b, lc.heads * maps, lc.vdim, s));
        }
        n_in = std::max(n_in, (size_t)L.n_in);
        hd = std::max(hd, (size_t)lc.heads * lc.dim * maps);
        hv = std::max(hv, (size_t)lc.heads * lc.vdim);
        if (latent) {
            hr = std::max(hr, (size_t)lc.heads * L.rank_cols);
            ha = std::max(ha, (size_t)lc.heads * L.row_cols);
        }
        if (lc.ff_kind == ZL_FF_DENSE) ffw = std::max(ffw, (size_t)lc.ff);
        if (lc.ff_kind == ZL_FF_MOE) {
            ffw = std::max(ffw, (size_t)lc.top * lc.ff);
            top = std::max(top, (size_t)lc.top);
            experts = std::max(experts, (size_t)lc.experts);
        }
    }
    for (auto& U : m->runs) {
        const KLayer& L = m->layers[U.layer];
        const auto& lc = L.c;
        if (lc.type == ZL_DEKALORN_LATENT) {
            RCHECK(U.a.create(B, (size_t)c.max_seq * L.row_cols * m->esz, m->stream));
        } else {
            const int maps = lc.type == ZL_DEKALORN_DIFF ? 2 : 1;
            RCHECK(U.a.create(B, (size_t)c.max_seq * lc.kv_heads * lc.dim * maps * m->esz, m->stream));
            RCHECK(U.b.create(B, (size_t)c.max_seq * lc.kv_heads * lc.vdim * m->esz, m->stream));
        }
    }
    for (auto& r : m->rots) {
        const int half = r.dims / 2;
        std::vector<double> f(half);
        RCHECK(zl_rope_inv_freq_wavelength(r.base, r.dims, r.factor, r.low, r.high, r.original, f.data()));
        RCHECK(dmalloc((void**)&r.inv_freq, (size_t)half * 8));
        ZL_CHECK_CUDA(cudaMemcpy(r.inv_freq, f.data(), (size_t)half * 8, cudaMemcpyHostToDevice));
        RCHECK(dmalloc((void**)&r.table, (size_t)T * half * 8));
    }
    const size_t e = m->esz;
    RCHECK(dmalloc((void**)&m->x, (size_t)T * D * 4));
    RCHECK(dmalloc((void**)&m->proj, (size_t)T * n_in * 4));
    RCHECK(dmalloc((void**)&m->y, (size_t)T * top * D * 4));
    RCHECK(dmalloc((void**)&m->qa, (size_t)T * ha * 4));
    ZL_CHECK_CUDA(cudaMemsetAsync(m->qa, 0, (size_t)T * ha * 4, m->stream));   // padding columns are never written: keep them finite
    RCHECK(dmalloc((void**)&m->xw, (size_t)T * D * 4));
    RCHECK(dmalloc((void**)&m->logits, (size_t)T * c.vocab * 4));
    RCHECK(dmalloc((void**)&m->top_w, (size_t)T * top * 4));
    RCHECK(dmalloc(&m->h, (size_t)T * D * e));
    RCHECK(dmalloc(&m->xcat, (size_t)T * 2 * D * e));
    RCHECK(dmalloc(&m->q, (size_t)T * hd * e));
    RCHECK(dmalloc(&m->olat, (size_t)T * hr * e));
    RCHECK(dmalloc(&m->att, (size_t)T * hv * e));
    RCHECK(dmalloc(&m->act, (size_t)T * ffw * e));
    RCHECK(dmalloc(&m->xn, (size_t)T * D * e));
    for (int32_t** p : {&m->d_tokens, &m->d_slots, &m->d_pos, &m->d_want, &m->d_next, &m->d_run0, &m->d_runlen})
        RCHECK(dmalloc((void**)p, (size_t)T * 4));
    RCHECK(dmalloc((void**)&m->top_e, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->list_token, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->list_pair, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->grp_off, (experts + 1) * 4));
    RCHECK(dmalloc(&m->attn_ws, m->attn_ws_bytes));
    RCHECK(dmalloc(&m->argmax_ws, zl_argmax_workspace_bytes(T)));
    ZL_CHECK_CUDA(cudaMallocHost((void**)&m->h_stage, sizeof(int32_t) * 7 * (size_t)T));
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

// Which kernels of a step of at most 8 rows are launched with a programmatic dependency: 1 skinny Linears, 2 other GEMMs,
// 4 row kernels, 8 attention, 32 the tail.  Larger steps use none.  ZL_DEKALORN_PDL_MASK overrides the default.
constexpr int kDefaultPdlMask = 1;
int pdl_mask() {
    static int v = -1;
    if (v < 0) {
        const char* e = getenv("ZL_DEKALORN_PDL_MASK");
        v = e ? atoi(e) : kDefaultPdlMask;
    }
    return v;
}
int pdl_for(const zl_dekalorn* m, int bit, int T) { return (m->cfg.use_pdl && T <= 8 && (pdl_mask() & bit)) ? 1 : 0; }

// y (M, N) = x (M, K) @ w (N, K)^T
int linear(zl_dekalorn* m, const void* x, int K, const void* w, int N, void* y, int M, int out_dtype) {
    const auto& c = m->cfg;
    if (c.dtype != ZL_F32 && M <= 32 && K % 32 == 0 && N >= 64 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 &&
        (reinterpret_cast<uintptr_t>(w) & 15) == 0)
        return zl_dense_gemm_skinny_act(x, K, w, nullptr, y, M, N, K, c.dtype, out_dtype, 0, pdl_for(m, 1, M), m->stream);
    return zl_gemm_nt_bias(x, K, w, K, nullptr, y, N, M, N, K, c.dtype, out_dtype, ZL_GEMM_EPI_NONE, pdl_for(m, 2, M), m->stream);
}

int enqueue_mixer(zl_dekalorn* m, KRun& U, int T, int n_runs, int max_run, int max_len) {
    const auto& c = m->cfg;
    KLayer& L = m->layers[U.layer];
    const auto& lc = L.c;
    const int D = c.width, dt = c.dtype, H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
    const int pg = pdl_for(m, 2, T), pr = pdl_for(m, 4, T), pa = pdl_for(m, 8, T);
    cudaStream_t st = m->stream;
    const float* tab = L.rot >= 0 ? m->rots[L.rot].table : nullptr;
    const int splits = attn_splits(lc, L.rank_cols, T, n_runs, max_len);
    RCHECK(linear(m, m->h, D, L.w_in, L.n_in, m->proj, T, ZL_F32));
    if (lc.type == ZL_DEKALORN_LATENT) {
        const int RC = L.rank_cols, RS = L.row_cols;
        RCHECK(zl_latent_rope_append(m->proj, L.n_in, 0, H, d, lc.rot_dim, tab, m->q, m->qa, L.c_off, lc.kv_rank, L.dkv_norm, RC, RS,
                                     U.a.addrs, m->d_slots, m->d_pos, T, c.eps, dt, pr, st));
        RCHECK(zl_gemm_nt(m->q, (long long)H * d, d, L.uk_t, d, (long long)RC * d, m->qa, (long long)H * RS, RS, T, RC, d, H, dt, ZL_F32,
                          ZL_GEMM_EPI_NONE, nullptr, 0, 0, pg, st));
        RCHECK(zl_latent_attention_ex(m->qa, U.a.addrs, m->d_slots, m->d_pos, nullptr, m->proj + L.g_off, L.n_in, lc.scale, m->olat, T, H,
                                      RC, RS, splits, m->attn_ws, m->attn_ws_bytes, m->d_run0, m->d_runlen, n_runs, max_run, dt, pa,
                                      st));
        RCHECK(zl_gemm_nt(m->olat, (long long)H * RC, RC, L.uv, RC, (long long)vd * RC, m->att, (long long)H * vd, vd, T, vd, RC, H, dt,
                          dt, ZL_GEMM_EPI_NONE, nullptr, 0, 0, pg, st));
    } else if (lc.type == ZL_DEKALORN_DIFF) {
        // no rotation: a head's two maps travel as one head of twice the size
        RCHECK(zl_qkv_table_rope_append(m->proj, L.n_in, 0, L.k_off, L.v_off, H, G, 2 * d, vd, nullptr, 0, nullptr, ZL_ROT_ADJACENT,
                                        m->q, U.a.addrs, U.b.addrs, m->d_slots, m->d_pos, T, dt, pr, st));
        RCHECK(zl_window_attention(m->q, U.a.addrs, U.b.addrs, m->d_slots, m->d_pos, lc.scale, lc.window, 2, L.lambda, c.eps,
                                   1.0f - lc.diff, m->proj + L.g_off, L.n_in, m->att, T, H, G, d, vd, splits, m->attn_ws,
                                   m->attn_ws_bytes, m->d_run0, m->d_runlen, n_runs, max_run, dt, pa, st));
    } else {
        RCHECK(zl_qkv_table_rope_append(m->proj, L.n_in, 0, L.k_off, L.v_off, H, G, d, vd, tab, lc.rot_dims, nullptr, ZL_ROT_ADJACENT,
                                        m->q, U.a.addrs, U.b.addrs, m->d_slots, m->d_pos, T, dt, pr, st));
        RCHECK(zl_mixed_head_attention(m->q, U.a.addrs, U.b.addrs, m->d_slots, m->d_pos, L.mix, L.factor, lc.window, m->att, T, H, G, d, vd,
                                       splits, m->attn_ws, m->attn_ws_bytes, m->d_run0, m->d_runlen, n_runs, max_run, dt, pa, st));
    }
    return linear(m, m->att, H * vd, L.o, D, m->y, T, ZL_F32);
}

int enqueue_step(zl_dekalorn* m, int T, int n_want, int n_runs, int max_run, int max_len) {
    const auto& c = m->cfg;
    const int D = c.width, dt = c.dtype;
    cudaStream_t st = m->stream;
    const int pg = pdl_for(m, 2, T), pr = pdl_for(m, 4, T), pt = pdl_for(m, 32, T);
    const size_t e = m->esz;
    void* x0_half = static_cast<char*>(m->xcat) + (size_t)D * e;   // columns D .. 2 D of [x; x0]
    const bool loop = m->loop_in != nullptr;
    const bool enters0 = m->runs[0].enters;
    RCHECK(zl_embed_norm(m->d_tokens, m->embed, c.vocab, m->x, enters0 ? nullptr : m->layers[m->runs[0].layer].norm1, m->h,
                         loop ? x0_half : nullptr, enters0 ? m->xcat : nullptr, 2 * D, dt, T, D, c.eps, 0, st));
    for (auto& r : m->rots) RCHECK(zl_rope_table(m->d_pos, T, r.inv_freq, r.dims / 2, r.table, pr, st));
    for (size_t u = 0; u < m->runs.size(); ++u) {
        KRun& U = m->runs[u];
        KLayer& L = m->layers[U.layer];
        const auto& lc = L.c;
        if (U.enters) {
            RCHECK(linear(m, m->xcat, 2 * D, m->loop_in, D, m->x, T, ZL_F32));
            RCHECK(zl_residual_norm(m->x, D, nullptr, 0, nullptr, 0, L.norm1, m->h, nullptr, 0, dt, T, D, c.eps, pr, st));
        }
        RCHECK(enqueue_mixer(m, U, T, n_runs, max_run, max_len));
        // what the run's last update of x also writes: the next run's normed input, or x itself for the next pass
        const KRun* next = u + 1 < m->runs.size() ? &m->runs[u + 1] : nullptr;
        const float* next_w = next && !next->enters ? m->layers[next->layer].norm1 : nullptr;
        void* copy = next && next->enters ? m->xcat : nullptr;
        const bool ff = lc.ff_kind != ZL_FF_NONE;
        RCHECK(zl_residual_norm(m->x, D, m->y, D, nullptr, 1, ff ? L.norm2 : next_w, m->h, ff ? nullptr : copy, 2 * D, dt, T, D, c.eps,
                                pr, st));
        if (lc.ff_kind == ZL_FF_DENSE) {
            RCHECK(zl_gemm_nt_fused(m->h, D, L.w_gu, D, nullptr, m->act, lc.ff, T, 2 * lc.ff, D, dt, dt, ZL_GEMM_EPI_REGLU, nullptr, 0,
                                    0.f, pg, st));
            RCHECK(linear(m, m->act, lc.ff, L.w_down, D, m->y, T, ZL_F32));
            RCHECK(zl_residual_norm(m->x, D, m->y, D, nullptr, 1, next_w, m->h, copy, 2 * D, dt, T, D, c.eps, pr, st));
        } else if (lc.ff_kind == ZL_FF_MOE) {
            const int E = lc.experts, F = lc.ff;
            RCHECK(zl_moe_route_ex(m->h, D, L.router, dt, nullptr, m->top_e, m->top_w, m->grp_off, m->list_token, m->list_pair, T, D, E,
                                   lc.top, lc.groups, lc.keep, ZL_MOE_GROUP_TOP2, ZL_MOE_SCORE_SIGMOID, 1, 1e-20f, lc.router_scale, pr,
                                   st));
            // g sigmoid(g) u: the clamped unit without its clamp
            RCHECK(zl_gemm_nt_grouped(m->h, D, m->list_token, L.w_gu, D, (long long)2 * F * D, m->act, F, nullptr, m->grp_off, E, T, 2 * F,
                                      D, dt, dt, ZL_GEMM_EPI_GLU_CLAMP, INFINITY, 1.f, 0.f, pg, st));
            RCHECK(zl_gemm_nt_grouped(m->act, F, nullptr, L.w_down, F, (long long)D * F, m->y, D, m->list_pair, m->grp_off, E, T, D, F,
                                      dt, ZL_F32, ZL_GEMM_EPI_NONE, 0.f, 1.f, 0.f, pg, st));
            RCHECK(zl_residual_norm(m->x, D, m->y, D, m->top_w, lc.top, next_w, m->h, copy, 2 * D, dt, T, D, c.eps, pr, st));
        }
        if (m->capture && m->layer_dump)
            ZL_CHECK_CUDA(cudaMemcpyAsync(m->layer_dump + u * m->tcap * D, m->x, (size_t)T * D * 4, cudaMemcpyDeviceToDevice, st));
    }
    if (n_want > 0) {
        ZL_CHECK_CUDA(launch(k_gather_rows_f32, dim3(n_want), dim3(128), 0, st, false, (const float*)m->x,
                             (const int32_t*)m->d_want, m->xw, D));
        RCHECK(zl_group_rmsnorm(m->xw, D, m->final_norm, m->xn, D, n_want, D, 1, c.eps, dt, pt, st));
        RCHECK(linear(m, m->xn, D, m->head, c.vocab, m->logits, n_want, ZL_F32));
        RCHECK(zl_argmax(m->logits, m->d_next, n_want, c.vocab, m->argmax_ws, zl_argmax_workspace_bytes(n_want), pt, st));
    }
    return ZL_OK;
}

// decode-sized steps replay a CUDA graph per (rows, wanted rows, runs, length bucket); prompt portions are enqueued directly
// (max_run: the longest run; a captured step is sized for the longest run its row count allows)
int run_step(zl_dekalorn* m, int T, int n_want, int n_runs, int max_run, int max_len) {
    const int bucket = len_bucket(m, max_len);
    if (!m->cfg.use_graph || T > m->cfg.max_batch || m->capture) return enqueue_step(m, T, n_want, n_runs, max_run, bucket);
    const long long key = ((long long)T << 48) | ((long long)n_want << 32) | ((long long)n_runs << 16) | (long long)(bucket >> 8);
    auto it = m->graphs.find(key);
    if (it == m->graphs.end()) {
        cudaGraph_t graph = nullptr;
        ZL_CHECK_CUDA(cudaStreamBeginCapture(m->stream, cudaStreamCaptureModeThreadLocal));
        const int rc = enqueue_step(m, T, n_want, n_runs, T - n_runs + 1, bucket);
        const cudaError_t ce = cudaStreamEndCapture(m->stream, &graph);
        if (rc != ZL_OK) {
            if (graph) cudaGraphDestroy(graph);
            return rc;
        }
        ZL_CHECK_CUDA(ce);
        cudaGraphExec_t exec = nullptr;
        ZL_CHECK_CUDA(cudaGraphInstantiate(&exec, graph, 0));
        size_t n_nodes = 0;
        cudaGraphGetNodes(graph, nullptr, &n_nodes);
        m->kernels_per_step = (int)n_nodes;
        cudaGraphDestroy(graph);
        it = m->graphs.emplace(key, exec).first;
    }
    ZL_CHECK_CUDA(cudaGraphLaunch(it->second, m->stream));
    return ZL_OK;
}

}  // namespace

extern "C" int zl_dekalorn_create(const zl_dekalorn_config_t* cfg, const zl_dekalorn_layer_t* layers, zl_dekalorn_t** out) {
    ZL_CHECK_ARG(cfg && layers && out);
    ZL_CHECK_ARG(cfg->num_layers > 0 && cfg->width > 0 && cfg->vocab > 0 && cfg->max_batch > 0 && cfg->max_seq > 0);
    ZL_CHECK_ARG(cfg->eps >= 0.f);
    ZL_CHECK_SUPPORTED(cfg->dtype == ZL_BF16 || cfg->dtype == ZL_F32);
    ZL_CHECK_ARG(cfg->max_step_tokens >= 0 && cfg->max_step_tokens <= 65535);
    ZL_CHECK_ARG(cfg->loop_times == 0 || (cfg->loop_times > 0 && cfg->loop_start >= 0 && cfg->loop_start < cfg->loop_stop &&
                                          cfg->loop_stop <= cfg->num_layers));
    for (int l = 0; l < cfg->num_layers; ++l) {
        const auto& lc = layers[l];
        ZL_CHECK_ARG(lc.type == ZL_DEKALORN_LATENT || lc.type == ZL_DEKALORN_DIFF || lc.type == ZL_DEKALORN_MIXED);
        ZL_CHECK_ARG(lc.heads > 0 && lc.dim > 0 && lc.kv_heads > 0 && lc.heads % lc.kv_heads == 0 && lc.vdim > 0 && lc.window >= 0);
        const int rot_max = lc.type == ZL_DEKALORN_LATENT ? lc.rot_dim : (lc.type == ZL_DEKALORN_MIXED ? lc.dim : 0);
        ZL_CHECK_ARG(lc.rot_dims >= 0 && lc.rot_dims <= rot_max && lc.rot_dims % 2 == 0 && (lc.rot_dims == 0 || lc.rot_base > 1.0));
        if (lc.type == ZL_DEKALORN_LATENT)
            ZL_CHECK_ARG(lc.kv_rank > 0 && lc.rot_dim >= 0 && lc.rot_dims == lc.rot_dim && lc.window == 0);
        ZL_CHECK_ARG(lc.ff_kind == ZL_FF_NONE || lc.ff_kind == ZL_FF_DENSE || lc.ff_kind == ZL_FF_MOE);
        if (lc.ff_kind != ZL_FF_NONE) ZL_CHECK_ARG(lc.ff > 0);
        if (lc.ff_kind == ZL_FF_MOE)
            ZL_CHECK_ARG(lc.experts > 0 && lc.top > 0 && lc.top <= lc.experts && lc.groups >= 1 && lc.experts % lc.groups == 0 &&
                         lc.keep >= 1 && lc.keep <= lc.groups && lc.keep * (lc.experts / lc.groups) >= lc.top);
    }
    zl_dekalorn* m = new zl_dekalorn();
    m->cfg = *cfg;
    m->esz = cfg->dtype == ZL_F32 ? 4 : 2;
    m->tcap = cfg->max_step_tokens > cfg->max_batch ? cfg->max_step_tokens : cfg->max_batch;
    m->layers.resize(cfg->num_layers);
    for (int l = 0; l < cfg->num_layers; ++l) m->layers[l].c = layers[l];
    const int a = cfg->loop_times > 0 ? cfg->loop_start : 0, b = cfg->loop_times > 0 ? cfg->loop_stop : 0;
    auto add = [&](int l, bool enters) {
        m->runs.emplace_back();
        m->runs.back().layer = l;
        m->runs.back().enters = enters;
    };
    for (int l = 0; l < a; ++l) add(l, false);
    for (int t = 0; t < cfg->loop_times; ++t)
        for (int l = a; l < b; ++l) add(l, l == a);
    for (int l = b; l < cfg->num_layers; ++l) add(l, false);
    if (cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) != cudaSuccess) {
        delete m;
        zl_set_last_error(__FILE__, __LINE__, "cudaStreamCreate failed (no CUDA device? there is no CPU fallback)");
        return ZL_ERR_CUDA;
    }
    *out = m;
    return ZL_OK;
}

extern "C" void zl_dekalorn_destroy(zl_dekalorn_t* m) {
    if (!m) return;
    cudaStreamSynchronize(m->stream);
    for (auto& g : m->graphs) cudaGraphExecDestroy(g.second);
    for (auto& s : m->staged) cudaFree(s.second.ptr);
    for (auto& L : m->layers)
        for (void* p : {(void*)L.norm1, (void*)L.norm2, L.w_in, L.o, (void*)L.dkv_norm, L.uk_t, L.uv, (void*)L.mix, (void*)L.factor, L.w_gu, L.w_down,
                        L.router})
            if (p) cudaFree(p);
    for (auto& U : m->runs) {
        U.a.destroy();
        U.b.destroy();
    }
    for (auto& r : m->rots)
        for (void* p : {(void*)r.inv_freq, (void*)r.table})
            if (p) cudaFree(p);
    for (void* p : {m->embed, m->head, m->loop_in, (void*)m->final_norm, (void*)m->x, (void*)m->proj, (void*)m->y, (void*)m->qa,
                    (void*)m->xw, (void*)m->logits, (void*)m->top_w, m->h, m->xcat, m->q, m->olat, m->att, m->act, m->xn,
                    (void*)m->d_tokens, (void*)m->d_slots, (void*)m->d_pos, (void*)m->d_want, (void*)m->d_next, (void*)m->d_run0,
                    (void*)m->d_runlen, (void*)m->top_e, (void*)m->grp_off, (void*)m->list_token, (void*)m->list_pair, m->attn_ws,
                    m->argmax_ws, (void*)m->layer_dump})
        if (p) cudaFree(p);
    if (m->h_stage) cudaFreeHost(m->h_stage);
    cudaStreamDestroy(m->stream);
    delete m;
}

extern "C" int zl_dekalorn_load_tensor(zl_dekalorn_t* m, const char* name, const void* data_host, int rows, int cols,
                                       int elem_bytes) {
    ZL_CHECK_ARG(m && name && data_host && rows > 0 && cols > 0 && (elem_bytes == 2 || elem_bytes == 4));
    if (m->finalized) return fail(__LINE__, "model already finalized");
    return staged_load(m->staged, name, data_host, rows, cols, elem_bytes, m->stream);
}

extern "C" int zl_dekalorn_finalize(zl_dekalorn_t* m) {
    ZL_CHECK_ARG(m);
    if (m->finalized) return ZL_OK;
    const int D = m->cfg.width;
    for (int l = 0; l < m->cfg.num_layers; ++l)
        if (!m->layers[l].ready) RCHECK(finalize_layer(m, l));
    if (m->cfg.loop_times > 0) RCHECK(take_weight(m, "loop.in", D, 2 * D, &m->loop_in));
    RCHECK(take_weight(m, "embed", m->cfg.vocab, D, &m->embed));
    m->weight_bytes -= (double)m->cfg.vocab * D * m->esz;   // gathered, not streamed
    RCHECK(take_weight(m, "head", m->cfg.vocab, D, &m->head));
    RCHECK(take_f32(m, "final.norm", 1, D, &m->final_norm));
    RCHECK(alloc_runtime(m));
    m->finalized = true;
    return ZL_OK;
}

extern "C" int zl_dekalorn_init_synthetic(zl_dekalorn_t* m, uint64_t seed) {
    ZL_CHECK_ARG(m);
    if (m->finalized) return fail(__LINE__, "model already finalized");
    const auto& c = m->cfg;
    const int D = c.width;
    auto lin = [&](const std::string& name, int n, int k) {
        const float a = sqrtf(3.0f / (float)k);   // unit-variance outputs for unit-variance inputs
        return stage_random(m, name, n, k, -a, a, seed);
    };
    auto ones = [&](const std::string& name, int n) { return stage_random(m, name, 1, n, 0.9f, 1.1f, seed); };
    for (int l = 0; l < c.num_layers; ++l) {
        const auto& lc = m->layers[l].c;
        const std::string p = "l" + std::to_string(l) + ".", mx = p + "mix.", ml = p + "mlp.";
        const int H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
        RCHECK(ones(p + "norm1", D));
        if (lc.type == ZL_DEKALORN_LATENT) {
            RCHECK(lin(mx + "q", H * (d + lc.rot_dim), D));
            RCHECK(lin(mx + "dkv", lc.kv_rank + lc.rot_dim, D));
            RCHECK(ones(mx + "dkv.norm", lc.kv_rank));
            RCHECK(lin(mx + "uk", H * d, lc.kv_rank));
            RCHECK(lin(mx + "uv", H * vd, lc.kv_rank));
            RCHECK(lin(mx + "g", H, D));
        } else {
            const int maps = lc.type == ZL_DEKALORN_DIFF ? 2 : 1;
            RCHECK(lin(mx + "q", H * maps * d, D));
            RCHECK(lin(mx + "k", G * maps * d, D));
            RCHECK(lin(mx + "v", G * vd, D));
            if (maps == 2) {
                for (const char* n : {"lq1", "lk1", "lq2", "lk2"}) RCHECK(stage_random(m, mx + n, 1, d, -0.1f, 0.1f, seed));
                RCHECK(lin(mx + "g", H * vd, D));
            } else {
                RCHECK(ones(mx + "temp", H));
                RCHECK(lin(mx + "talk", H, H));
            }
        }
        RCHECK(lin(mx + "o", D, H * vd));
        if (lc.ff_kind != ZL_FF_NONE) RCHECK(ones(p + "norm2", D));
        if (lc.ff_kind == ZL_FF_DENSE) {
            RCHECK(lin(ml + "gate", lc.ff, D));
            RCHECK(lin(ml + "up", lc.ff, D));
            RCHECK(lin(ml + "down", D, lc.ff));
        } else if (lc.ff_kind == ZL_FF_MOE) {
            RCHECK(lin(ml + "router", lc.experts, D));
            for (int e = 0; e < lc.experts; ++e) {
                const std::string pe = ml + "e" + std::to_string(e) + ".";
                RCHECK(lin(pe + "gate", lc.ff, D));
                RCHECK(lin(pe + "up", lc.ff, D));
                RCHECK(lin(pe + "down", D, lc.ff));
            }
        }
        RCHECK(finalize_layer(m, l));   // bound the staging memory to one layer
    }
    if (c.loop_times > 0) RCHECK(lin("loop.in", D, 2 * D));
    RCHECK(stage_random(m, "embed", c.vocab, D, -1.7f, 1.7f, seed));
    RCHECK(lin("head", c.vocab, D));
    RCHECK(ones("final.norm", D));
    return zl_dekalorn_finalize(m);
}

extern "C" int zl_dekalorn_step(zl_dekalorn_t* m, const int32_t* tokens_host, const int32_t* slots_host,
                               const int32_t* positions_host, int T, const int32_t* want_rows_host, int n_want,
                               float* logits_host, int32_t* next_host) {
    ZL_CHECK_ARG(m && tokens_host && slots_host && positions_host && T > 0 && n_want >= 0);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    ZL_CHECK_ARG(T <= m->tcap && n_want <= T && (n_want == 0 || want_rows_host));
    const auto& c = m->cfg;
    int32_t* hs = m->h_stage;
    int max_len = 0, n_runs = 0, max_run = 1;
    for (int i = 0; i < T; ++i) {
        ZL_CHECK_ARG(tokens_host[i] >= 0 && tokens_host[i] < c.vocab);
        ZL_CHECK_ARG(slots_host[i] >= 0 && slots_host[i] < c.max_batch);
        ZL_CHECK_ARG(positions_host[i] >= 0 && positions_host[i] < c.max_seq);
        // rows of one slot are consecutive and at consecutive positions; a slot appears in one run only
        if (i > 0 && slots_host[i] == slots_host[i - 1]) {
            ZL_CHECK_ARG(positions_host[i] == positions_host[i - 1] + 1);
            hs[6 * T + n_runs - 1] += 1;
            if (hs[6 * T + n_runs - 1] > max_run) max_run = hs[6 * T + n_runs - 1];
        } else {
            hs[5 * T + n_runs] = i;
            hs[6 * T + n_runs] = 1;
            ++n_runs;
        }
        hs[i] = tokens_host[i];
        hs[T + i] = slots_host[i];
        hs[2 * T + i] = positions_host[i];
        if (positions_host[i] + 1 > max_len) max_len = positions_host[i] + 1;
    }
    for (int i = 0; i < n_want; ++i) {
        ZL_CHECK_ARG(want_rows_host[i] >= 0 && want_rows_host[i] < T);
        hs[3 * T + i] = want_rows_host[i];
    }
    cudaStream_t st = m->stream;
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_tokens, hs, (size_t)T * 4, cudaMemcpyHostToDevice, st));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_slots, hs + T, (size_t)T * 4, cudaMemcpyHostToDevice, st));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_pos, hs + 2 * T, (size_t)T * 4, cudaMemcpyHostToDevice, st));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_run0, hs + 5 * T, (size_t)n_runs * 4, cudaMemcpyHostToDevice, st));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_runlen, hs + 6 * T, (size_t)n_runs * 4, cudaMemcpyHostToDevice, st));
    if (n_want) ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_want, hs + 3 * T, (size_t)n_want * 4, cudaMemcpyHostToDevice, st));
    RCHECK(run_step(m, T, n_want, n_runs, max_run, max_len));
    if (n_want && next_host) ZL_CHECK_CUDA(cudaMemcpyAsync(hs + 4 * T, m->d_next, (size_t)n_want * 4, cudaMemcpyDeviceToHost, st));
    if (n_want && logits_host)
        ZL_CHECK_CUDA(cudaMemcpyAsync(logits_host, m->logits, (size_t)n_want * c.vocab * 4, cudaMemcpyDeviceToHost, st));
    ZL_CHECK_CUDA(cudaStreamSynchronize(st));
    if (n_want && next_host)
        for (int i = 0; i < n_want; ++i) next_host[i] = hs[4 * T + i];
    if (max_len > m->cur_max_len) m->cur_max_len = max_len;
    return ZL_OK;
}

extern "C" int zl_dekalorn_set_state(zl_dekalorn_t* m, const int32_t* tokens_host, const int32_t* positions_host, int B) {
    ZL_CHECK_ARG(m && tokens_host && positions_host && B > 0 && B <= m->cfg.max_batch);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));   // the staging buffer is free again
    int32_t* hs = m->h_stage;
    const int T = m->tcap;
    int mx = 0;
    for (int i = 0; i < B; ++i) {
        ZL_CHECK_ARG(tokens_host[i] >= 0 && tokens_host[i] < m->cfg.vocab);
        ZL_CHECK_ARG(positions_host[i] >= 0 && positions_host[i] < m->cfg.max_seq);
        hs[i] = tokens_host[i];
        hs[T + i] = positions_host[i];
        hs[2 * T + i] = 1;
        if (positions_host[i] + 1 > mx) mx = positions_host[i] + 1;
    }
    m->cur_max_len = mx;
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_tokens, hs, (size_t)B * 4, cudaMemcpyHostToDevice, m->stream));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_pos, hs + T, (size_t)B * 4, cudaMemcpyHostToDevice, m->stream));
    ZL_CHECK_CUDA(cudaMemcpyAsync(m->d_runlen, hs + 2 * T, (size_t)B * 4, cudaMemcpyHostToDevice, m->stream));
    k_iota_i32<<<cdiv(B, 256), 256, 0, m->stream>>>(m->d_slots, m->d_want, B);
    k_iota_i32<<<cdiv(B, 256), 256, 0, m->stream>>>(m->d_run0, m->d_want, B);
    ZL_CHECK_LAUNCH();
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

extern "C" int zl_dekalorn_step_device(zl_dekalorn_t* m, int B) {
    ZL_CHECK_ARG(m && B > 0 && B <= m->cfg.max_batch);
    if (m->cur_max_len >= m->cfg.max_seq) return fail(__LINE__, "caches full (max_seq reached)");
    RCHECK(run_step(m, B, B, B, 1, m->cur_max_len));
    k_decode_advance<<<cdiv(B, 64), 64, 0, m->stream>>>(m->d_tokens, m->d_pos, m->d_next, B);
    ZL_CHECK_LAUNCH();
    m->cur_max_len += 1;
    return ZL_OK;
}

extern "C" int zl_dekalorn_sync(zl_dekalorn_t* m) {
    ZL_CHECK_ARG(m);
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

extern "C" zl_stream_t zl_dekalorn_stream(zl_dekalorn_t* m) { return m ? (zl_stream_t)m->stream : nullptr; }

extern "C" int zl_dekalorn_capture_layers(zl_dekalorn_t* m, int on) {
    ZL_CHECK_ARG(m);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    if (on && !m->layer_dump)
        RCHECK(dmalloc((void**)&m->layer_dump, m->runs.size() * m->tcap * m->cfg.width * 4));
    m->capture = on != 0;
    return ZL_OK;
}

extern "C" int zl_dekalorn_read_layers(zl_dekalorn_t* m, float* out_host, int T) {
    ZL_CHECK_ARG(m && out_host && T > 0 && T <= m->tcap);
    if (!m->layer_dump) return fail(__LINE__, "layer capture was not switched on");
    const size_t row = (size_t)m->cfg.width * 4;
    ZL_CHECK_CUDA(cudaMemcpy2DAsync(out_host, (size_t)T * row, m->layer_dump, (size_t)m->tcap * row, (size_t)T * row,
                                    m->runs.size(), cudaMemcpyDeviceToHost, m->stream));
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

extern "C" int zl_dekalorn_read_cache(zl_dekalorn_t* m, int run, int slot, int n_rows, float* a_host, float* b_host) {
    ZL_CHECK_ARG(m && a_host && b_host && run >= 0 && slot >= 0 && slot < m->cfg.max_batch);
    ZL_CHECK_ARG(n_rows > 0 && n_rows <= m->cfg.max_seq && run < (int)m->runs.size());
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    const KRun& U = m->runs[run];
    const KLayer& L = m->layers[U.layer];
    const auto& lc = L.c;
    const bool latent = lc.type == ZL_DEKALORN_LATENT;
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    const size_t kw = (size_t)lc.kv_heads * lc.dim * (lc.type == ZL_DEKALORN_DIFF ? 2 : 1), vw = (size_t)lc.kv_heads * lc.vdim;
    // per output: the cache, elements per cached row, first element, elements wanted
    const SlotCache* caches[2] = {&U.a, latent ? &U.a : &U.b};
    const size_t rows[2] = {latent ? (size_t)L.row_cols : kw, latent ? (size_t)L.row_cols : vw};
    const size_t first[2] = {0, latent ? (size_t)L.rank_cols : 0};
    const size_t wanted[2] = {latent ? (size_t)lc.kv_rank : kw, latent ? (size_t)lc.rot_dim : vw};
    float* outs[2] = {a_host, b_host};
    for (int i = 0; i < 2; ++i) {
        std::vector<unsigned char> tmp((size_t)n_rows * rows[i] * m->esz);
        ZL_CHECK_CUDA(cudaMemcpy(tmp.data(), (const char*)caches[i]->buf + (size_t)slot * caches[i]->slot_bytes, tmp.size(),
                                 cudaMemcpyDeviceToHost));
        for (size_t r = 0; r < (size_t)n_rows; ++r)
            for (size_t j = 0; j < wanted[i]; ++j) {
                const unsigned char* src = tmp.data() + (r * rows[i] + first[i] + j) * m->esz;
                float* dst = outs[i] + r * wanted[i] + j;
                if (m->esz == 4) {
                    memcpy(dst, src, 4);
                } else {
                    const uint32_t u = ((uint32_t)src[0] | (uint32_t)src[1] << 8) << 16;
                    memcpy(dst, &u, 4);
                }
            }
    }
    return ZL_OK;
}

extern "C" int zl_dekalorn_stats(zl_dekalorn_t* m, double* weight_bytes, int* kernels_per_step) {
    ZL_CHECK_ARG(m);
    if (weight_bytes) *weight_bytes = m->weight_bytes;
    if (kernels_per_step) *kernels_per_step = m->kernels_per_step;
    return ZL_OK;
}
