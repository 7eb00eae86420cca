// Host-side driver of the Bezasun model family: weights, slot caches and states, the per-step kernel chain and its CUDA graph.
// Same driver shape as dekalorn_runner.cu (task slots, host (token, slot, position) rows in, logits / greedy picks out), built
// from the shared pieces of runner_common.cuh.
//
// The residual is a set of fp32 streams joined by hyper-connections: ONE kernel (hyper_residual.cu) takes a sublayer's result
// -- for experts the weighted sum of a token's choices and the shared expert -- into all streams and writes the next sublayer's
// normed input.  Everything that is a Linear of the mixer's input is ONE projection with fp32 output.
//   attention:   [W_q; W_k; W_v] -> per-head norms, query temperature, append -> attention with soft-capped scores, distance
//                slope and sink (sink_attn.cu) -> W_o.
//   latent:      [W_dq; W_dkv] -> norm of the query latent -> W_uq -> rotation of the queries' and the shared key part, norm of the
//                latent, append (latent_attn.cu) -> queries absorbed through W_uk per head -> attention over the cached latents
//                in a sliding window -> W_uv per head -> W_o.
//   state space: W_in -> convolution, silu, step sizes -> scan (ssm_scan.cu) -> silu gate and norm in groups -> W_o.
//   experts:     routing on the device (moe_route.cu) -> two grouped GEMMs over the (token, choice) pairs with the silu-gated
//                unit as the first one's epilogue; the shared expert runs beside them on a second stream.
// One step takes T rows in any mix of prompt portions and single decode tokens; every kernel indexes caches by
// (slot, position).
#include "runner_common.cuh"

#include <algorithm>
#include <cmath>
#include <cstdlib>
#include <cstring>

namespace {

using namespace zl;

// how a sublayer hangs on the streams: mix (S, S), out (S) times the residual multiplier, in (S)
struct Hyper {
    float *mix = nullptr, *out = nullptr, *in = nullptr;
};

struct BLayer {
    zl_bezasun_layer_t c{};
    Hyper hc1, hc2;
    float *norm1 = nullptr, *norm2 = nullptr;
    void* w_in = nullptr;                        // fused projection (n_in, width)
    int n_in = 0, k_off = 0, v_off = 0, c_off = 0, x_off = 0, dt_off = 0;   // columns of the projection
    void* o = nullptr;                           // (width, heads * vdim)
    // attention
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *slopes = nullptr;
    // latent
    int rank_cols = 0, row_cols = 0;             // padded latent columns, columns of a cached row
    float *dq_norm = nullptr, *dkv_norm = nullptr;
    void *uq = nullptr, *uk_t = nullptr, *uv = nullptr;   // (heads * (dim + rot_dim), q_rank), (heads, rank_cols, dim), (heads * vdim, rank_cols)
    int rot = -1;                                // index into the model's rotation tables
    // state space
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *d_skip = nullptr, *gn_w = nullptr;
    // feed-forward: rows 2j / 2j+1 of w_gu = gate_j / up_j
    void *w_gu = nullptr, *w_down = nullptr, *router = nullptr, *shared_gu = nullptr, *shared_down = nullptr;
    SlotCache a, b;                              // keys / values; latent rows; state / convolution ring
    bool ready = false;
};

// one (cos, sin) table per distinct (base, size, scaling): filled once per step from the rows' positions
struct RotTable {
    double base = 0, factor = 0, original = 0, fast = 0, slow = 0;
    int dims = 0;
    float mult = 1.f;             // factor on cos and sin
    double* inv_freq = nullptr;   // device (dims / 2)
    float* table = nullptr;       // device (tcap, dims / 2) float pairs
};

}  // namespace

struct zl_bezasun {
    zl_bezasun_config_t cfg{};
    cudaStream_t stream = nullptr, side = nullptr;
    StagedMap staged;
    std::vector<BLayer> layers;
    std::vector<RotTable> rots;
    std::vector<cudaEvent_t> ev_h, ev_ff;        // per layer: feed-forward input ready (main) / shared expert done (side)
    void *embed = nullptr, *head = nullptr;
    float* final_norm = nullptr;                 // (1 + w) * logit_scale
    bool finalized = false;
    int esz = 2;
    int tcap = 0;
    float *x = nullptr, *u = nullptr, *proj = nullptr, *qp = nullptr, *y = nullptr, *ysh = nullptr, *qa = nullptr, *so = nullptr, *xw = nullptr,
          *logits = nullptr, *top_w = nullptr;
    void *h = nullptr, *cq = nullptr, *q = nullptr, *olat = nullptr, *att = nullptr, *act = nullptr, *act_sh = nullptr, *xn = nullptr;
    int32_t *d_tokens = nullptr, *d_slots = nullptr, *d_pos = nullptr, *d_want = nullptr, *d_next = nullptr;
    int32_t *d_run0 = nullptr, *d_runlen = nullptr, *top_e = nullptr, *grp_off = nullptr, *list_token = nullptr,
            *list_pair = nullptr;
    int32_t* h_stage = nullptr;   // pinned: tokens | slots | pos | want | next | run0 | runlen
    void *attn_ws = nullptr, *ssm_ws = nullptr, *argmax_ws = nullptr;
    size_t attn_ws_bytes = 0, ssm_ws_bytes = 0;
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

int rot_index(zl_bezasun* m, const zl_bezasun_layer_t& c) {
    for (size_t i = 0; i < m->rots.size(); ++i) {
        const RotTable& r = m->rots[i];
        if (r.base == c.rot_base && r.dims == c.rot_dim && r.factor == c.rot_factor && r.original == c.rot_original && r.fast == c.rot_fast &&
            r.slow == c.rot_slow)
            return (int)i;
    }
    RotTable r;
    r.base = c.rot_base, r.dims = c.rot_dim;
    r.factor = c.rot_factor, r.original = c.rot_original, r.fast = c.rot_fast, r.slow = c.rot_slow;
    m->rots.push_back(r);
    return (int)m->rots.size() - 1;
}

int ssm_channels(const zl_bezasun_layer_t& c) { return c.heads * c.vdim + 2 * c.groups * c.state; }

int take_hyper(zl_bezasun* m, const std::string& p, Hyper& hc) {
    const int S = m->cfg.streams;
    RCHECK(take_f32(m, p + "in", 1, S, &hc.in));
    RCHECK(take_f32(m, p + "mix", S, S, &hc.mix));
    std::vector<double> out;
    RCHECK(take_host(m, p + "out", 1, S, out));
    for (double& v : out) v *= (double)m->cfg.residual_mult;
    return upload_f32(out, &hc.out);
}

int take_gated(zl_bezasun* m, const std::string& p, int F, void* gu, size_t gu_off, void* down, size_t down_off) {
    const int D = m->cfg.width;
    RCHECK(put_interleaved(m, p + "gate", p + "up", F, D, gu, gu_off, false));
    return put_weight(m, p + "down", D, F, down, down_off);
}

int finalize_ff(zl_bezasun* m, int l) {
    BLayer& L = m->layers[l];
    const auto& lc = L.c;
    const int D = m->cfg.width, F = lc.ff, E = lc.experts;
    const std::string p = "l" + std::to_string(l) + ".";
    RCHECK(take_norm_plus_one(m, p + "norm2", D, &L.norm2));
    RCHECK(take_hyper(m, p + "hc2.", L.hc2));
    RCHECK(take_weight(m, p + "mlp.router", E, D, &L.router));
    RCHECK(dmalloc(&L.w_gu, (size_t)E * 2 * F * D * m->esz));
    RCHECK(dmalloc(&L.w_down, (size_t)E * D * F * m->esz));
    for (int e = 0; e < E; ++e)
        RCHECK(take_gated(m, p + "mlp.e" + std::to_string(e) + ".", F, L.w_gu, (size_t)e * 2 * F * D, L.w_down, (size_t)e * D * F));
    if (lc.shared_ff > 0) {
        RCHECK(dmalloc(&L.shared_gu, (size_t)2 * lc.shared_ff * D * m->esz));
        RCHECK(dmalloc(&L.shared_down, (size_t)D * lc.shared_ff * m->esz));
        RCHECK(take_gated(m, p + "mlp.shared.", lc.shared_ff, L.shared_gu, 0, L.shared_down, 0));
    }
    return ZL_OK;
}

int finalize_layer(zl_bezasun* m, int l) {
    BLayer& L = m->layers[l];
    const auto& lc = L.c;
    const std::string p = "l" + std::to_string(l) + ".", mx = p + "mix.";
    const int D = m->cfg.width, H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
    const bool f32 = m->cfg.dtype == ZL_F32;
    RCHECK(take_norm_plus_one(m, p + "norm1", D, &L.norm1));
    RCHECK(take_hyper(m, p + "hc1.", L.hc1));
    // (name, rows) of the fused projection's segments in order
    std::vector<std::pair<std::string, int>> seg;
    if (lc.type == ZL_BEZASUN_ATTENTION) {
        seg = {{"q", H * d}, {"k", G * d}, {"v", G * vd}};
        L.k_off = seg[0].second;
        L.v_off = L.k_off + seg[1].second;
    } else if (lc.type == ZL_BEZASUN_LATENT) {
        seg = {{"dq", lc.q_rank}, {"dkv", lc.kv_rank + lc.rot_dim}};
        L.c_off = seg[0].second;
    } else {
        seg = {{"in", H * vd + ssm_channels(lc) + H}};   // gate | x | B | C | step sizes
        L.x_off = H * vd;
        L.dt_off = L.x_off + ssm_channels(lc);
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
    if (lc.type == ZL_BEZASUN_ATTENTION) {
        RCHECK(take_f32(m, mx + "q.norm", 1, d, &L.q_norm));
        RCHECK(take_f32(m, mx + "k.norm", 1, d, &L.k_norm));
        RCHECK(take_f32(m, mx + "sink", 1, H, &L.sink));
        std::vector<double> slopes(H);
        for (int h = 0; h < H; ++h) slopes[h] = exp2(-8.0 * (h + 1) / H);
        RCHECK(upload_f32(slopes, &L.slopes));
    } else if (lc.type == ZL_BEZASUN_LATENT) {
        // 16-bit runs pad the latent to the tensor-core kernel's column step and the rotated part to its contraction step (zero
        // weights and never-written cache columns)
        L.rank_cols = f32 ? lc.kv_rank : round_up(lc.kv_rank, lc.kv_rank <= 512 ? 64 : 8);
        L.row_cols = L.rank_cols + (f32 ? lc.rot_dim : round_up(lc.rot_dim, 16));
        RCHECK(take_f32(m, mx + "dq.norm", 1, lc.q_rank, &L.dq_norm));
        RCHECK(take_f32(m, mx + "dkv.norm", 1, lc.kv_rank, &L.dkv_norm));
        RCHECK(take_weight(m, mx + "uq", H * (d + lc.rot_dim), lc.q_rank, &L.uq));
        RCHECK(take_latent(m, mx + "uk", true, H, d, lc.kv_rank, L.rank_cols, &L.uk_t));
        RCHECK(take_latent(m, mx + "uv", false, H, vd, lc.kv_rank, L.rank_cols, &L.uv));
        if (lc.rot_dim > 0) L.rot = rot_index(m, lc);
    } else {
        const int C = ssm_channels(lc);
        std::vector<double> w, wt((size_t)C * lc.conv);
        RCHECK(take_host(m, mx + "conv", C, lc.conv, w));
        for (int c = 0; c < C; ++c)
            for (int j = 0; j < lc.conv; ++j) wt[(size_t)j * C + c] = w[(size_t)c * lc.conv + j];
        RCHECK(upload_f32(wt, &L.conv_w));
        RCHECK(take_f32(m, mx + "conv.b", 1, C, &L.conv_b));
        RCHECK(take_f32(m, mx + "dt_bias", 1, H, &L.dt_bias));
        RCHECK(take_f32(m, mx + "A_log", 1, H, &L.a_log));
        RCHECK(take_f32(m, mx + "D", 1, H, &L.d_skip));
        RCHECK(take_f32(m, mx + "norm", 1, H * vd, &L.gn_w));
    }
    RCHECK(take_weight(m, mx + "o", D, H * vd, &L.o));
    if (lc.ff_kind != ZL_FF_NONE) RCHECK(finalize_ff(m, l));
    L.ready = true;
    return ZL_OK;
}

int len_bucket(const zl_bezasun* m, int max_len) {
    int b = 256;
    while (b < max_len) b <<= 1;
    return b < m->cfg.max_seq ? b : (m->cfg.max_seq > 256 ? m->cfg.max_seq : 256);
}

int attn_splits(const BLayer& L, int T, int max_len) {
    const auto& lc = L.c;
    if (lc.type == ZL_BEZASUN_LATENT)
        // (a window is full, a length bucket is not: splits half as long)
        return zl_latent_attention_splits(T, lc.heads, L.rank_cols, lc.window > 0 && lc.window < max_len / 2 ? 2 * lc.window : max_len);
    return lc.type == ZL_BEZASUN_ATTENTION ? zl_sink_attention_splits(T, lc.heads, lc.kv_heads, max_len) : 1;
}

int alloc_runtime(zl_bezasun* m) {
    const auto& c = m->cfg;
    const int D = c.width, T = m->tcap, B = c.max_batch, len = len_bucket(m, c.max_seq);
    size_t n_in = 1, n_q = 1, qr = 1, hd = 1, hv = 1, hr = 1, ha = 1, so = 1, ffw = 1, shw = 1, top = 1, experts = 1;
    for (auto& L : m->layers) {
        const auto& lc = L.c;
        const size_t H = lc.heads;
        n_in = std::max(n_in, (size_t)L.n_in);
        hv = std::max(hv, H * lc.vdim);
        if (lc.type == ZL_BEZASUN_LATENT) {
            RCHECK(zl_latent_attention_prepare_ex(lc.heads, L.rank_cols, L.row_cols, c.dtype));
            qr = std::max(qr, (size_t)lc.q_rank);
            n_q = std::max(n_q, H * (lc.dim + lc.rot_dim));
            hd = std::max(hd, H * lc.dim);
            hr = std::max(hr, H * L.rank_cols);
            ha = std::max(ha, H * L.row_cols);
            RCHECK(L.a.create(B, (size_t)c.max_seq * L.row_cols * m->esz, m->stream));
        } else if (lc.type == ZL_BEZASUN_ATTENTION) {
            hd = std::max(hd, H * lc.dim);
            RCHECK(L.a.create(B, (size_t)c.max_seq * lc.kv_heads * lc.dim * m->esz, m->stream));
            RCHECK(L.b.create(B, (size_t)c.max_seq * lc.kv_heads * lc.vdim * m->esz, m->stream));
        } else {
            RCHECK(zl_ssm_prepare(lc.vdim, lc.state));
            so = std::max(so, H * lc.vdim);
            m->ssm_ws_bytes = std::max(m->ssm_ws_bytes, zl_ssm_workspace_bytes(T, lc.heads, lc.vdim, lc.state, lc.groups));
            RCHECK(L.a.create(B, H * lc.vdim * lc.state * 4, m->stream));
            RCHECK(L.b.create(B, (size_t)std::max(lc.conv - 1, 1) * ssm_channels(lc) * 4, m->stream));
        }
        if (lc.type != ZL_BEZASUN_SSM)   // the split count falls as the rows grow: size for the worst product
            for (int b = 1; b <= T; ++b) {
                const int s = attn_splits(L, b, len);
                m->attn_ws_bytes = std::max(m->attn_ws_bytes, lc.type == ZL_BEZASUN_LATENT
                                                                  ? zl_latent_attention_workspace_bytes(b, lc.heads, L.rank_cols, s)
                                                                  : zl_sink_attention_workspace_bytes(b, lc.heads, lc.vdim, s));
            }
        if (lc.ff_kind == ZL_FF_MOE) {
            ffw = std::max(ffw, (size_t)lc.top * lc.ff);
            shw = std::max(shw, (size_t)lc.shared_ff);
            top = std::max(top, (size_t)lc.top);
            experts = std::max(experts, (size_t)lc.experts);
        }
    }
    for (auto& r : m->rots) {
        const int half = r.dims / 2;
        std::vector<double> f(half);
        RCHECK(zl_rope_inv_freq_yarn(r.base, r.dims, r.factor, r.original, r.fast, r.slow, f.data(), &r.mult));
        RCHECK(dmalloc((void**)&r.inv_freq, (size_t)half * 8));
        ZL_CHECK_CUDA(cudaMemcpy(r.inv_freq, f.data(), (size_t)half * 8, cudaMemcpyHostToDevice));
        RCHECK(dmalloc((void**)&r.table, (size_t)T * half * 8));
    }
    const size_t e = m->esz;
    RCHECK(dmalloc((void**)&m->x, (size_t)T * c.streams * D * 4));
    RCHECK(dmalloc((void**)&m->u, (size_t)T * D * 4));
    RCHECK(dmalloc((void**)&m->proj, (size_t)T * n_in * 4));
    RCHECK(dmalloc((void**)&m->qp, (size_t)T * n_q * 4));
    RCHECK(dmalloc((void**)&m->y, (size_t)T * top * D * 4));
    RCHECK(dmalloc((void**)&m->ysh, (size_t)T * D * 4));
    RCHECK(dmalloc((void**)&m->qa, (size_t)T * ha * 4));
    ZL_CHECK_CUDA(cudaMemsetAsync(m->qa, 0, (size_t)T * ha * 4, m->stream));   // padding columns are never written: keep them finite
    RCHECK(dmalloc((void**)&m->so, (size_t)T * so * 4));
    RCHECK(dmalloc((void**)&m->xw, (size_t)T * D * 4));
    RCHECK(dmalloc((void**)&m->logits, (size_t)T * c.vocab * 4));
    RCHECK(dmalloc((void**)&m->top_w, (size_t)T * top * 4));
    RCHECK(dmalloc(&m->h, (size_t)T * D * e));
    RCHECK(dmalloc(&m->cq, (size_t)T * qr * e));
    RCHECK(dmalloc(&m->q, (size_t)T * hd * e));
    RCHECK(dmalloc(&m->olat, (size_t)T * hr * e));
    RCHECK(dmalloc(&m->att, (size_t)T * hv * e));
    RCHECK(dmalloc(&m->act, (size_t)T * ffw * e));
    RCHECK(dmalloc(&m->act_sh, (size_t)T * shw * e));
    RCHECK(dmalloc(&m->xn, (size_t)T * D * e));
    for (int32_t** p : {&m->d_tokens, &m->d_slots, &m->d_pos, &m->d_want, &m->d_next, &m->d_run0, &m->d_runlen})
        RCHECK(dmalloc((void**)p, (size_t)T * 4));
    RCHECK(dmalloc((void**)&m->top_e, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->list_token, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->list_pair, (size_t)T * top * 4));
    RCHECK(dmalloc((void**)&m->grp_off, (experts + 1) * 4));
    RCHECK(dmalloc(&m->attn_ws, m->attn_ws_bytes));
    RCHECK(dmalloc(&m->ssm_ws, m->ssm_ws_bytes));
    RCHECK(dmalloc(&m->argmax_ws, zl_argmax_workspace_bytes(T)));
    ZL_CHECK_CUDA(cudaMallocHost((void**)&m->h_stage, sizeof(int32_t) * 7 * (size_t)T));
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

// Which kernels of a step of at most 8 rows are launched with a programmatic dependency: 1 skinny Linears, 2 other GEMMs,
// 4 row kernels, 8 attention, 16 the scan, 32 the tail.  Larger steps use none.  ZL_BEZASUN_PDL_MASK overrides the default.
constexpr int kDefaultPdlMask = 1;
int pdl_mask() {
    static int v = -1;
    if (v < 0) {
        const char* e = getenv("ZL_BEZASUN_PDL_MASK");
        v = e ? atoi(e) : kDefaultPdlMask;
    }
    return v;
}
int pdl_for(const zl_bezasun* m, int bit, int T) { return (m->cfg.use_pdl && T <= 8 && (pdl_mask() & bit)) ? 1 : 0; }

// y (M, N) = x (M, K) @ w (N, K)^T; on the side stream without programmatic dependencies (its predecessor is an event)
int linear(zl_bezasun* m, const void* x, int K, const void* w, int N, void* y, int M, int out_dtype, bool side = false) {
    const auto& c = m->cfg;
    cudaStream_t st = side ? m->side : m->stream;
    if (c.dtype != ZL_F32 && M <= 32 && K % 32 == 0 && N >= 64 && (reinterpret_cast<uintptr_t>(x) & 15) == 0 &&
        (reinterpret_cast<uintptr_t>(w) & 15) == 0)
        return zl_dense_gemm_skinny_act(x, K, w, nullptr, y, M, N, K, c.dtype, out_dtype, 0, side ? 0 : pdl_for(m, 1, M), st);
    return zl_gemm_nt_bias(x, K, w, K, nullptr, y, N, M, N, K, c.dtype, out_dtype, ZL_GEMM_EPI_NONE, side ? 0 : pdl_for(m, 2, M), st);
}

int enqueue_mixer(zl_bezasun* m, BLayer& L, int T, int n_runs, int max_run, int max_len) {
    const auto& c = m->cfg;
    const auto& lc = L.c;
    const int D = c.width, dt = c.dtype, H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
    const int pg = pdl_for(m, 2, T), pr = pdl_for(m, 4, T), pa = pdl_for(m, 8, T);
    cudaStream_t st = m->stream;
    const int splits = attn_splits(L, T, max_len);
    RCHECK(linear(m, m->h, D, L.w_in, L.n_in, m->proj, T, ZL_F32));
    if (lc.type == ZL_BEZASUN_ATTENTION) {
        RCHECK(zl_qkv_headnorm_append_ex(m->proj, L.n_in, 0, L.k_off, L.v_off, H, G, d, vd, L.q_norm, L.k_norm, 0, lc.temp_coef,
                                         lc.temp_every, nullptr, 0, 1.f, c.eps, m->q, L.a.addrs, L.b.addrs, m->d_slots, m->d_pos, T,
                                         dt, pr, st));
        RCHECK(zl_biased_sink_attention(m->q, L.a.addrs, L.b.addrs, m->d_slots, m->d_pos, L.sink, 0, lc.scale, lc.softcap, L.slopes, 0,
                                        m->att, T, H, G, d, vd, splits, m->attn_ws, m->attn_ws_bytes, m->d_run0, m->d_runlen, n_runs,
                                        max_run, dt, pa, st));
    } else if (lc.type == ZL_BEZASUN_LATENT) {
        const int RC = L.rank_cols, RS = L.row_cols, nq = H * (d + lc.rot_dim);
        const float* tab = L.rot >= 0 ? m->rots[L.rot].table : nullptr;
        RCHECK(zl_group_rmsnorm(m->proj, L.n_in, L.dq_norm, m->cq, lc.q_rank, T, lc.q_rank, 1, c.eps, dt, pr, st));
        RCHECK(linear(m, m->cq, lc.q_rank, L.uq, nq, m->qp, T, ZL_F32));
        RCHECK(zl_latent_rope_append_split(m->qp, nq, H, d, lc.rot_dim, tab, m->q, m->qa, m->proj, L.n_in, L.c_off, lc.kv_rank,
                                           L.dkv_norm, RC, RS, L.a.addrs, m->d_slots, m->d_pos, T, c.eps, dt, pr, st));
        RCHECK(zl_gemm_nt(m->q, (long long)H * d, d, L.uk_t, d, (long long)RC * d, m->qa, (long long)H * RS, RS, T, RC, d, H, dt, ZL_F32,
                          ZL_GEMM_EPI_NONE, nullptr, 0, 0, pg, st));
        RCHECK(zl_latent_window_attention(m->qa, L.a.addrs, m->d_slots, m->d_pos, nullptr, nullptr, 0, lc.scale, lc.window, m->olat, T, H,
                                          RC, RS, splits, m->attn_ws, m->attn_ws_bytes, m->d_run0, m->d_runlen, n_runs, max_run, dt,
                                          pa, st));
        RCHECK(zl_gemm_nt(m->olat, (long long)H * RC, RC, L.uv, RC, (long long)vd * RC, m->att, (long long)H * vd, vd, T, vd, RC, H, dt,
                          dt, ZL_GEMM_EPI_NONE, nullptr, 0, 0, pg, st));
    } else {
        RCHECK(zl_ssm_scan(m->proj, L.n_in, L.x_off, L.dt_off, L.conv_w, L.conv_b, lc.conv, L.dt_bias, L.a_log, L.d_skip, L.b.addrs,
                           m->d_run0, m->d_runlen, n_runs, m->d_slots, m->d_pos, L.a.addrs, m->so, (long long)H * vd, H, vd, lc.state,
                           lc.groups, T, m->ssm_ws, m->ssm_ws_bytes, pdl_for(m, 16, T), st));
        RCHECK(zl_silu_gate_group_rmsnorm(m->so, (long long)H * vd, m->proj, L.n_in, L.gn_w, m->att, (long long)H * vd, T, H * vd,
                                          lc.norm_groups, c.eps, dt, pr, st));
    }
    return linear(m, m->att, H * vd, L.o, D, m->y, T, ZL_F32);
}

int enqueue_step(zl_bezasun* m, int T, int n_want, int n_runs, int max_run, int max_len) {
    const auto& c = m->cfg;
    const int D = c.width, dt = c.dtype, S = c.streams;
    cudaStream_t st = m->stream;
    const int pg = pdl_for(m, 2, T), pr = pdl_for(m, 4, T), pt = pdl_for(m, 32, T);
    RCHECK(zl_hyper_embed(m->d_tokens, m->embed, c.vocab, c.embed_scale, m->x, S, m->layers[0].hc1.in, m->layers[0].norm1, m->h, nullptr,
                          dt, T, D, c.eps, 0, st));
    for (auto& r : m->rots)
        RCHECK(zl_rope_table_scaled(m->d_pos, T, r.inv_freq, r.dims / 2, (double)r.mult, r.table, pr, st));
    for (size_t l = 0; l < m->layers.size(); ++l) {
        BLayer& L = m->layers[l];
        const auto& lc = L.c;
        const bool ff = lc.ff_kind != ZL_FF_NONE;
        RCHECK(enqueue_mixer(m, L, T, n_runs, max_run, max_len));
        // a layer's last update of the streams reads the next layer's input; the model's last one reads the sum of the streams
        const BLayer* next = l + 1 < m->layers.size() ? &m->layers[l + 1] : nullptr;
        const float *next_in = next ? next->hc1.in : nullptr, *next_w = next ? next->norm1 : nullptr;
        float* u = next ? nullptr : m->u;
        RCHECK(zl_hyper_update(m->x, S, m->y, D, nullptr, 1, nullptr, 0, L.hc1.mix, L.hc1.out, ff ? L.hc2.in : next_in,
                               ff ? L.norm2 : next_w, m->h, ff ? nullptr : u, dt, T, D, c.eps, pr, st));
        if (ff) {
            const int E = lc.experts, F = lc.ff, F2 = lc.shared_ff;
            if (F2 > 0) {
                ZL_CHECK_CUDA(cudaEventRecord(m->ev_h[l], st));
                ZL_CHECK_CUDA(cudaStreamWaitEvent(m->side, m->ev_h[l], 0));
                RCHECK(zl_gemm_nt_glu_clamp(m->h, D, L.shared_gu, D, nullptr, m->act_sh, F2, T, 2 * F2, D, dt, dt, INFINITY, 1.f, 0.f, 0,
                                            m->side));
                RCHECK(linear(m, m->act_sh, F2, L.shared_down, D, m->ysh, T, ZL_F32, true));
                ZL_CHECK_CUDA(cudaEventRecord(m->ev_ff[l], m->side));
            }
            RCHECK(zl_moe_route_ex(m->h, D, L.router, dt, nullptr, m->top_e, m->top_w, m->grp_off, m->list_token, m->list_pair, T, D, E,
                                   lc.top, 1, 1, ZL_MOE_GROUP_MAX, ZL_MOE_SCORE_SOFTMAX, 0, 0.f, 1.f, pr, st));
            // g sigmoid(g) u: the clamped unit without its clamp
            RCHECK(zl_gemm_nt_grouped(m->h, D, m->list_token, L.w_gu, D, (long long)2 * F * D, m->act, F, nullptr, m->grp_off, E, T, 2 * F,
                                      D, dt, dt, ZL_GEMM_EPI_GLU_CLAMP, INFINITY, 1.f, 0.f, pg, st));
            RCHECK(zl_gemm_nt_grouped(m->act, F, nullptr, L.w_down, F, (long long)D * F, m->y, D, m->list_pair, m->grp_off, E, T, D, F,
                                      dt, ZL_F32, ZL_GEMM_EPI_NONE, 0.f, 1.f, 0.f, pg, st));
            if (F2 > 0) ZL_CHECK_CUDA(cudaStreamWaitEvent(st, m->ev_ff[l], 0));
            RCHECK(zl_hyper_update(m->x, S, m->y, D, m->top_w, lc.top, F2 > 0 ? m->ysh : nullptr, D, L.hc2.mix, L.hc2.out, next_in, next_w,
                                   m->h, u, dt, T, D, c.eps, F2 > 0 ? 0 : pr, st));
        }
        if (m->capture && m->layer_dump)
            RCHECK(zl_hyper_update(m->x, S, nullptr, 0, nullptr, 0, nullptr, 0, nullptr, nullptr, nullptr, nullptr, nullptr,
                                   m->layer_dump + l * m->tcap * D, dt, T, D, c.eps, 0, st));
    }
    if (n_want > 0) {
        ZL_CHECK_CUDA(launch(k_gather_rows_f32, dim3(n_want), dim3(128), 0, st, false, (const float*)m->u,
                             (const int32_t*)m->d_want, m->xw, D));
        RCHECK(zl_group_rmsnorm(m->xw, D, m->final_norm, m->xn, D, n_want, D, 1, c.eps, dt, pt, st));
        RCHECK(linear(m, m->xn, D, m->head, c.vocab, m->logits, n_want, ZL_F32));
        RCHECK(zl_argmax(m->logits, m->d_next, n_want, c.vocab, m->argmax_ws, zl_argmax_workspace_bytes(n_want), pt, st));
    }
    return ZL_OK;
}

// decode-sized steps replay a CUDA graph per (rows, wanted rows, runs, length bucket); prompt portions are enqueued directly
// (max_run: the longest run; a captured step is sized for the longest run its row count allows)
int run_step(zl_bezasun* m, int T, int n_want, int n_runs, int max_run, int max_len) {
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

extern "C" int zl_bezasun_create(const zl_bezasun_config_t* cfg, const zl_bezasun_layer_t* layers, zl_bezasun_t** out) {
    ZL_CHECK_ARG(cfg && layers && out);
    ZL_CHECK_ARG(cfg->num_layers > 0 && cfg->width > 0 && cfg->vocab > 0 && cfg->max_batch > 0 && cfg->max_seq > 0);
    ZL_CHECK_ARG(cfg->eps >= 0.f && cfg->streams >= 1 && cfg->streams <= 16);
    ZL_CHECK_SUPPORTED(cfg->dtype == ZL_BF16 || cfg->dtype == ZL_F32);
    ZL_CHECK_ARG(cfg->max_step_tokens >= 0 && cfg->max_step_tokens <= 65535);
    for (int l = 0; l < cfg->num_layers; ++l) {
        const auto& lc = layers[l];
        ZL_CHECK_ARG(lc.heads > 0 && lc.vdim > 0);
        if (lc.type == ZL_BEZASUN_ATTENTION) {
            ZL_CHECK_ARG(lc.dim > 0 && lc.kv_heads > 0 && lc.heads % lc.kv_heads == 0 && lc.softcap >= 0.f);
            ZL_CHECK_ARG(lc.temp_coef == 0.f || lc.temp_every > 0);
        } else if (lc.type == ZL_BEZASUN_LATENT) {
            ZL_CHECK_ARG(lc.dim > 0 && lc.q_rank > 0 && lc.kv_rank > 0 && lc.rot_dim >= 0 && lc.rot_dim % 2 == 0 && lc.window >= 0);
            ZL_CHECK_ARG(lc.rot_dim == 0 || lc.rot_base > 1.0);
        } else {
            ZL_CHECK_ARG(lc.type == ZL_BEZASUN_SSM && lc.state > 0 && lc.groups > 0 && lc.heads % lc.groups == 0 && lc.conv >= 1);
            ZL_CHECK_ARG(lc.norm_groups > 0 && lc.heads * lc.vdim % lc.norm_groups == 0);
        }
        ZL_CHECK_ARG(lc.ff_kind == ZL_FF_NONE || lc.ff_kind == ZL_FF_MOE);
        if (lc.ff_kind == ZL_FF_MOE)
            ZL_CHECK_ARG(lc.ff > 0 && lc.experts > 0 && lc.top > 0 && lc.top <= lc.experts && lc.shared_ff >= 0);
    }
    zl_bezasun* m = new zl_bezasun();
    m->cfg = *cfg;
    m->esz = cfg->dtype == ZL_F32 ? 4 : 2;
    m->tcap = cfg->max_step_tokens > cfg->max_batch ? cfg->max_step_tokens : cfg->max_batch;
    m->layers.resize(cfg->num_layers);
    m->ev_h.resize(cfg->num_layers);
    m->ev_ff.resize(cfg->num_layers);
    for (int l = 0; l < cfg->num_layers; ++l) m->layers[l].c = layers[l];
    bool ok = cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking) == cudaSuccess &&
              cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking) == cudaSuccess;
    for (auto* evs : {&m->ev_h, &m->ev_ff})
        for (auto& e : *evs) ok = ok && cudaEventCreateWithFlags(&e, cudaEventDisableTiming) == cudaSuccess;
    if (!ok) {
        zl_bezasun_destroy(m);
        zl_set_last_error(__FILE__, __LINE__, "creating streams failed (no CUDA device? there is no CPU fallback)");
        return ZL_ERR_CUDA;
    }
    *out = m;
    return ZL_OK;
}

extern "C" void zl_bezasun_destroy(zl_bezasun_t* m) {
    if (!m) return;
    if (m->stream) cudaStreamSynchronize(m->stream);
    if (m->side) cudaStreamSynchronize(m->side);
    for (auto& g : m->graphs) cudaGraphExecDestroy(g.second);
    for (auto& s : m->staged) cudaFree(s.second.ptr);
    for (auto& L : m->layers) {
        for (void* p : {(void*)L.hc1.mix, (void*)L.hc1.out, (void*)L.hc1.in, (void*)L.hc2.mix, (void*)L.hc2.out, (void*)L.hc2.in,
                        (void*)L.norm1, (void*)L.norm2, L.w_in, L.o, (void*)L.q_norm, (void*)L.k_norm, (void*)L.sink, (void*)L.slopes,
                        (void*)L.dq_norm, (void*)L.dkv_norm, L.uq, L.uk_t, L.uv, (void*)L.conv_w, (void*)L.conv_b, (void*)L.dt_bias,
                        (void*)L.a_log, (void*)L.d_skip, (void*)L.gn_w, L.w_gu, L.w_down, L.router, L.shared_gu, L.shared_down})
            if (p) cudaFree(p);
        L.a.destroy();
        L.b.destroy();
    }
    for (auto& r : m->rots)
        for (void* p : {(void*)r.inv_freq, (void*)r.table})
            if (p) cudaFree(p);
    for (void* p : {m->embed, m->head, (void*)m->final_norm, (void*)m->x, (void*)m->u, (void*)m->proj, (void*)m->qp, (void*)m->y,
                    (void*)m->ysh, (void*)m->qa, (void*)m->so, (void*)m->xw, (void*)m->logits, (void*)m->top_w, m->h, m->cq, m->q, m->olat,
                    m->att, m->act, m->act_sh, m->xn, (void*)m->d_tokens, (void*)m->d_slots, (void*)m->d_pos, (void*)m->d_want,
                    (void*)m->d_next, (void*)m->d_run0, (void*)m->d_runlen, (void*)m->top_e, (void*)m->grp_off, (void*)m->list_token,
                    (void*)m->list_pair, m->attn_ws, m->ssm_ws, m->argmax_ws, (void*)m->layer_dump})
        if (p) cudaFree(p);
    if (m->h_stage) cudaFreeHost(m->h_stage);
    for (auto* evs : {&m->ev_h, &m->ev_ff})
        for (auto& e : *evs)
            if (e) cudaEventDestroy(e);
    if (m->side) cudaStreamDestroy(m->side);
    if (m->stream) cudaStreamDestroy(m->stream);
    delete m;
}

extern "C" int zl_bezasun_load_tensor(zl_bezasun_t* m, const char* name, const void* data_host, int rows, int cols,
                                       int elem_bytes) {
    ZL_CHECK_ARG(m && name && data_host && rows > 0 && cols > 0 && (elem_bytes == 2 || elem_bytes == 4));
    if (m->finalized) return fail(__LINE__, "model already finalized");
    return staged_load(m->staged, name, data_host, rows, cols, elem_bytes, m->stream);
}

extern "C" int zl_bezasun_finalize(zl_bezasun_t* m) {
    ZL_CHECK_ARG(m);
    if (m->finalized) return ZL_OK;
    const int D = m->cfg.width;
    for (int l = 0; l < m->cfg.num_layers; ++l)
        if (!m->layers[l].ready) RCHECK(finalize_layer(m, l));
    RCHECK(take_weight(m, "embed", m->cfg.vocab, D, &m->embed));
    m->weight_bytes -= (double)m->cfg.vocab * D * m->esz;   // gathered, not streamed
    RCHECK(take_weight(m, "head", m->cfg.vocab, D, &m->head));
    // the logits' constant factor rides on the last norm's multipliers, in fp32
    std::vector<double> w;
    RCHECK(take_host(m, "final.norm", 1, D, w));
    for (double& v : w) v = (1.0 + v) * (double)m->cfg.logit_scale;
    RCHECK(upload_f32(w, &m->final_norm));
    RCHECK(alloc_runtime(m));
    m->finalized = true;
    return ZL_OK;
}

extern "C" int zl_bezasun_init_synthetic(zl_bezasun_t* m, uint64_t seed) {
    ZL_CHECK_ARG(m);
    if (m->finalized) return fail(__LINE__, "model already finalized");
    const auto& c = m->cfg;
    const int D = c.width, S = c.streams;
    auto lin = [&](const std::string& name, int n, int k) {
        const float a = sqrtf(3.0f / (float)k);   // unit-variance outputs for unit-variance inputs
        return stage_random(m, name, n, k, -a, a, seed);
    };
    auto near = [&](const std::string& name, int n, float lo, float hi) { return stage_random(m, name, 1, n, lo, hi, seed); };
    auto hyper = [&](const std::string& p) {
        RCHECK(near(p + "in", S, 0.9f / S, 1.1f / S));
        RCHECK(near(p + "out", S, 0.5f, 1.5f));
        return stage_random(m, p + "mix", S, S, 0.8f / S, 1.2f / S, seed);
    };
    for (int l = 0; l < c.num_layers; ++l) {
        const auto& lc = m->layers[l].c;
        const std::string p = "l" + std::to_string(l) + ".", mx = p + "mix.", ml = p + "mlp.";
        const int H = lc.heads, G = lc.kv_heads, d = lc.dim, vd = lc.vdim;
        RCHECK(near(p + "norm1", D, -0.1f, 0.1f));
        RCHECK(hyper(p + "hc1."));
        if (lc.type == ZL_BEZASUN_ATTENTION) {
            RCHECK(lin(mx + "q", H * d, D));
            RCHECK(lin(mx + "k", G * d, D));
            RCHECK(lin(mx + "v", G * vd, D));
            RCHECK(near(mx + "q.norm", d, 0.9f, 1.1f));
            RCHECK(near(mx + "k.norm", d, 0.9f, 1.1f));
            RCHECK(near(mx + "sink", H, -1.f, 1.f));
        } else if (lc.type == ZL_BEZASUN_LATENT) {
            RCHECK(lin(mx + "dq", lc.q_rank, D));
            RCHECK(near(mx + "dq.norm", lc.q_rank, 0.9f, 1.1f));
            RCHECK(lin(mx + "uq", H * (d + lc.rot_dim), lc.q_rank));
            RCHECK(lin(mx + "dkv", lc.kv_rank + lc.rot_dim, D));
            RCHECK(near(mx + "dkv.norm", lc.kv_rank, 0.9f, 1.1f));
            RCHECK(lin(mx + "uk", H * d, lc.kv_rank));
            RCHECK(lin(mx + "uv", H * vd, lc.kv_rank));
        } else {
            const int C = ssm_channels(lc);
            RCHECK(lin(mx + "in", H * vd + C + H, D));
            RCHECK(lin(mx + "conv", C, lc.conv));
            RCHECK(near(mx + "conv.b", C, -0.1f, 0.1f));
            RCHECK(near(mx + "dt_bias", H, -4.f, -1.f));
            RCHECK(near(mx + "A_log", H, 0.f, 2.f));
            RCHECK(near(mx + "D", H, 0.5f, 1.5f));
            RCHECK(near(mx + "norm", H * vd, 0.9f, 1.1f));
        }
        RCHECK(lin(mx + "o", D, H * vd));
        if (lc.ff_kind == ZL_FF_MOE) {
            RCHECK(near(p + "norm2", D, -0.1f, 0.1f));
            RCHECK(hyper(p + "hc2."));
            RCHECK(lin(ml + "router", lc.experts, D));
            for (int e = 0; e <= lc.experts; ++e) {
                const int F = e < lc.experts ? lc.ff : lc.shared_ff;
                const std::string pe = ml + (e < lc.experts ? "e" + std::to_string(e) : std::string("shared")) + ".";
                if (F == 0) continue;
                RCHECK(lin(pe + "gate", F, D));
                RCHECK(lin(pe + "up", F, D));
                RCHECK(lin(pe + "down", D, F));
            }
        }
        RCHECK(finalize_layer(m, l));   // bound the staging memory to one layer
    }
    RCHECK(stage_random(m, "embed", c.vocab, D, -1.7f, 1.7f, seed));
    RCHECK(lin("head", c.vocab, D));
    RCHECK(near("final.norm", D, -0.1f, 0.1f));
    return zl_bezasun_finalize(m);
}

extern "C" int zl_bezasun_step(zl_bezasun_t* m, const int32_t* tokens_host, const int32_t* slots_host,
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

extern "C" int zl_bezasun_set_state(zl_bezasun_t* m, const int32_t* tokens_host, const int32_t* positions_host, int B) {
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

extern "C" int zl_bezasun_step_device(zl_bezasun_t* m, int B) {
    ZL_CHECK_ARG(m && B > 0 && B <= m->cfg.max_batch);
    if (m->cur_max_len >= m->cfg.max_seq) return fail(__LINE__, "caches full (max_seq reached)");
    RCHECK(run_step(m, B, B, B, 1, m->cur_max_len));
    k_decode_advance<<<cdiv(B, 64), 64, 0, m->stream>>>(m->d_tokens, m->d_pos, m->d_next, B);
    ZL_CHECK_LAUNCH();
    m->cur_max_len += 1;
    return ZL_OK;
}

extern "C" int zl_bezasun_sync(zl_bezasun_t* m) {
    ZL_CHECK_ARG(m);
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

extern "C" zl_stream_t zl_bezasun_stream(zl_bezasun_t* m) { return m ? (zl_stream_t)m->stream : nullptr; }

extern "C" int zl_bezasun_capture_layers(zl_bezasun_t* m, int on) {
    ZL_CHECK_ARG(m);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    if (on && !m->layer_dump)
        RCHECK(dmalloc((void**)&m->layer_dump, m->layers.size() * m->tcap * m->cfg.width * 4));
    m->capture = on != 0;
    return ZL_OK;
}

extern "C" int zl_bezasun_read_layers(zl_bezasun_t* m, float* out_host, int T) {
    ZL_CHECK_ARG(m && out_host && T > 0 && T <= m->tcap);
    if (!m->layer_dump) return fail(__LINE__, "layer capture was not switched on");
    const size_t row = (size_t)m->cfg.width * 4;
    ZL_CHECK_CUDA(cudaMemcpy2DAsync(out_host, (size_t)T * row, m->layer_dump, (size_t)m->tcap * row, (size_t)T * row,
                                    m->layers.size(), cudaMemcpyDeviceToHost, m->stream));
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    return ZL_OK;
}

extern "C" int zl_bezasun_read_cache(zl_bezasun_t* m, int layer, int slot, int n_rows, float* a_host, float* b_host) {
    ZL_CHECK_ARG(m && a_host && b_host && layer >= 0 && layer < m->cfg.num_layers && slot >= 0 && slot < m->cfg.max_batch);
    ZL_CHECK_ARG(n_rows > 0 && n_rows <= m->cfg.max_seq);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    const BLayer& L = m->layers[layer];
    const auto& lc = L.c;
    ZL_CHECK_ARG(lc.type != ZL_BEZASUN_SSM);
    const bool latent = lc.type == ZL_BEZASUN_LATENT;
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    const size_t kw = (size_t)lc.kv_heads * lc.dim, vw = (size_t)lc.kv_heads * lc.vdim;
    // per output: the cache, elements per cached row, first element, elements wanted
    const SlotCache* caches[2] = {&L.a, latent ? &L.a : &L.b};
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

extern "C" int zl_bezasun_read_state(zl_bezasun_t* m, int layer, int slot, float* out_host) {
    ZL_CHECK_ARG(m && out_host && layer >= 0 && layer < m->cfg.num_layers && slot >= 0 && slot < m->cfg.max_batch);
    if (!m->finalized) return fail(__LINE__, "model not finalized");
    const BLayer& L = m->layers[layer];
    ZL_CHECK_ARG(L.c.type == ZL_BEZASUN_SSM);
    ZL_CHECK_CUDA(cudaStreamSynchronize(m->stream));
    ZL_CHECK_CUDA(cudaMemcpy(out_host, (const char*)L.a.buf + (size_t)slot * L.a.slot_bytes, L.a.slot_bytes, cudaMemcpyDeviceToHost));
    return ZL_OK;
}

extern "C" int zl_bezasun_stats(zl_bezasun_t* m, double* weight_bytes, int* kernels_per_step) {
    ZL_CHECK_ARG(m);
    if (weight_bytes) *weight_bytes = m->weight_bytes;
    if (kernels_per_step) *kernels_per_step = m->kernels_per_step;
    return ZL_OK;
}
