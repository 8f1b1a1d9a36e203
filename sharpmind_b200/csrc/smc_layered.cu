// Decoders described layer by layer (smc_layered_desc): the model object, its per-sequence state and the forward pass.
// One pass serves prompts, portions of prompts and decoding: the rows of a batch are consecutive tokens of one sequence,
// or one token for each of the first sequence slots; kernels find a row's slot and position through smc_rows.
//
// State of a sequence slot, per layer: a latent layer's ring of compressed rows, a state-space layer's fp32 state and
// convolution inputs, a head layer's ring of keys and values and its linear heads' fp32 states.  Positions live on the device (a captured step can advance them itself, SMC_POS_NEXT); the host
// keeps its own count where it knows it and refuses a call that would continue a recurrence at another place.
#include <math.h>

#include <algorithm>
#include <utility>
#include <vector>

#include "smc_common.cuh"

struct smc_layered {
    smc_ctx *ctx = nullptr;
    smc_layered_desc d{};
    std::vector<smc_layer_desc> layers;
    int slots = 0, rows = 0;  // sequence slots; rows a pass may hold
    bool bf16 = false;
    int *pos = nullptr;                // [slots] first position of the pass, [slots] length after it
    std::vector<long long> held;       // tokens a slot holds, -1: only the device knows
    struct State {
        void *ring = nullptr, *conv = nullptr;
        float *ssm = nullptr;  // state-space or linear-attention states
        int ring_rows = 0, bias_len = 0;
        float *bias = nullptr, *decay = nullptr;  // by distance; [heads]
        double *log2_decay = nullptr;
        const float *cosT = nullptr, *sinT = nullptr;
        const void *ukt = nullptr;
    };
    std::vector<State> state;
    struct Table {
        smc_rotation rot;
        float *c, *s;
    };
    std::vector<Table> tables;  // layers with the same rotation share one
    std::vector<std::pair<const smc_weight *, void *>> ukt;  // transposed key expansions, one per weight
    void *oc = nullptr;
    float *x = nullptr, *y = nullptr, *qa = nullptr, *dt_raw = nullptr, *ssm_y = nullptr;
    void *x16 = nullptr, *wide = nullptr, *cq = nullptr, *q = nullptr, *o = nullptr, *keys = nullptr, *kv = nullptr, *xbc = nullptr, *act = nullptr,
         *head = nullptr, *xn = nullptr, *qk = nullptr, *starts = nullptr;
    float *parts = nullptr;
    float *dump = nullptr;
};

namespace {

smc_latent_dims latent_dims(const smc_layered *m, int l)
{
    const smc_layer_desc &L = m->layers[l];
    return smc_latent_dims{L.heads, L.dim, L.rot_dim, L.vdim, L.q_rank, L.kv_rank, L.window, m->state[l].ring_rows, L.scale, m->d.eps};
}
smc_ssm_dims ssm_dims(const smc_layered *m, const smc_layer_desc &L)
{
    return smc_ssm_dims{L.heads, L.vdim, L.state, L.groups, L.conv, L.norm_groups, m->d.eps};
}

smc_attn_dims attn_dims(const smc_layered *m, int l)
{
    const smc_attn_desc &A = m->layers[l].attn;
    return smc_attn_dims{A.heads, A.kv_heads, A.dim, A.vdim, A.window, m->state[l].ring_rows, m->state[l].bias_len, A.scale, A.out_scale, m->d.eps};
}
smc_linear_dims linear_dims(const smc_layered *m, const smc_layer_desc &L)
{
    const smc_linear_desc &A = L.linear;
    return smc_linear_dims{A.heads, A.dim, A.vdim, A.rot.dims, A.norm_parts, A.gate, A.k_scale, A.out_scale, m->d.eps};
}
// rows of a head layer's input projection (attention part, linear part) and columns of its output projection
int attn_in(const smc_layer_desc &L) { return L.attn.heads ? L.attn.heads * L.attn.dim + L.attn.kv_heads * (L.attn.dim + L.attn.vdim) : 0; }
int linear_in(const smc_layer_desc &L) { return 2 * L.linear.heads * (L.linear.dim + L.linear.vdim); }
int mix_out(const smc_layer_desc &L)
{
    return L.mixer == SMC_MIX_HEADS ? L.attn.heads * L.attn.vdim + L.linear.heads * L.linear.vdim : L.heads * L.vdim;
}

bool shape_is(const smc_weight *w, long long n, long long k) { return w && w->dtype == SMC_BF16 && w->N == n && w->K == k; }

int check_layer(smc_ctx *ctx, const smc_layered_desc &d, const smc_layer_desc &L, int l)
{
    auto bad = [&](const char *what) { return smc_fail(ctx, SMC_E_INVALID, "model_create_layered: layer %d: %s", l, what); };
    const int H = d.hidden;
    if ((L.mixer != SMC_MIX_HEADS && (L.heads <= 0 || L.vdim <= 0)) || !L.norm1) return bad("incomplete description");
    if (!shape_is(L.w_out, H, mix_out(L))) return bad("output projection shape");
    if (L.mixer == SMC_MIX_LATENT) {
        if (L.dim <= 0 || L.rot_dim <= 0 || L.q_rank <= 0 || L.kv_rank <= 0 || L.window < 0 || !L.q_norm || !L.kv_norm) return bad("latent attention sizes");
        if (L.rot.dims != L.rot_dim) return bad("the rotation covers another width than the rotated part");
        if (!shape_is(L.w_down, (long long)L.q_rank + L.kv_rank + L.rot_dim, H) || !shape_is(L.w_uq, (long long)L.heads * (L.dim + L.rot_dim), L.q_rank) ||
            !shape_is(L.w_ukv, (long long)L.heads * (L.dim + L.vdim), L.kv_rank))
            return bad("latent attention weight shapes");
        smc_latent_dims ld{L.heads, L.dim, L.rot_dim, L.vdim, L.q_rank, L.kv_rank, L.window, 0, L.scale, d.eps};
        int rc = smc_latent_check(ctx, ld);
        if (rc) return rc;
    } else if (L.mixer == SMC_MIX_MAMBA2) {
        if (L.state <= 0 || L.groups <= 0 || L.heads % L.groups || L.conv <= 0 || L.norm_groups <= 0 || (L.heads * L.vdim) % L.norm_groups || !L.conv_w ||
            !L.conv_b || !L.dt_bias || !L.a_log || !L.d_skip || !L.mix_norm)
            return bad("state-space sizes");
        if (L.state > 512) return smc_fail(ctx, SMC_E_UNSUPPORTED, "model_create_layered: layer %d: state %d (up to 512 are built)", l, L.state);
        if (!shape_is(L.w_in, 2LL * L.heads * L.vdim + 2LL * L.groups * L.state + L.heads, H)) return bad("input projection shape");
    } else if (L.mixer == SMC_MIX_HEADS) {
        const smc_attn_desc &A = L.attn;
        const smc_linear_desc &R = L.linear;
        if (A.heads < 0 || R.heads < 0 || A.heads + R.heads == 0) return bad("no heads");
        if (A.heads) {
            if (A.kv_heads <= 0 || A.heads % A.kv_heads || A.dim <= 0 || A.vdim <= 0 || A.window < 0) return bad("attention head sizes");
            if (A.bias && (A.buckets < 2 || !(A.bias_max > A.buckets / 2))) return bad("distance buckets");
            int rc = smc_attn_check(ctx, smc_attn_dims{A.heads, A.kv_heads, A.dim, A.vdim, A.window, 0, 0, A.scale, A.out_scale, d.eps});
            if (rc) return rc;
        }
        if (R.heads) {
            if (R.dim <= 0 || R.vdim <= 0 || R.norm_parts <= 0 || R.heads * R.vdim % R.norm_parts || R.rot.dims < 0 || !R.decay) return bad("linear attention sizes");
            for (int h = 0; h < R.heads; ++h)
                if (!(R.decay[h] > 0.0 && R.decay[h] <= 1.0)) return bad("a decay outside (0, 1]");
            int rc = smc_linear_check(ctx, smc_linear_dims{R.heads, R.dim, R.vdim, R.rot.dims, R.norm_parts, R.gate, R.k_scale, R.out_scale, d.eps});
            if (rc) return rc;
        }
        if (!shape_is(L.w_in, attn_in(L) + linear_in(L), H)) return bad("input projection shape");
    } else {
        return smc_fail(ctx, SMC_E_UNSUPPORTED, "model_create_layered: layer %d: mixer %d", l, L.mixer);
    }
    if (L.ffn < 0 || (L.ffn > 0 && (!L.norm2 || !shape_is(L.w_gu, 2LL * L.ffn, H) || !shape_is(L.w_ffn_down, H, L.ffn)))) return bad("feed-forward");
    return SMC_OK;
}

bool same_rotation(const smc_rotation &a, const smc_rotation &b)
{
    return a.dims == b.dims && a.base == b.base && a.factor == b.factor && a.original == b.original && a.fast == b.fast && a.slow == b.slow;
}

}  // namespace

void smc_layered_free(smc_layered *m)
{
    if (!m) return;
    for (auto &s : m->state) cudaFree(s.ring), cudaFree(s.conv), cudaFree(s.ssm), cudaFree(s.bias), cudaFree(s.decay), cudaFree(s.log2_decay);
    for (auto &t : m->tables) cudaFree(t.c), cudaFree(t.s);
    for (auto &t : m->ukt) cudaFree(t.second);
    void *bufs[] = {m->pos, m->x, m->y, m->qa, m->oc, m->dt_raw, m->ssm_y, m->x16, m->wide, m->cq, m->q, m->o, m->keys, m->kv, m->xbc, m->act, m->head,
                    m->xn, m->qk, m->starts, m->parts};
    for (void *p : bufs) cudaFree(p);
    delete m;
}

int smc_layered_slots(const smc_layered *m) { return m->slots; }
int smc_layered_length(const smc_layered *m, int seq) { return (int)m->held[seq]; }
void smc_layered_reset(smc_layered *m, int seq) { m->held[seq] = 0; }
void smc_layered_dump(smc_layered *m, float *d_dump) { m->dump = d_dump; }

int smc_layered_create(smc_ctx *ctx, const smc_layered_desc *desc, int max_batch, smc_layered **out)
{
    const smc_layered_desc &d = *desc;
    if (d.n_layers <= 0 || d.hidden <= 0 || d.vocab <= 0 || d.max_seq <= 0 || d.max_chunk <= 0 || !d.layers || !d.final_norm)
        return smc_fail(ctx, SMC_E_INVALID, "model_create_layered: incomplete description");
    if (d.act_dtype != SMC_F32 && d.act_dtype != SMC_BF16)
        return smc_fail(ctx, SMC_E_UNSUPPORTED, "model_create_layered: act_dtype %d (fp32 = 0 and bfloat16 = 30)", d.act_dtype);
    if ((d.norm_place != SMC_NORM_AFTER && d.norm_place != SMC_NORM_BEFORE) || (d.ffn_act != SMC_FFN_SILU && d.ffn_act != SMC_FFN_GELU_TANH))
        return smc_fail(ctx, SMC_E_UNSUPPORTED, "model_create_layered: norm_place %d, ffn_act %d", d.norm_place, d.ffn_act);
    if (!shape_is(d.embedding, d.vocab, d.hidden)) return smc_fail(ctx, SMC_E_SIZE_MISMATCH, "model_create_layered: the embedding must be bfloat16 [vocab, hidden]");
    for (int l = 0; l < d.n_layers; ++l) {
        int rc = check_layer(ctx, d, d.layers[l], l);
        if (rc) return rc;
    }
    cudaSetDevice(ctx->device);
    smc_layered *m = new smc_layered();
    m->ctx = ctx, m->d = d, m->layers.assign(d.layers, d.layers + d.n_layers), m->d.layers = nullptr;
    m->slots = max_batch, m->bf16 = d.act_dtype == SMC_BF16;
    m->d.max_chunk = std::min(d.max_chunk, d.max_seq);
    m->rows = std::max(max_batch, m->d.max_chunk);
    m->held.assign(max_batch, 0);
    m->state.resize(d.n_layers);
    const size_t R = m->rows, el = m->bf16 ? 2 : 4, B = max_batch;
    cudaError_t e = cudaSuccess;
    int rc = SMC_OK;
    auto alloc = [&](auto **p, size_t bytes, bool zero = false) {
        if (e == cudaSuccess && bytes) e = cudaMalloc(p, bytes);
        if (e == cudaSuccess && bytes && zero) e = cudaMemset(*p, 0, bytes);
    };
    // cosine and sine tables of a rotation
    auto table = [&](const smc_rotation &rot, smc_layered::State &st) {
        auto it = std::find_if(m->tables.begin(), m->tables.end(), [&](const smc_layered::Table &t) { return same_rotation(t.rot, rot); });
        if (it == m->tables.end()) {
            smc_layered::Table t{rot, nullptr, nullptr};
            const size_t bytes = (size_t)d.max_seq * (rot.dims / 2) * sizeof(float);
            alloc(&t.c, bytes), alloc(&t.s, bytes);
            m->tables.push_back(t);
            if (e == cudaSuccess) rc = smc_rope_tables_yarn(ctx, &rot, d.max_seq, t.c, t.s);
            it = m->tables.end() - 1;
        }
        st.cosT = it->c, st.sinT = it->s;
    };
    size_t qk = 0, parts = 0;
    size_t wide = 0, cq = 0, q = 0, qa = 0, oc = 0, o = 0, keys = 0, kv = 0, dt = 0, xbc = 0, sy = 0, act = 0;
    for (int l = 0; l < d.n_layers; ++l) {
        smc_layer_desc &L = m->layers[l];
        smc_layered::State &st = m->state[l];
        o = std::max(o, (size_t)mix_out(L)), act = std::max(act, (size_t)L.ffn);
        if (L.mixer == SMC_MIX_LATENT) {
            const size_t row = (size_t)L.kv_rank + L.rot_dim;
            st.ring_rows = L.window > 0 ? (int)std::min<long long>(d.max_seq, (long long)L.window - 1 + m->d.max_chunk) : d.max_seq;
            alloc(&st.ring, B * st.ring_rows * row * el, true);
            wide = std::max(wide, L.q_rank + row), cq = std::max(cq, (size_t)L.q_rank), q = std::max(q, (size_t)L.heads * (L.dim + L.rot_dim));
            qa = std::max(qa, L.heads * row), oc = std::max(oc, (size_t)L.heads * L.kv_rank);
            if (m->bf16 && smc_latent_prefill_supported(latent_dims(m, l))) {
                const size_t seen = (size_t)std::min<long long>(d.max_seq, (L.window > 0 ? L.window - 1 : d.max_seq) + (long long)m->d.max_chunk);
                keys = std::max(keys, seen * row), kv = std::max(kv, seen * L.heads * (L.dim + L.vdim));
            }
            table(L.rot, st);
            if (m->bf16 && smc_latent_decode_supported(latent_dims(m, l))) {
                auto u = std::find_if(m->ukt.begin(), m->ukt.end(), [&](auto &t) { return t.first == L.w_ukv; });
                if (u == m->ukt.end()) {
                    void *t = nullptr;
                    alloc(&t, (size_t)L.heads * L.dim * L.kv_rank * 2);
                    m->ukt.emplace_back(L.w_ukv, t);
                    if (e == cudaSuccess && !rc) rc = smc_latent_transpose_uk(ctx, latent_dims(m, l), L.w_ukv, t, ctx->stream);
                    u = m->ukt.end() - 1;
                }
                st.ukt = u->second;
            }
        } else if (L.mixer == SMC_MIX_HEADS) {
            const smc_attn_desc &A = L.attn;
            smc_linear_desc &R = L.linear;
            wide = std::max(wide, (size_t)attn_in(L) + linear_in(L));
            if (A.heads) {
                st.ring_rows = A.window > 0 ? (int)std::min<long long>(d.max_seq, (long long)A.window - 1 + m->d.max_chunk) : d.max_seq;
                alloc(&st.ring, B * st.ring_rows * A.kv_heads * (A.dim + A.vdim) * el, true);
                q = std::max(q, (size_t)A.heads * A.dim);
                if (A.bias) {
                    st.bias_len = A.window > 0 ? std::min(A.window, d.max_seq) : d.max_seq;
                    alloc(&st.bias, (size_t)A.heads * st.bias_len * sizeof(float));
                    if (e == cudaSuccess && !rc) rc = smc_attn_expand_bias(ctx, A.bias, A.heads, A.buckets, A.bias_max, st.bias_len, st.bias, ctx->stream);
                }
            }
            if (R.heads) {
                const size_t inner = (size_t)R.heads * R.vdim;
                std::vector<float> decay(R.heads);
                std::vector<double> l2(R.heads);
                for (int h = 0; h < R.heads; ++h) decay[h] = (float)R.decay[h], l2[h] = log2(R.decay[h]);
                alloc(&st.decay, decay.size() * sizeof(float)), alloc(&st.log2_decay, l2.size() * sizeof(double));
                if (e == cudaSuccess) e = cudaMemcpy(st.decay, decay.data(), decay.size() * sizeof(float), cudaMemcpyHostToDevice);
                if (e == cudaSuccess) e = cudaMemcpy(st.log2_decay, l2.data(), l2.size() * sizeof(double), cudaMemcpyHostToDevice);
                alloc(&st.ssm, B * inner * R.dim * sizeof(float), true);
                sy = std::max(sy, inner);
                if (R.rot.dims) table(R.rot, st);
                if (m->bf16 && smc_linear_chunks_supported(linear_dims(m, L))) {
                    if (R.rot.dims) qk = std::max(qk, 2 * (size_t)R.heads * R.dim);
                    parts = std::max(parts, (m->d.max_chunk + SMC_LINEAR_CHUNK - 1) / SMC_LINEAR_CHUNK * inner * R.dim);
                }
            }
            R.decay = nullptr;  // the caller's array
        } else {
            const size_t inner = (size_t)L.heads * L.vdim, ch = inner + 2 * (size_t)L.groups * L.state;
            alloc(&st.conv, B * L.conv * ch * el, true);
            alloc(&st.ssm, B * inner * L.state * sizeof(float), true);
            wide = std::max(wide, inner + ch), dt = std::max(dt, (size_t)L.heads), xbc = std::max(xbc, ch), sy = std::max(sy, inner);
        }
        if (rc || e != cudaSuccess) break;
    }
    alloc(&m->pos, 2 * B * sizeof(int), true);
    alloc(&m->x, R * d.hidden * 4), alloc(&m->y, d.norm_place == SMC_NORM_AFTER ? R * d.hidden * 4 : 0), alloc(&m->x16, m->bf16 ? R * d.hidden * 2 : 0);
    alloc(&m->xn, !m->bf16 && d.norm_place == SMC_NORM_BEFORE ? R * d.hidden * 4 : 0), alloc(&m->qk, R * qk * el);
    alloc(&m->parts, parts * 4), alloc(&m->starts, parts * 4), alloc(&m->head, R * d.hidden * el);
    alloc(&m->wide, R * wide * el), alloc(&m->cq, R * cq * el), alloc(&m->q, R * q * el), alloc(&m->qa, R * qa * 4), alloc(&m->oc, R * oc * 4);
    alloc(&m->o, R * o * el), alloc(&m->keys, keys * el), alloc(&m->kv, kv * el), alloc(&m->dt_raw, R * dt * 4), alloc(&m->xbc, R * xbc * el);
    alloc(&m->ssm_y, R * sy * 4), alloc(&m->act, R * act * el);
    if (e != cudaSuccess && !rc) rc = smc_fail(ctx, SMC_E_CUDA, "model_create_layered: allocation failed: %s", cudaGetErrorString(e));
    if (rc) {
        smc_layered_free(m);
        return rc;
    }
    SMC_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    *out = m;
    return SMC_OK;
}

int smc_layered_forward(smc_ctx *ctx, smc_layered *m, const int *d_tokens, int count, int seq0, int pos, int mode, int all_rows, const int *d_rows,
                        int n_rows, float *d_logits, int *d_argmax, float *d_hidden, cudaStream_t s)
{
    const smc_layered_desc &d = m->d;
    if (mode != (m->bf16 ? SMC_ACT_BF16 : SMC_ACT_F32))
        return smc_fail(ctx, SMC_E_UNSUPPORTED, "layered model: mode %d, the model was created for %s activations", mode, m->bf16 ? "bfloat16" : "fp32");
    if (count <= 0 || (seq0 < 0 ? count > m->slots : count > m->d.max_chunk))
        return smc_fail(ctx, SMC_E_RANGE, "layered model: %d tokens in one pass (chunk %d, slots %d)", count, d.max_chunk, m->slots);
    if (seq0 >= m->slots) return smc_fail(ctx, SMC_E_RANGE, "layered model: sequence %d outside [0, %d)", seq0, m->slots);
    if (pos < SMC_POS_NEXT || (pos == SMC_POS_NEXT && seq0 >= 0) || (long long)pos + (seq0 < 0 ? 1 : count) > d.max_seq)
        return smc_fail(ctx, SMC_E_RANGE, "layered model: position %d + %d tokens exceeds %d", pos, seq0 < 0 ? 1 : count, d.max_seq);
    const int a = seq0 < 0 ? 0 : seq0, b = seq0 < 0 ? count : seq0 + 1;
    for (int i = a; i < b && pos > 0; ++i)
        if (m->held[i] >= 0 && m->held[i] != pos)
            return smc_fail(ctx, SMC_E_RANGE, "layered model: sequence %d holds %lld tokens, it cannot continue at position %d", i, m->held[i], pos);
    for (int i = a; i < b; ++i) m->held[i] = pos == SMC_POS_NEXT ? -1 : pos + (seq0 < 0 ? 1 : count);

    const int H = d.hidden, n = count, bf = m->bf16;
    const smc_rows rw{m->pos, seq0, n};
    int rc;
#define SMC_TRY(call)        \
    do {                     \
        rc = (call);         \
        if (rc) return rc;   \
    } while (0)
    auto to = [&](void *y, int ld, int y_bf16) {
        smc_dense_out out{};
        out.y = y, out.ldy = ld, out.y_bf16 = y_bf16;
        return out;
    };
    const bool before = d.norm_place == SMC_NORM_BEFORE;
    void *xin = bf ? m->x16 : (before ? m->xn : static_cast<void *>(m->x));  // what the matmuls of a layer read
    const float escale = d.embed_scale != 0.f ? d.embed_scale : 1.0f;
    SMC_TRY(smc_launch_embed_bf16(ctx, d.embedding, d_tokens, n, m->x, before ? nullptr : m->x16, m->pos, m->slots, seq0, pos, d.max_seq, escale, s));
    // a part's output joins x: summed by the matmul that makes it, or scaled, summed and normed after it
    auto join = [&](const void *a, int k, const smc_weight *w, const float *norm) -> int {
        smc_dense_out out = to(before ? m->x : m->y, H, 0);
        out.accumulate = before;
        int rc = smc_launch_dense(ctx, a, bf, k, w, n, out, s);
        return rc || before ? rc : smc_scaled_add_rmsnorm_dev(ctx, m->x, m->y, norm, m->x16, n, H, d.alpha, 1.0f, d.eps, s);
    };
    // a matmul over the layer's input, normed first where the norm comes before
    auto project = [&](const float *norm, const smc_weight *w, const smc_dense_out &out) -> int {
        if (before) return smc_launch_dense_layernorm(ctx, m->x, norm, d.eps, xin, bf, w, n, out, s);
        return smc_launch_dense(ctx, xin, bf, H, w, n, out, s);
    };
    for (int l = 0; l < d.n_layers; ++l) {
        const smc_layer_desc &L = m->layers[l];
        smc_layered::State &st = m->state[l];
        if (L.mixer == SMC_MIX_LATENT) {
            const smc_latent_dims ld = latent_dims(m, l);
            const smc_latent_bufs lb{m->wide, m->cq, m->q, m->qa, m->oc, st.ukt, m->o, m->keys, m->kv, st.ring};
            SMC_TRY(project(L.norm1, L.w_down, to(m->wide, L.w_down->N, bf)));
            SMC_TRY(smc_latent_post(ctx, ld, lb, rw, bf, L.q_norm, L.kv_norm, st.cosT, st.sinT, d.max_seq, s));
            SMC_TRY(smc_launch_dense(ctx, m->cq, bf, L.q_rank, L.w_uq, n, to(m->q, L.w_uq->N, bf), s));
            SMC_TRY(smc_latent_attend(ctx, ld, lb, rw, bf, L.w_ukv, L.sink, st.cosT, st.sinT, d.max_seq, pos, s));
        } else if (L.mixer == SMC_MIX_HEADS) {
            const int ld = L.w_in->N, ldo = mix_out(L), lc = attn_in(L);
            smc_dense_out out = to(m->wide, ld, bf);
            out.bias = L.b_in;
            if (L.linear.heads && L.linear.silu) out.silu_from = lc, out.silu_to = ld - L.linear.heads * L.linear.vdim;
            SMC_TRY(project(L.norm1, L.w_in, out));
            char *o2 = static_cast<char *>(m->o) + (size_t)L.attn.heads * L.attn.vdim * (bf ? 2 : 4);  // the linear heads' columns
            if (L.attn.heads) {
                const smc_attn_bufs ab{m->wide, ld, 0, m->q, st.ring, m->o, ldo, L.attn.q_norm, L.attn.k_norm, st.bias};
                SMC_TRY(smc_attn_mix(ctx, attn_dims(m, l), ab, rw, bf, pos, s));
            }
            if (L.linear.heads) {
                const smc_linear_bufs lb{m->wide, ld, lc, m->qk, m->ssm_y, m->parts, m->starts, st.ssm, o2, ldo, st.log2_decay, st.decay, L.linear.mix_norm,
                                         st.cosT, st.sinT, d.max_seq};
                SMC_TRY(smc_linear_mix(ctx, linear_dims(m, L), lb, rw, bf, s));
            }
        } else {
            const int ld = 2 * L.heads * L.vdim + 2 * L.groups * L.state;
            smc_dense_out out = to(m->wide, ld, bf);
            out.y32 = m->dt_raw, out.ld32 = L.heads, out.split = ld;  // step sizes stay fp32
            SMC_TRY(project(L.norm1, L.w_in, out));
            const smc_ssm_bufs sb{m->wide, ld, m->dt_raw, m->xbc, m->ssm_y, m->o, st.conv, st.ssm};
            SMC_TRY(smc_ssm_mix(ctx, ssm_dims(m, L), sb, rw, bf, L.conv_w, L.conv_b, L.dt_bias, L.a_log, L.d_skip, L.mix_norm, s));
        }
        SMC_TRY(join(m->o, mix_out(L), L.w_out, L.norm1));
        if (L.ffn) {
            smc_dense_out out = to(m->act, L.ffn, bf);
            out.woven = d.ffn_act == SMC_FFN_GELU_TANH ? 2 : 1;
            SMC_TRY(project(L.norm2, L.w_gu, out));
            SMC_TRY(join(m->act, L.ffn, L.w_ffn_down, L.norm2));
        }
        if (m->dump)
            SMC_CUDA(ctx, cudaMemcpyAsync(m->dump + (size_t)l * d.max_chunk * H, m->x,
                                          (size_t)std::min(n, d.max_chunk) * H * sizeof(float),
                                          cudaMemcpyDeviceToDevice, s));
    }
    auto final_norm = [&](const int *rows, int first, int count, void *out, int out_bf16) -> int {
        if (before) return smc_launch_layernorm(ctx, m->x, rows, first, count, d.final_norm, out, out_bf16, H, d.eps, s);
        return smc_launch_rmsnorm_gather(ctx, m->x, rows, first, count, d.final_norm, out, out_bf16, H, 1.0f, d.eps, s);
    };
    if (d_hidden) SMC_TRY(final_norm(nullptr, 0, n, d_hidden, 0));
    const int wanted = all_rows == 0 ? 1 : (all_rows == 1 ? n : n_rows);
    if (wanted == 0) return SMC_OK;
    if (wanted > m->rows) return smc_fail(ctx, SMC_E_RANGE, "layered model: %d logit rows of a pass of %d tokens", wanted, n);
    smc_dense_out logits = to(d_logits, d.vocab, 0);
    logits.softcap = d.softcap;
    if (before && wanted == 1 && all_rows != 2) {
        SMC_TRY(smc_launch_dense_layernorm(ctx, m->x + (size_t)(n - 1) * H, d.final_norm, d.eps, m->head, bf, d.embedding, 1, logits, s));
    } else {
        SMC_TRY(final_norm(all_rows == 2 ? d_rows : nullptr, all_rows == 0 ? n - 1 : 0, wanted, m->head, bf));
        SMC_TRY(smc_launch_dense(ctx, m->head, bf, H, d.embedding, wanted, logits, s));
    }
    if (d_argmax) SMC_TRY(smc_argmax_dev(ctx, d_logits, wanted, d.vocab, d_argmax, s));
#undef SMC_TRY
    return SMC_OK;
}
