// Models whose layers are listed one by one (oxg4_model_create_layered): every layer names its mixer, its sizes and an
// optional feed-forward. Two blocks: x += norm1b(mixer(norm1(x))), x += norm2b(ff(norm2(x))), and the parallel one,
// h = norm1(x), x += mixer(h) + ff(h), whose input matrices (mixer, gate and up rows) are one matrix and whose output
// matrices are one matrix over [mixer output | feed-forward activations]. This file turns the list into plans,
// adds the caches and states of the mixers to the cache table and sequences a pass over the layers; positions, pages,
// chunks of prompts, graphs, sampling and generation are those of oxg4.cu, which includes it.
//
// A pass takes one of three forms:
//   one row (a decode step of one sequence)  gemv.cuh with norms, token shift and output norms in the prologues
//   BF16 weights, many rows                  tc_gemm.cuh, row kernels around it
//   f32 weights, many rows                   gemv.cuh in passes of up to four rows, the same row kernels
//
// Residual rows, weight rows and weight columns are zero-padded to multiples of 8, so that every size of a model is
// allowed while the kernels keep their 16-byte accesses; means divide by the true width.

static inline int pad_to(int v, int q) { return (v + q - 1) / q * q; }
constexpr int kSegTile = kTcTileM;            // segments start at a tile of the tcgen05 projection

extern "C" int32_t oxg4_model_create_layered(const oxg4_layered_config* lc, int32_t device, oxg4_model** out) {
    if (!lc || !out) return fail(OXG4_INVALID_ARGUMENT, "null argument");
    *out = nullptr;
    if (lc->vocab_size <= 0 || lc->width <= 0 || lc->num_layers <= 0 || !lc->layers)
        return fail(OXG4_INVALID_SHAPE, "invalid layered configuration");
    if (lc->weight_dtype != OXG4_F32 && lc->weight_dtype != OXG4_BF16)
        return fail(OXG4_INVALID_ARGUMENT, "weight_dtype must be OXG4_F32 or OXG4_BF16");
    const int max_width = std::min(kSimtMaxJ * kSimtThreads, kRowsMaxJ * 4 * kRowsThreads);
    if (lc->width > std::min(max_width, kGemvMaxJ * kGemvThreads))
        return fail(OXG4_UNSUPPORTED, "width above %d is not supported", std::min(max_width, kGemvMaxJ * kGemvThreads));
    const int L = lc->num_layers;
    if (lc->block != OXG4_BLOCK_SANDWICH && lc->block != OXG4_BLOCK_PARALLEL) return fail(OXG4_INVALID_ARGUMENT, "unknown block %d", lc->block);
    if (lc->act != OXG4_ACT_GELU_TANH && lc->act != OXG4_ACT_SILU && lc->act != OXG4_ACT_RELU)
        return fail(OXG4_INVALID_ARGUMENT, "unknown activation %d", lc->act);
    const bool parallel = lc->block == OXG4_BLOCK_PARALLEL;
    for (int l = 0; l < L; ++l) {
        const oxg4_layer_spec& s = lc->layers[l];
        if (s.heads <= 0 || s.dim <= 0 || s.vdim <= 0 || s.ff < 0) return fail(OXG4_INVALID_SHAPE, "layer %d: invalid sizes", l);
        if (s.weights_of < -1 || s.weights_of >= L || s.weights_of == l || (s.weights_of >= 0 && lc->layers[s.weights_of].weights_of >= 0 &&
                                                                            lc->layers[s.weights_of].weights_of == l))
            return fail(OXG4_INVALID_ARGUMENT, "layer %d: invalid weights_of", l);
        switch (s.mixer) {
            case OXG4_MIXER_LATENT_ATTENTION:
                if (s.q_rank <= 0 || s.kv_rank <= 0 || s.rot_dim < 0 || s.rot_dims < 0 || s.rot_dims > s.rot_dim || s.rot_dims % 2)
                    return fail(OXG4_INVALID_SHAPE, "layer %d: invalid latent attention sizes", l);
                if (s.kv_rank > 512) return fail(OXG4_UNSUPPORTED, "layer %d: kv_rank above 512 is not supported", l);
                break;
            case OXG4_MIXER_LIGHTNING:
                if (!s.decay) return fail(OXG4_INVALID_ARGUMENT, "layer %d: decay is missing", l);
                if (s.dim > 512) return fail(OXG4_UNSUPPORTED, "layer %d: key size above 512 is not supported", l);
                break;
            case OXG4_MIXER_WKV:
                if (s.vdim != s.dim) return fail(OXG4_INVALID_SHAPE, "layer %d: invalid time-mixing sizes", l);
                if (s.dim > 512) return fail(OXG4_UNSUPPORTED, "layer %d: key size above 512 is not supported", l);
                break;
            case OXG4_MIXER_RETENTION:
                if (!s.decay) return fail(OXG4_INVALID_ARGUMENT, "layer %d: decay is missing", l);
                if (s.rot_dims < 0 || s.rot_dims > s.dim || s.rot_dims % 2) return fail(OXG4_INVALID_SHAPE, "layer %d: invalid rotation", l);
                if (s.dim > 512) return fail(OXG4_UNSUPPORTED, "layer %d: key size above 512 is not supported", l);
                break;
            case OXG4_MIXER_ATTENTION:
                if (s.kv_heads <= 0 || s.heads % s.kv_heads) return fail(OXG4_INVALID_SHAPE, "layer %d: query heads must be a multiple of kv heads", l);
                if (s.q_temp_every <= 0) return fail(OXG4_INVALID_ARGUMENT, "layer %d: q_temp_every must be positive", l);
                if (s.vdim > 512) return fail(OXG4_UNSUPPORTED, "layer %d: value size above 512 is not supported", l);
                if (s.dim > 1024) return fail(OXG4_UNSUPPORTED, "layer %d: key size above 1024 is not supported", l);
                if ((size_t)s.heads * s.dim * 4 > 200 * 1024)
                    return fail(OXG4_UNSUPPORTED, "layer %d: more than 51200 query values per token are not supported", l);
                break;
            default:
                return fail(OXG4_INVALID_ARGUMENT, "layer %d: unknown mixer %d", l, s.mixer);
        }
        if (parallel != (s.mixer == OXG4_MIXER_RETENTION || s.mixer == OXG4_MIXER_ATTENTION))
            return fail(OXG4_UNSUPPORTED, "layer %d: mixer %d is not available in block %d", l, s.mixer, lc->block);
    }
    // the rest of the model is created as a one-kind attention model of the same depth and vocabulary would be
    std::vector<int32_t> sliding(L, 0), rotary(L, 64);
    std::vector<float> theta(L, 10000.0f), factor(L, 1.0f);
    oxg4_config c{};
    c.vocab_size = lc->vocab_size;
    c.hidden_size = pad_to(lc->width, 8);
    c.num_hidden_layers = L;
    c.num_attention_heads = c.num_key_value_heads = 1;
    c.head_dim = c.global_head_dim = 64;
    c.intermediate_size = 8;
    c.sliding_window = 1;
    c.rms_norm_eps = lc->norm_eps;
    c.weight_dtype = lc->weight_dtype;
    c.layer_is_sliding = sliding.data();
    c.rotary_dim = rotary.data();
    c.rope_theta = theta.data();
    c.rope_factor = factor.data();
    c.tp_size = 1;
    TRY(oxg4_model_create(&c, device, out));
    oxg4_model* m = *out;
    m->layered = true;
    m->parallel = parallel;
    m->ff_act = lc->act;
    m->norm_offset = lc->norm_weight_offset ? 1.0f : 0.0f;
    m->Hn = lc->width;
    m->specs.assign(lc->layers, lc->layers + L);
    m->spec_decay.resize(L);
    for (int l = 0; l < L; ++l) {
        if (m->specs[l].mixer == OXG4_MIXER_LIGHTNING || m->specs[l].mixer == OXG4_MIXER_RETENTION)
            m->spec_decay[l].assign(m->specs[l].decay, m->specs[l].decay + m->specs[l].heads);
        m->specs[l].decay = m->spec_decay[l].data();
    }
    return OXG4_OK;
}

// ---- weights --------------------------------------------------------------------------------------------------
static int32_t owned_alloc(oxg4_model* m, void** d, size_t bytes) {
    CK(cudaMalloc(d, std::max<size_t>(bytes, 16)));
    m->owned.push_back(*d);
    m->owned_bytes += (int64_t)bytes;
    CK(cudaMemset(*d, 0, std::max<size_t>(bytes, 16)));
    return OXG4_OK;
}

// f32 copy of a small tensor (matrices of a BF16 model are widened) plus `offset`, padded with zeros to n_pad values
static int32_t small_f32(oxg4_model* m, const std::string& name, int64_t n, int64_t n_pad, const float** out, float offset = 0.0f) {
    const Tensor* t;
    TRY(need(m, name, {n}, &t));
    std::vector<float> f((size_t)n_pad, 0.0f);
    if (t->dtype == OXG4_F32) {
        CK(cudaMemcpy(f.data(), t->d, sizeof(float) * n, cudaMemcpyDeviceToHost));
    } else {
        std::vector<uint16_t> h((size_t)n);
        CK(cudaMemcpy(h.data(), t->d, 2 * n, cudaMemcpyDeviceToHost));
        for (int64_t i = 0; i < n; ++i) f[i] = host_bf16_to_f32(h[i]);
    }
    for (int64_t i = 0; i < n; ++i) f[i] += offset;
    void* d;
    TRY(owned_alloc(m, &d, sizeof(float) * n_pad));
    CK(cudaMemcpy(d, f.data(), sizeof(float) * n_pad, cudaMemcpyHostToDevice));
    *out = (const float*)d;
    return OXG4_OK;
}

struct StackPart {
    std::string name;
    int64_t rows;
    int64_t at;              // first row in the stacked matrix
    int64_t step = 1;        // distance of its rows there
    int64_t col = 0;         // first column
    int64_t cols = 0;        // columns; 0: the stack's
};
// [N, K] matrix with the given tensors (each [rows, cols]) at their places, everything else zero. A single tensor that needs
// no padding is used as it is; the parts of a stack are released.
static int32_t stack_rows(oxg4_model* m, const std::vector<StackPart>& parts, int64_t cols, int64_t N, int64_t K, const void** out) {
    const Tensor* t;
    for (auto& p : parts) TRY(need(m, p.name, {p.rows, p.cols ? p.cols : cols}, &t));
    if (parts.size() == 1 && parts[0].rows == N && cols == K) {
        *out = t->d;
        return OXG4_OK;
    }
    void* d;
    TRY(owned_alloc(m, &d, (size_t)N * K * m->es));
    for (auto& p : parts) {
        const int64_t pc = p.cols ? p.cols : cols;
        TRY(need(m, p.name, {p.rows, pc}, &t));
        CK(cudaMemcpy2D((char*)d + ((size_t)p.at * K + p.col) * m->es, (size_t)p.step * K * m->es, t->d, (size_t)pc * m->es, (size_t)pc * m->es,
                        (size_t)p.rows, cudaMemcpyDeviceToDevice));
    }
    CK(cudaDeviceSynchronize());
    for (auto& p : parts) {
        auto it = m->tensors.find(p.name);
        cudaFree(it->second.d);
        m->tensors.erase(it);
    }
    *out = d;
    return OXG4_OK;
}

static Proj make_proj(const oxg4_model* m, const void* w, int N, int K, int nseg = 1, int seg_rows = 0) {
    Proj p;
    p.w = w;
    p.N = N;
    p.K = K;
    p.nseg = nseg;
    p.seg_rows = seg_rows;
    p.gp = make_plan(N, K, m->es, m->num_sms, 1);
    return p;
}

// w[h][d][r] (heads x dim x rank) -> t[h][r][d], rows of a head padded to seg_rows, columns to ld
__global__ void transpose_heads_kernel(const uint16_t* w, uint16_t* t, int heads, int dim, int rank, int seg_rows, int ld) {
    const size_t n = (size_t)heads * dim * rank;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) {
        const int r = (int)(i % rank), d = (int)(i / rank % dim), h = (int)(i / ((size_t)rank * dim));
        t[((size_t)h * seg_rows + r) * ld + d] = w[i];
    }
}

// layer of the parallel block: one input matrix (mixer rows, then alternately gate and up rows), one output matrix over
// [mixer output | feed-forward]
static int32_t finalize_parallel(oxg4_model* m, const std::string& pre, const oxg4_layer_spec& s, MixPlan& x) {
    const std::string mx = pre + "mix.";
    const int H = m->Hn, Hp = m->H, HD = x.heads * x.dim;
    const bool attention = x.kind == MIX_ATTENTION;
    const int kn = attention ? x.kv_heads * x.dim : HD, vn = attention ? x.kv_heads * x.vdim : x.ow;
    x.c_k = pad_to(HD, 8);
    x.c_v = x.c_k + pad_to(kn, 8);
    x.c_g = x.c_v + pad_to(vn, 8);
    x.c_ff = x.c_g + (attention ? 0 : pad_to(x.ow, 8));
    std::vector<StackPart> parts = {{mx + "q", HD, 0}, {mx + "k", kn, x.c_k}, {mx + "v", vn, x.c_v}};
    if (!attention) parts.push_back({mx + "g", x.ow, x.c_g});
    if (x.ff > 0) {
        parts.push_back({pre + "mlp.gate", x.ff, x.c_ff, 2});
        parts.push_back({pre + "mlp.up", x.ff, x.c_ff + 1, 2});
    }
    const void* w = nullptr;
    const int N = x.c_ff + 2 * x.ffp;
    TRY(stack_rows(m, parts, H, N, Hp, &w));
    x.in = make_proj(m, w, N, Hp);
    if (x.ff > 0) {
        x.in.glu_from = x.c_ff;
        x.in.gp = make_plan(N, Hp, m->es, m->num_sms, 2);
    }
    parts = {{mx + "o", H, 0, 1, 0, x.ow}};
    if (x.ff > 0) parts.push_back({pre + "mlp.down", H, 0, 1, x.owp, x.ff});
    TRY(stack_rows(m, parts, x.ow, Hp, x.owp + x.ffp, &w));
    x.o = make_proj(m, w, Hp, x.owp + x.ffp);
    void* d;
    if (attention) {
        TRY(small_f32(m, mx + "q.norm", HD, HD, &x.q_norm));
        TRY(small_f32(m, mx + "k.norm", kn, kn, &x.k_norm));
        TRY(small_f32(m, mx + "q.b", HD, HD, &x.q_b));
        TRY(small_f32(m, mx + "k.b", kn, kn, &x.k_b));
        TRY(small_f32(m, mx + "v.b", vn, vn, &x.v_b));
        TRY(small_f32(m, mx + "sink", x.heads, x.heads, &x.sink));
        return OXG4_OK;
    }
    TRY(owned_alloc(m, &d, sizeof(float) * x.heads));
    CK(cudaMemcpy(d, s.decay, sizeof(float) * x.heads, cudaMemcpyHostToDevice));
    x.decay = (const float*)d;
    std::vector<float2> freq(std::max(1, x.rot_dims / 2));
    for (int i = 0; i < x.rot_dims / 2; ++i) {
        const double f = std::pow((double)s.rot_base, -2.0 * i / (double)x.rot_dims) / 6.283185307179586476925;   // turns
        freq[i].x = (float)f;
        freq[i].y = (float)(f - (double)freq[i].x);
    }
    TRY(owned_alloc(m, &d, sizeof(float2) * freq.size()));
    CK(cudaMemcpy(d, freq.data(), sizeof(float2) * freq.size(), cudaMemcpyHostToDevice));
    x.freq2 = (const float2*)d;
    return OXG4_OK;
}

static int32_t finalize_mixer(oxg4_model* m, int l, const oxg4_layer_spec& s, MixPlan& x) {
    const std::string pre = "l" + std::to_string(l) + ".", mx = pre + "mix.";
    const int H = m->Hn, Hp = m->H;
    const Tensor* t;
    TRY(small_f32(m, pre + "norm1", H, Hp, &x.norm1, m->norm_offset));
    if (m->parallel) return finalize_parallel(m, pre, s, x);
    TRY(small_f32(m, pre + "norm1b", H, Hp, &x.norm1b, m->norm_offset));
    const int HD = x.heads * x.dim;
    const void* w = nullptr;
    if (x.kind == MIX_WKV) {
        TRY(need(m, mx + "w1", {}, &t));
        if (t->shape.size() != 2) return fail(OXG4_INVALID_SHAPE, "weight `%sw1` has an unexpected shape", mx.c_str());
        x.low_rank = (int)t->shape[0];
        const int sr = pad_to(std::max(HD, x.low_rank), kSegTile), N = 4 * sr + pad_to(x.low_rank, 8);
        TRY(stack_rows(m, {{mx + "r", HD, 0}, {mx + "k", HD, sr}, {mx + "v", HD, 2 * sr}, {mx + "g", HD, 3 * sr},
                           {mx + "w1", x.low_rank, 4 * sr}}, H, N, Hp, &w));
        x.in = make_proj(m, w, N, Hp, 5, sr);
        x.c_q = 0; x.c_k = sr; x.c_v = 2 * sr; x.c_g = 3 * sr; x.c_low = 4 * sr;
        void* mu;
        TRY(owned_alloc(m, &mu, sizeof(float) * 5 * Hp));
        const char* seg[5] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
        for (int i = 0; i < 5; ++i) {
            TRY(need(m, mx + seg[i], {H}, &t));
            CK(cudaMemcpy((float*)mu + (size_t)i * Hp, t->d, sizeof(float) * H, cudaMemcpyDeviceToDevice));
        }
        x.mu = (const float*)mu;
        TRY(need(m, mx + "w2", {HD, x.low_rank}, &t));
        x.w2 = t->d;
        TRY(small_f32(m, mx + "w0", HD, HD, &x.w0));
        TRY(small_f32(m, mx + "u", HD, HD, &x.u));
    } else if (x.kind == MIX_LIGHTNING) {
        x.c_q = 0;
        x.c_k = pad_to(HD, 8);
        x.c_v = x.c_k + pad_to(HD, 8);
        x.c_g = x.c_v + pad_to(x.ow, 8);
        const int N = x.c_g + pad_to(x.ow, 8);
        TRY(stack_rows(m, {{mx + "q", HD, x.c_q}, {mx + "k", HD, x.c_k}, {mx + "v", x.ow, x.c_v}, {mx + "g", x.ow, x.c_g}}, H, N, Hp, &w));
        x.in = make_proj(m, w, N, Hp);
        void* d;
        TRY(owned_alloc(m, &d, sizeof(float) * x.heads));
        CK(cudaMemcpy(d, s.decay, sizeof(float) * x.heads, cudaMemcpyHostToDevice));
        x.decay = (const float*)d;
    } else {
        const int kv = x.rank + x.rot, hq = x.heads * (x.dim + x.rot);
        x.c_dq = 0;
        x.c_dkv = pad_to(x.q_rank, 8);
        x.c_g = x.c_dkv + pad_to(kv, 8);
        const int N = x.c_g + pad_to(x.ow, 8);
        TRY(stack_rows(m, {{mx + "dq", x.q_rank, x.c_dq}, {mx + "dkv", kv, x.c_dkv}, {mx + "g", x.ow, x.c_g}}, H, N, Hp, &w));
        x.in = make_proj(m, w, N, Hp);
        TRY(small_f32(m, mx + "dq.norm", x.q_rank, x.q_rank, &x.dq_norm));
        TRY(small_f32(m, mx + "dkv.norm", x.rank, x.rank, &x.dkv_norm));
        TRY(stack_rows(m, {{mx + "uq", hq, 0}}, x.q_rank, pad_to(hq, 8), x.q_rankp, &w));
        x.uq = make_proj(m, w, pad_to(hq, 8), x.q_rankp);
        TRY(need(m, mx + "uk", {(int64_t)HD, x.rank}, &t));
        x.w_uk = t->d;
        TRY(need(m, mx + "uv", {(int64_t)x.ow, x.rank}, &t));
        x.w_uv = t->d;
        if (m->es == 2) {
            // per-head products on the tensor cores: W_uk^T [heads][rank, dim], W_uv [heads][vdim, rank], padded per head
            const int ur = pad_to(x.rank, kSegTile), ud = pad_to(x.dim, 8), rp = pad_to(x.rank, 8);
            void *ukt, *uvp;
            TRY(owned_alloc(m, &ukt, (size_t)x.heads * ur * ud * 2));
            transpose_heads_kernel<<<m->num_sms * 4, 256>>>((const uint16_t*)x.w_uk, (uint16_t*)ukt, x.heads, x.dim, x.rank, ur, ud);
            CK(cudaGetLastError());
            x.uk = make_proj(m, ukt, x.heads * ur, ud, x.heads, ur);
            x.vpad = pad_to(x.vdim, kSegTile);
            if (x.vpad == x.vdim && rp == x.rank) {
                x.uv = make_proj(m, x.w_uv, x.ow, x.rank, x.heads, x.vdim);
            } else {
                TRY(owned_alloc(m, &uvp, (size_t)x.heads * x.vpad * rp * 2));
                for (int h = 0; h < x.heads; ++h)
                    CK(cudaMemcpy2D((uint16_t*)uvp + (size_t)h * x.vpad * rp, (size_t)rp * 2, (const uint16_t*)x.w_uv + (size_t)h * x.vdim * x.rank,
                                    (size_t)x.rank * 2, (size_t)x.rank * 2, (size_t)x.vdim, cudaMemcpyDeviceToDevice));
                x.uv = make_proj(m, uvp, x.heads * x.vpad, rp, x.heads, x.vpad);
            }
        }
        std::vector<float> inv(std::max(1, x.rot_dims / 2));
        for (int i = 0; i < x.rot_dims / 2; ++i) inv[i] = (float)std::pow((double)s.rot_base, -2.0 * i / (double)x.rot_dims);
        void* d;
        TRY(owned_alloc(m, &d, sizeof(float) * inv.size()));
        CK(cudaMemcpy(d, inv.data(), sizeof(float) * inv.size(), cudaMemcpyHostToDevice));
        x.inv_freq = (const float*)d;
    }
    if (x.kind != MIX_LATENT) TRY(small_f32(m, mx + "norm", x.ow, x.ow, &x.out_norm));
    TRY(stack_rows(m, {{mx + "o", H, 0}}, x.ow, Hp, x.owp, &w));
    x.o = make_proj(m, w, Hp, x.owp);
    if (x.ff > 0) {
        TRY(small_f32(m, pre + "norm2", H, Hp, &x.norm2, m->norm_offset));
        TRY(small_f32(m, pre + "norm2b", H, Hp, &x.norm2b, m->norm_offset));
        TRY(stack_rows(m, {{pre + "mlp.gate", x.ff, 0}}, H, x.ffp, Hp, &w));
        x.gateup = make_proj(m, w, x.ffp, Hp);
        TRY(stack_rows(m, {{pre + "mlp.up", x.ff, 0}}, H, x.ffp, Hp, &x.gateup.w1));
        x.gateup.gp = make_plan(2 * x.ffp, Hp, m->es, m->num_sms, 2);
        TRY(stack_rows(m, {{pre + "mlp.down", H, 0}}, x.ff, Hp, x.ffp, &w));
        x.down = make_proj(m, w, Hp, x.ffp);
    }
    return OXG4_OK;
}

static int32_t finalize_layered(oxg4_model* m) {
    const int L = m->cfg.num_hidden_layers, H = m->Hn, Hp = m->H;
    TRY(stack_rows(m, {{"embed", m->V, 0}}, H, m->V, Hp, &m->embed));
    TRY(stack_rows(m, {{"head", m->V, 0}}, H, m->V, Hp, &m->head));
    TRY(small_f32(m, "final.norm", H, Hp, &m->final_norm, m->norm_offset));
    m->p_lm = make_plan(m->V, Hp, m->es, m->num_sms, 1);
    m->p_lm_simt_grid = std::min(m->num_sms, std::max(1, (m->V + 2 * kSimtWarps - 1) / (2 * kSimtWarps)));
    m->layers.resize(L);
    for (int l = 0; l < L; ++l) {
        const oxg4_layer_spec& s = m->specs[l];
        MixPlan& x = m->layers[l].mix;
        x.kind = s.mixer;
        x.heads = s.heads;
        x.dim = s.dim;
        x.vdim = s.vdim;
        x.ow = s.heads * s.vdim;
        x.owp = pad_to(x.ow, 8);
        x.q_rank = s.q_rank;
        x.q_rankp = pad_to(s.q_rank, 8);
        x.rank = s.kv_rank;
        x.rot = s.rot_dim;
        x.rot_dims = s.rot_dims;
        x.ld = pad_to(s.kv_rank + s.rot_dim, 16);
        if (x.kind == MIX_ATTENTION) {
            x.kv_heads = s.kv_heads;
            x.kd = pad_to(s.dim, 16);
            x.ld = x.kd + pad_to(s.vdim, 16);
            x.temp_coef = s.q_temp_coef;
            x.temp_every = s.q_temp_every;
        }
        x.scale = s.scale;
        x.ff = s.ff;
        x.ffp = pad_to(s.ff, 8);
        m->layers[l].source = l;
        if (s.weights_of < 0) TRY(finalize_mixer(m, l, s, x));
    }
    for (int l = 0; l < L; ++l) {
        int j = l, hops = 0;
        while (m->specs[j].weights_of >= 0 && ++hops <= L) j = m->specs[j].weights_of;
        if (hops > L) return fail(OXG4_INVALID_ARGUMENT, "layer %d: weights_of forms a loop", l);
        if (j == l) continue;
        const oxg4_layer_spec &a = m->specs[l], &b = m->specs[j];
        if (a.mixer != b.mixer || a.heads != b.heads || a.dim != b.dim || a.vdim != b.vdim || a.q_rank != b.q_rank ||
            a.kv_rank != b.kv_rank || a.rot_dim != b.rot_dim || a.ff != b.ff || a.kv_heads != b.kv_heads)
            return fail(OXG4_INVALID_SHAPE, "layer %d uses the tensors of layer %d but differs in size", l, j);
        m->layers[l].mix = m->layers[j].mix;
    }
    return OXG4_OK;
}

// ---- cache table ----------------------------------------------------------------------------------------------
// K-splits of a tcgen05 projection for R rows: as in the Gemma 4 path (few extra bytes for a decode step, more for the 256
// rows of a chunk)
static int layered_splits(const oxg4_model* m, const Proj& p, int R, bool chunk) {
    const int n = p.N * (p.w1 ? 2 : 1), tiles = (p.N + kTcTileM - 1) / kTcTileM * (p.w1 ? 2 : 1);
    return tc_pick_splits(tiles, (p.K + kTcTileK - 1) / kTcTileK, m->num_sms, chunk ? kPrefillRows : R, n, p.K, chunk ? 1.0 : 0.3);
}

static int32_t latent_mma_setup(const MixPlan& x);
static int32_t head_attn_setup(const MixPlan& x);
constexpr int kLatentChunkSplits = 4;     // most splits of the visible positions in a prompt chunk

static int32_t layered_cache_build(oxg4_cache* c, int pages_full) {
    oxg4_model* m = c->m;
    const int B = c->B, L = m->cfg.num_hidden_layers, H = m->H, R = c->rows_cap;
    const bool tc = c->tc_ok;
    const size_t kes = c->kv_dtype == OXG4_BF16 ? 2 : 4, xes = tc ? 2 : 4;
    c->state.assign(L, nullptr);
    c->shift.assign(L, nullptr);
    auto floats = [&](const Proj& p) {       // of a projection's output, K-split partials included
        const size_t n = (size_t)p.N * (p.w1 ? 2 : 1);
        if (!tc) return (size_t)R * n;
        return n * std::max((size_t)layered_splits(m, p, B, false) * B, (size_t)layered_splits(m, p, kPrefillRows, true) * kPrefillRows);
    };
    size_t in_n = 1, o_n = 1, gu_n = 1, down_n = 1, q_n = 1, uk_n = 1, uv_n = 1, dec = 1, latq = 1, rh = 1, rh_rank = 1, xo = 1, xi = 1, xq = 1,
           xu = 1, xl = 1, rot = 1, act = 1, block_n = 1;
    bool any_shift = false;
    const int max_tiles = (*std::max_element(c->max_seq.begin(), c->max_seq.end()) + kLmTile - 1) / kLmTile;
    c->lat_splits = std::max(2, std::min({max_tiles, 64, (4 * m->num_sms + B - 1) / B}));
    for (int l = 0; l < L; ++l) {
        const MixPlan& x = m->layers[l].mix;
        in_n = std::max(in_n, floats(x.in));
        o_n = std::max(o_n, floats(x.o));
        xo = std::max(xo, (size_t)x.o.K);
        act = std::max(act, (size_t)x.owp);
        if (x.ff > 0 && !m->parallel) {
            gu_n = std::max(gu_n, floats(x.gateup));
            down_n = std::max(down_n, floats(x.down));
            xi = std::max(xi, (size_t)x.ffp);
        }
        if (x.kind == MIX_LATENT) {
            uint8_t* pool;
            const size_t bytes = (size_t)pages_full * c->PT * x.ld * kes;
            TRY(dalloc(c, &pool, bytes));
            c->kpool[l] = pool;
            c->pool_bytes[l] = bytes;
            c->kv_bytes += (int64_t)bytes;
            q_n = std::max(q_n, floats(x.uq));
            xq = std::max(xq, (size_t)x.q_rankp);
            latq = std::max(latq, (size_t)x.heads * (x.rank + x.rot));
            rh = std::max(rh, (size_t)x.heads);
            rh_rank = std::max(rh_rank, (size_t)x.heads * x.rank);
            if (tc) {
                uk_n = std::max(uk_n, (size_t)R * x.uk.N);
                uv_n = std::max(uv_n, floats(x.uv));
                xu = std::max(xu, (size_t)x.heads * x.uk.K);
                xl = std::max(xl, (size_t)x.heads * x.uv.K);
                rot = std::max(rot, (size_t)x.heads * x.rot);
                TRY(latent_mma_setup(x));
            }
        } else if (x.kind == MIX_ATTENTION) {
            uint8_t* pool;
            const size_t bytes = (size_t)pages_full * x.kv_heads * c->PT * x.ld * kes;
            TRY(dalloc(c, &pool, bytes));
            c->kpool[l] = pool;
            c->pool_bytes[l] = bytes;
            c->kv_bytes += (int64_t)bytes;
            xu = std::max(xu, (size_t)x.heads * x.kd);
            latq = std::max(latq, (size_t)x.heads * x.dim);
            rh = std::max(rh, (size_t)x.heads);
            rh_rank = std::max(rh_rank, (size_t)x.ow);
            TRY(head_attn_setup(x));
        } else {
            const size_t n = (size_t)B * x.heads * x.dim * x.vdim;
            TRY(dalloc(c, &c->state[l], n));
            c->kv_bytes += (int64_t)(4 * n);
            if (x.kind != MIX_WKV) {
                block_n = std::max(block_n, (size_t)x.heads * x.dim * x.vdim);
                latq = std::max(latq, (size_t)x.heads * x.dim);
            }
            if (x.kind == MIX_WKV) {
                TRY(dalloc(c, &c->shift[l], (size_t)B * H));
                c->kv_bytes += (int64_t)(4 * (size_t)B * H);
                any_shift = true;
                dec = std::max(dec, (size_t)x.heads * x.dim);
            }
        }
        ++c->physical_caches;
    }
    auto bytes_alloc = [&](void** p, size_t bytes) {
        uint8_t* d = nullptr;
        const int32_t s = dalloc(c, &d, bytes);
        *p = d;
        return s;
    };
    TRY(dalloc(c, &c->in_buf, in_n));
    TRY(dalloc(c, &c->o_part, o_n));
    TRY(dalloc(c, &c->gu_part, gu_n));
    TRY(dalloc(c, &c->down_part, down_n));
    TRY(dalloc(c, &c->attn_out, (size_t)R * act));
    TRY(bytes_alloc(&c->mix_x, (size_t)R * H * xes * (any_shift ? 5 : 1)));
    TRY(bytes_alloc(&c->mix_y, (size_t)R * std::max(xo, xi) * xes));
    if (tc) TRY(dalloc(c, &c->x_h, (size_t)R * H));
    if (any_shift) {
        TRY(dalloc(c, &c->xf, (size_t)R * H));
        TRY(dalloc(c, &c->wdec, (size_t)R * dec));
    }
    TRY(dalloc(c, &c->block_state, 2 * (kPrefillRows / kRecBlock) * block_n));
    TRY(dalloc(c, &c->q_buf, q_n));
    TRY(bytes_alloc(&c->x_q, (size_t)R * xq * xes));
    TRY(dalloc(c, &c->lat_q, (size_t)R * latq));
    TRY(dalloc(c, &c->lat_rot, (size_t)R * rot));
    TRY(dalloc(c, &c->uk_buf, uk_n));
    TRY(dalloc(c, &c->uv_buf, uv_n));
    TRY(bytes_alloc(&c->x_u, (size_t)R * xu * 2));
    TRY(bytes_alloc(&c->x_l, (size_t)R * xl * 2));
    const size_t part_rows = std::max((size_t)B * c->lat_splits, (size_t)R * kLatentChunkSplits);
    TRY(dalloc(c, &c->lat_o, part_rows * rh_rank));
    TRY(dalloc(c, &c->lat_ml, part_rows * rh * 2));
    return OXG4_OK;
}

// ---- a pass over the layers -----------------------------------------------------------------------------------
static_assert(kRecMaxBlocks * kRecBlock == kPrefillRows, "blocks of a pass");
typedef void (*RecurFn)(const RecurArgs);
// lanes along the key channels and channels per lane for heads of `dim`
static void recur_shape(int dim, int* ks, int* kpt) {
    *kpt = dim <= 64 ? 8 : 16;
    *ks = dim <= 32 ? 4 : dim <= 128 ? 8 : dim <= 256 ? 16 : 32;
}
// step: decode step
template <int KIND, typename WT>
static RecurFn pick_recur(int ks, int kpt, bool step) {
#define PR(KS, KPT)                                                                          \
    if (ks == KS && kpt == KPT) {                                                            \
        if (step) return recur_kernel<KIND, WT, KS, KPT, 1>;                                 \
        if constexpr (KIND == REC_WKV) return recur_kernel<KIND, WT, KS, KPT, rec_tile(KS * KPT)>; \
        else return fixed_recur_kernel<KIND, KS, KPT>;                                       \
    }
    PR(4, 8) PR(8, 8) PR(8, 16) PR(16, 16) PR(32, 16)
#undef PR
    return nullptr;
}

static int32_t group_norm_setup() {
    TRY((allow_big_smem(group_norm_rows_kernel<uint16_t, 1>)));
    TRY((allow_big_smem(group_norm_rows_kernel<uint16_t, 4>)));
    TRY((allow_big_smem(group_norm_rows_kernel<float, 1>)));
    return allow_big_smem(group_norm_rows_kernel<float, 4>);
}

typedef void (*RowAttnFn)(const RowAttnArgs);
template <typename KT, bool LATENT>
static RowAttnFn pick_row_attn(int vw) {
    if (vw <= 128) return row_attn_kernel<KT, 4, LATENT>;
    if (vw <= 256) return row_attn_kernel<KT, 8, LATENT>;
    return row_attn_kernel<KT, 16, LATENT>;
}
static size_t row_attn_smem(int dk, int vw) { return sizeof(float) * ((size_t)dk + 8 * vw + 16); }

typedef void (*LatentMmaFn)(const LatentMmaArgs);
// the tensor-core kernel for `rows` (token, head) rows per run and cache rows of `ld` elements, null when it does not fit
static LatentMmaFn pick_latent_mma(int rank, int ld, int rows, int* tile_rows, int* groups, size_t* smem) {
    LatentMmaFn fn;
#define LM(MT, NST, GR)                                                                                         \
    {                                                                                                           \
        fn = rank <= 128 ? latent_mma_kernel<MT, 2, NST, GR> : rank <= 256 ? latent_mma_kernel<MT, 4, NST, GR> : latent_mma_kernel<MT, 8, NST, GR>; \
        *tile_rows = MT * 16;                                                                                   \
        *groups = GR;                                                                                           \
        *smem = latent_mma_smem<MT, NST, GR>(ld);                                                               \
    }
    const size_t limit = 226 * 1024;
    if (rows <= 16) {
        LM(1, 2, 2)
        if (*smem > limit) LM(1, 2, 1)
    } else if (rows <= 32) {
        LM(2, 2, 2)
        if (*smem > limit) LM(2, 2, 1)
    } else {
        LM(4, 3, 1)
        if (*smem > limit) LM(4, 2, 1)
    }
#undef LM
    return *smem <= limit ? fn : nullptr;
}

static int32_t latent_mma_setup(const MixPlan& x) {
    for (int rows : {16, 32, 64}) {
        int tr, gr;
        size_t smem;
        LatentMmaFn fn = pick_latent_mma(x.rank, x.ld, rows, &tr, &gr, &smem);
        if (fn) TRY(allow_big_smem(fn));
    }
    return OXG4_OK;
}

// Attention over [key | value] rows: the tensor-core kernel for `rows` (token, head) rows per run and kv head, null when the
// heads are too wide for it
typedef void (*HeadMmaFn)(const HeadMmaArgs);
static HeadMmaFn pick_head_mma(const MixPlan& x, int rows, int* tile_rows, size_t* smem) {
    const int vd = x.ld - x.kd, cols = std::max(x.kd, vd) <= 64 ? 64 : std::max(x.kd, vd) <= 128 ? 128 : 256, wr = rows <= 16 ? 1 : 4;
    if (std::max(x.kd, vd) > 256) return nullptr;
    *tile_rows = 16 * wr;
    *smem = head_mma_smem(cols, wr, x.ld, x.kd, vd);
    if (wr == 1) return cols == 64 ? head_mma_kernel<64, 1> : cols == 128 ? head_mma_kernel<128, 1> : head_mma_kernel<256, 1>;
    return cols == 64 ? head_mma_kernel<64, 4> : cols == 128 ? head_mma_kernel<128, 4> : head_mma_kernel<256, 4>;
}

static int32_t head_attn_setup(const MixPlan& x) {
    for (int rows : {16, 64}) {
        int tr;
        size_t smem;
        HeadMmaFn fn = pick_head_mma(x, rows, &tr, &smem);
        if (fn) TRY(allow_big_smem(fn));
    }
    for (auto fn : {head_prep_kernel<uint16_t, uint16_t, 1>, head_prep_kernel<uint16_t, uint16_t, 4>}) TRY(allow_big_smem(fn));
    for (auto fn : {head_prep_kernel<float, uint16_t, 1>, head_prep_kernel<float, uint16_t, 4>}) TRY(allow_big_smem(fn));
    for (auto fn : {head_prep_kernel<float, float, 1>, head_prep_kernel<float, float, 4>}) TRY(allow_big_smem(fn));
    return OXG4_OK;
}

// Splits of `tiles` cache tiles when `units` row tiles share the GPU: the cheapest number of rounds times tiles per CTA, with
// about four tiles' worth of start-up per CTA and a little for every partial the merge has to read.
static int latent_splits(int units, int tiles, int most, int num_sms) {
    int best = 1;
    double best_cost = 1e30;
    for (int s = 1; s <= std::min(most, std::max(1, tiles)); ++s) {
        const double rounds = (units * s + num_sms - 1) / num_sms;
        const double cost = rounds * ((tiles + s - 1) / s + 4) + 0.1 * s;
        if (cost < best_cost - 1e-9) { best_cost = cost; best = s; }
    }
    return best;
}

namespace {

struct LayeredPass {
    oxg4_cache* c;
    Launcher& ln;
    const RowSet& rs;
    const bool tc;                       // BF16 projections on the tensor cores
    const bool fused;                    // one row: prologues carry the row kernels' work
    const TraceCtx* tr;
    oxg4_model* m = c->m;
    const int R = rs.R, H = m->H;
    const float eps = m->cfg.rms_norm_eps;
    float* cur = nullptr;                // residual stream before the pending update (null: the embedding rows)
    float* nxt = c->hA;
    Pending pd;

    RunRows runs() const { return RunRows{rs.run_row0, rs.run_n, rs.pos, rs.seq, rs.tok}; }

    void advance() {                     // the residual stream with its update closed is in nxt from now on
        cur = nxt;
        nxt = cur == c->hA ? c->hB : c->hA;
        pd = Pending{};
    }
    void pend(const SplitIn& raw, const float* w_post) {
        pd.raw = raw.p;
        pd.splits = raw.splits;
        pd.w_post = w_post;
    }
    void residual_args(GemvArgs& a, const float* w_norm) {
        a.h_out = nxt;
        a.w_norm = w_norm;
        a.scalar = 1.0f;
        if (cur == nullptr) {
            a.embed = m->embed;
            a.tokens = rs.tok;
            a.embed_scale = 1.0f;
        } else {
            a.h_in = cur;
            a.raw = pd.raw;
            a.w_post = pd.w_post;
        }
    }
    // what an output projection of the parallel block reads behind the mixer's columns; in: fused input projection
    OutTail ff_tail(const MixPlan& x, const SplitIn& in) const {
        OutTail t{};
        t.in = in;
        t.col = x.c_ff;
        t.n = m->parallel ? x.ffp : 0;
        t.at = x.owp;
        t.act = tc ? m->ff_act : ACT_NONE;
        return t;
    }
    // row kernels: close the pending update, norm; x and / or x_f32 may be null
    void close_rows(const float* w_norm, void* x, float* x_f32) {
        RowsNormArgs n{};
        n.B = R; n.H = H; n.norm_n = m->Hn;
        n.h_in = cur; n.h_out = nxt;
        n.raw = pd.raw; n.raw_splits = pd.splits;
        n.w_post = pd.w_post;
        n.scalar = 1.0f;
        n.w_norm = w_norm;
        n.eps = eps;
        n.x = x;
        n.x_f32 = x_f32;
        if (cur == nullptr) {
            n.embed = m->embed;
            n.tokens = rs.tok;
            n.embed_scale = 1.0f;
        }
        if (m->es == 2) ln.go("norm", rows_norm_kernel<uint16_t>, dim3(R), dim3(kRowsThreads), 0, n);
        else ln.go("norm", rows_norm_kernel<float>, dim3(R), dim3(kRowsThreads), 0, n);
        advance();
    }
    // out = x . W^T for all rows; x holds the projection's operand type
    SplitIn project(const char* kind, const Proj& p, const void* x, float* out) {
        const int n = p.N * (p.w1 ? 2 : 1);
        if (tc) {
            const int S = layered_splits(m, p, R, rs.chunk);
            ln.tc(kind, c, R, p.w, p.w1, (const uint16_t*)x, p.N, p.K, S, out, n, 0, p.nseg > 1 ? p.seg_rows / kTcTileM : 0);
            return SplitIn{out, S, (size_t)R * n, n};
        }
        GemvArgs a{};
        a.W0 = p.w;
        a.in = (const float*)x;
        a.out = out;
        if (p.glu_from >= 0) {
            a.glu_from = p.glu_from;
            a.act = m->ff_act;
            launch_gemv(ln, kind, c, R, a, p.gp, PRO_PLAIN, EPI_STORE_GLU);
            return one(out, (p.glu_from + p.N) / 2);
        }
        if (p.nseg > 1) { a.nseg = p.nseg; a.seg_rows = p.seg_rows; }
        launch_gemv(ln, kind, c, R, a, p.gp, PRO_PLAIN, EPI_STORE);
        return SplitIn{out, 1, 0, n};
    }
    SplitIn one(float* out, int n) const { return SplitIn{out, 1, 0, n}; }

    void group_norm(const GroupNormArgs& g, const OutTail& tail, void* x, int ld_x) {
        const size_t smem = sizeof(float) * g.n;
        const dim3 grid(R, 1 + tail.slices());
        if (ln.status == OXG4_OK && smem > 48 * 1024) ln.status = group_norm_setup();
        const bool vec = (g.n | g.n_pad | g.hs | g.hs_ld | g.o.ld | g.gate.ld | g.c_gate | ld_x) % 4 == 0 && (g.o.stride | g.gate.stride) % 4 == 0;
        if (m->es == 2) {
            if (vec) ln.go("outnorm", group_norm_rows_kernel<uint16_t, 4>, grid, dim3(256), smem, g, tail, (uint16_t*)x, ld_x);
            else ln.go("outnorm", group_norm_rows_kernel<uint16_t, 1>, grid, dim3(256), smem, g, tail, (uint16_t*)x, ld_x);
        } else {
            if (vec) ln.go("outnorm", group_norm_rows_kernel<float, 4>, grid, dim3(256), smem, g, tail, (float*)x, ld_x);
            else ln.go("outnorm", group_norm_rows_kernel<float, 1>, grid, dim3(256), smem, g, tail, (float*)x, ld_x);
        }
    }

    // output norm, gate and output projection of a mixer; o: raw head outputs
    void output(const MixPlan& x, const SplitIn& o, int hs_ld, int group, const float* w, const SplitIn& gate, int act) {
        if (fused) {
            GemvArgs a{};
            a.W0 = x.o.w;
            a.in = o.p;
            a.gn_n = x.ow;
            a.gn_group = group;
            a.gn_w = w;
            a.gn_gate = act == ACT_NONE ? nullptr : gate.p + x.c_g;
            a.act = act;
            if (m->parallel && x.ff > 0) {
                a.gn_tail = gate.p + x.c_ff;
                a.gn_tail_n = x.ffp;
                a.gn_tail_at = x.owp;
            }
            a.out = c->o_part;
            launch_gemv(ln, "o", c, R, a, x.o.gp, PRO_GNORM, EPI_STORE);
            pend(one(c->o_part, H), x.norm1b);
            return;
        }
        GroupNormArgs g{};
        g.o = o;
        g.hs = x.vdim;
        g.hs_ld = hs_ld;
        g.n = x.ow;
        g.n_pad = x.owp;
        g.group = group;
        g.w = w;
        g.gate = gate;
        g.c_gate = x.c_g;
        g.act = act;
        g.eps = eps;
        group_norm(g, ff_tail(x, gate), c->mix_y, x.o.K);
        pend(project("o", x.o, c->mix_y, c->o_part), x.norm1b);
    }

    // norm1 (closing what is pending) and the fused input projection
    SplitIn input(const MixPlan& x, int l) {
        const bool shift = x.kind == MIX_WKV;
        SplitIn in;
        if (fused) {
            GemvArgs a{};
            a.W0 = x.in.w;
            residual_args(a, x.norm1);
            a.out = c->in_buf;
            if (shift) {
                a.nseg = x.in.nseg;
                a.seg_rows = x.in.seg_rows;
                a.mu = x.mu;
                a.shift_state = c->shift[l];
                a.pos = rs.pos;
                a.x_f32 = c->xf;
            }
            if (x.in.glu_from >= 0) {
                a.glu_from = x.in.glu_from;
                a.act = m->ff_act;
            }
            launch_gemv(ln, "qkv", c, R, a, x.in.gp, shift ? PRO_SHIFT : PRO_NORM, x.in.glu_from >= 0 ? EPI_STORE_GLU : EPI_STORE);
            advance();
            in = one(c->in_buf, x.in.glu_from >= 0 ? (x.in.glu_from + x.in.N) / 2 : x.in.N);
        } else {
            close_rows(x.norm1, shift ? nullptr : c->mix_x, shift ? c->xf : nullptr);
            if (shift) {
                if (m->es == 2)
                    ln.go("shift", shift_mix_kernel<uint16_t>, dim3(R), dim3(256), 0, R, H, 5, (const float*)c->xf, (const float*)c->shift[l], x.mu,
                          runs(), (uint16_t*)c->mix_x);
                else
                    ln.go("shift", shift_mix_kernel<float>, dim3(R), dim3(256), 0, R, H, 5, (const float*)c->xf, (const float*)c->shift[l], x.mu,
                          runs(), (float*)c->mix_x);
            }
            in = project("qkv", x.in, c->mix_x, c->in_buf);
        }
        if (tr && ln.status == OXG4_OK &&
            cudaMemcpyAsync(tr->trace_dev + (size_t)l * R * H, cur, sizeof(float) * R * H, cudaMemcpyDeviceToDevice, m->stream) != cudaSuccess)
            ln.status = fail(OXG4_CUDA, "Gemma 4 CUDA error: trace copy failed");
        return in;
    }

    void recurrent(const MixPlan& x, int l, const SplitIn& in) {
        RecurArgs a{};
        a.in = in;
        a.c_q = x.c_q; a.c_k = x.c_k; a.c_v = x.c_v;
        a.heads = x.heads; a.dim = x.dim; a.vdim = x.vdim;
        a.state = c->state[l];
        a.rows = runs();
        a.out = c->attn_out;
        a.ld_out = x.owp;
        const bool wkv = x.kind == MIX_WKV, ret = x.kind == MIX_RETENTION;
        if (wkv) {
            a.u = x.u;
            a.c_low = x.c_low; a.rank = x.low_rank; a.w2 = x.w2; a.w0 = x.w0;
            a.shift_src = c->xf; a.shift_dst = c->shift[l]; a.shift_n = H;
            if (!fused) {
                const int N = x.heads * x.dim;
                const dim3 grid((N + 255) / 256, (R + kDecayRows - 1) / kDecayRows);
                const size_t smem = sizeof(float) * kDecayRows * x.low_rank;
                if (m->es == 2)
                    ln.go("decay", wkv_decay_kernel<uint16_t>, grid, dim3(256), smem, R, N, x.low_rank, in, x.c_low, (const uint16_t*)x.w2, x.w0, c->wdec);
                else
                    ln.go("decay", wkv_decay_kernel<float>, grid, dim3(256), smem, R, N, x.low_rank, in, x.c_low, (const float*)x.w2, x.w0, c->wdec);
                a.w = c->wdec;
            }
        } else {
            a.decay = x.decay;
            a.freq = x.freq2;
            a.rot_dims = x.rot_dims;
            a.k_scale = 1.0f / sqrtf((float)x.dim);
        }
        int ks, kpt;
        recur_shape(x.dim, &ks, &kpt);
        RecurFn fn;
        const bool step = !rs.chunk;
        if (wkv) fn = m->es == 2 ? pick_recur<REC_WKV, uint16_t>(ks, kpt, step) : pick_recur<REC_WKV, float>(ks, kpt, step);
        else fn = ret ? pick_recur<REC_RETENTION, float>(ks, kpt, step) : pick_recur<REC_LIGHTNING, float>(ks, kpt, step);
        const int vs = kRecThreads / ks * kRecCols, dp = ks * kpt, tile = step ? 1 : rec_tile(dp);
        size_t smem = sizeof(float) * ((step ? 1 : 2) * ((size_t)tile * dp * (wkv ? 3 : 2) + tile * vs + pad_to(tile, 4)) + (wkv ? dp + x.low_rank : 0));
        int parts = (int)rs.run_len.size();
        bool join = false;
        if (!step && !wkv) {               // blocks of the runs, joined where a run has several
            smem = fixed_recur_smem(ks, kpt);
            parts = 0;
            for (int n : rs.run_len) {
                parts += (n + kRecBlock - 1) / kRecBlock;
                join |= n > kRecBlock;
            }
            a.runs = (int)rs.run_len.size();
            a.block_state = c->block_state;
            a.block_q = c->lat_q;
        }
        if (ln.status == OXG4_OK && smem > 48 * 1024) ln.status = allow_big_smem(fn);
        ln.go("recur", fn, dim3(x.heads, (x.vdim + vs - 1) / vs, (unsigned)parts), dim3(kRecThreads), smem, a);
        if (join) {
            if (ln.status == OXG4_OK && join_smem(x.dim) > 48 * 1024) ln.status = allow_big_smem(recur_join_kernel);
            ln.go("recjoin", recur_join_kernel, dim3(x.heads, (x.vdim + kJoinCols - 1) / kJoinCols, (unsigned)parts), dim3(kJoinThreads), join_smem(x.dim), a);
        }
        if (ret) output(x, one(c->attn_out, x.owp), x.vdim, x.vdim, nullptr, in, ACT_SILU);
        else output(x, one(c->attn_out, x.owp), x.vdim, wkv ? x.dim : x.ow, x.out_norm, in, wkv ? ACT_SILU : ACT_SIGMOID);
    }

    LatentArgs latent_args(const MixPlan& x, int l, const SplitIn& in) const {
        LatentArgs a{};
        a.in = in;
        a.c_dq = x.c_dq; a.c_dkv = x.c_dkv;
        a.heads = x.heads; a.dim = x.dim; a.rot = x.rot; a.rot_dims = x.rot_dims; a.vdim = x.vdim;
        a.rank = x.rank; a.q_rank = x.q_rank;
        a.dq_norm = x.dq_norm; a.dkv_norm = x.dkv_norm; a.inv_freq = x.inv_freq;
        a.eps = eps;
        a.scale = x.scale;
        a.rows = runs();
        a.cache = RowCache{c->kpool[l], c->pt_full, c->pps_full, c->PT, x.ld, 1};
        return a;
    }

    template <typename WT, typename KT>
    void latent(const MixPlan& x, int l, const SplitIn& in) {
        const LatentArgs a = latent_args(x, l, in);
        SplitIn q;
        if (fused) {
            GemvArgs g{};
            g.W0 = x.uq.w;
            g.in = in.p + x.c_dq;
            g.gn_n = g.gn_group = x.q_rank;
            g.gn_w = x.dq_norm;
            g.out = c->q_buf;
            launch_gemv(ln, "uq", c, R, g, x.uq.gp, PRO_GNORM, EPI_STORE);
            q = one(c->q_buf, x.uq.N);
        } else {
            ln.go("latent", latent_prep_kernel<WT, KT>, dim3(R), dim3(256), 0, a, (WT*)c->x_q, x.q_rankp);
            q = project("uq", x.uq, c->x_q, c->q_buf);
        }
        AttnPart part{c->lat_o, c->lat_ml, rs.chunk ? 1 : c->lat_splits, (size_t)R * x.heads};
        int tile_rows = 0, groups = 1;
        size_t mma_smem = 0;
        int longest = 1;
        for (int n : rs.run_len) longest = std::max(longest, n);
        const LatentMmaFn mma = sizeof(WT) == 2 && sizeof(KT) == 2 ? pick_latent_mma(x.rank, x.ld, longest * x.heads, &tile_rows, &groups, &mma_smem) : nullptr;
        LatentMmaArgs ma{};
        int mma_tiles = 0;
        if (mma) {
            for (int n : rs.run_len) mma_tiles += (n * x.heads + tile_rows - 1) / tile_rows;
            const int most = rs.chunk ? kLatentChunkSplits : c->lat_splits, visible_tiles = (rs.max_visible + kLmTile - 1) / kLmTile;
            part.splits = groups * latent_splits(mma_tiles, (visible_tiles + groups - 1) / groups, std::max(1, most / groups), m->num_sms);
            ma.heads = x.heads; ma.rank = x.rank; ma.rot = x.rot;
            ma.scale = x.scale;
            ma.rows = a.rows;
            ma.runs = (int)rs.run_len.size();
            ma.step_tiles = rs.chunk ? 0 : (x.heads + tile_rows - 1) / tile_rows;
            ma.cache = a.cache;
            ma.part = part;
        }
        if (mma && tc) {
            // many rows: per-head products with W_uk^T and W_uv on the tensor cores
            ln.go("latsplit", latent_split_query_kernel, dim3(R), dim3(256), 0, a, R, q, (uint16_t*)c->x_u, x.uk.K, c->lat_rot);
            ln.tc("uk", c, R, x.uk.w, nullptr, (const uint16_t*)c->x_u, x.uk.N, x.uk.K, 1, c->uk_buf, x.uk.N, 0, x.uk.seg_rows / kTcTileM);
            ma.q_abs = c->uk_buf; ma.abs_row = x.uk.N; ma.abs_head = x.uk.seg_rows;
            ma.q_rot = c->lat_rot; ma.rot_row = (size_t)x.heads * x.rot; ma.rot_head = x.rot;
            ln.go("attn", mma, dim3(mma_tiles, part.splits / groups), dim3(kLmThreads * groups), mma_smem, ma);
            ln.go("latmerge", latent_merge_kernel, dim3(x.heads, R), dim3(128), sizeof(float) * part.splits, R, x.heads, x.rank, part,
                  (uint16_t*)c->x_l, x.uv.K);
            const SplitIn o = project("uv", x.uv, c->x_l, c->uv_buf);
            output(x, o, x.vpad, 0, nullptr, in, ACT_SIGMOID);
            return;
        }
        ln.go("latq", latent_query_kernel<WT, KT>, dim3(x.heads + (fused ? 1 : 0), R, (x.rank + kLqCols - 1) / kLqCols), dim3(256),
              sizeof(float) * (x.dim + x.rot + 256), a, q, (const WT*)x.w_uk, c->lat_q, (int)fused);
        if (mma) {
            ma.q_abs = c->lat_q; ma.abs_row = (size_t)x.heads * (x.rank + x.rot); ma.abs_head = x.rank + x.rot;
            ma.q_rot = c->lat_q + x.rank; ma.rot_row = ma.abs_row; ma.rot_head = ma.abs_head;
            ln.go("attn", mma, dim3(mma_tiles, part.splits / groups), dim3(kLmThreads * groups), mma_smem, ma);
        } else {
            const RowAttnArgs ra{c->lat_q, x.heads, x.heads, x.rank + x.rot, 0, x.rank, x.scale, a.rows, a.cache, part};
            ln.go("attn", pick_row_attn<KT, true>(x.rank), dim3(x.heads, R, part.splits), dim3(256), row_attn_smem(ra.dk, ra.vw), ra);
        }
        ln.go("latout", latent_out_kernel<WT>, dim3(x.heads, R, (x.vdim + 31) / 32), dim3(256), sizeof(float) * (pad_to(x.rank, 4) + part.splits), x.heads,
              x.rank, x.vdim, part, (const WT*)x.w_uv, x.rank, in, x.c_g, rs.tok, c->attn_out, x.owp);
        // the gate has been applied by the kernel that leaves latent space
        output(x, one(c->attn_out, x.owp), x.vdim, 0, nullptr, in, ACT_NONE);
    }

    // grouped-query attention with whole-projection norms and a sink
    template <typename WT, typename KT>
    void attention(const MixPlan& x, int l, const SplitIn& in) {
        HeadAttnArgs a{};
        a.in = in;
        a.c_q = x.c_q; a.c_k = x.c_k; a.c_v = x.c_v;
        a.heads = x.heads; a.kv_heads = x.kv_heads; a.dim = x.dim; a.vdim = x.vdim; a.kd = x.kd;
        a.q_b = x.q_b; a.k_b = x.k_b; a.v_b = x.v_b; a.q_norm = x.q_norm; a.k_norm = x.k_norm;
        a.eps = eps;
        a.temp_coef = x.temp_coef;
        a.temp_every = x.temp_every;
        a.rows = runs();
        a.cache = RowCache{c->kpool[l], c->pt_full, c->pps_full, c->PT, x.ld, x.kv_heads};
        const int group = x.heads / x.kv_heads;
        AttnPart part{c->lat_o, c->lat_ml, rs.chunk ? 1 : c->lat_splits, (size_t)R * x.heads};
        int longest = 1, tile_rows = 0;
        for (int n : rs.run_len) longest = std::max(longest, n);
        size_t mma_smem = 0;
        const HeadMmaFn mma = sizeof(WT) == 2 && sizeof(KT) == 2 ? pick_head_mma(x, longest * group, &tile_rows, &mma_smem) : nullptr;
        const size_t prep_smem = sizeof(float) * x.heads * x.dim;
        const bool vec = x.dim % 4 == 0 && x.vdim % 4 == 0;
        const dim3 prep_block(R <= m->num_sms ? 1024 : 256);
        if (mma) {
            ln.go("qkv_post", vec ? head_prep_kernel<uint16_t, uint16_t, 4> : head_prep_kernel<uint16_t, uint16_t, 1>, dim3(R, 3), prep_block, prep_smem, a,
                  (uint16_t*)c->x_u, x.kd);
            int units = 0;
            for (int n : rs.run_len) units += (n * group + tile_rows - 1) / tile_rows;
            const int most = rs.chunk ? kLatentChunkSplits : c->lat_splits;
            part.splits = latent_splits(units * x.kv_heads, (rs.max_visible + kHmTile - 1) / kHmTile, most, 2 * m->num_sms);
            HeadMmaArgs h{};
            h.q = (const uint16_t*)c->x_u;
            h.heads = x.heads; h.group = group; h.kd = x.kd; h.vd = x.ld - x.kd; h.vdim = x.vdim;
            h.scale = x.scale;
            h.rows = a.rows;
            h.runs = (int)rs.run_len.size();
            h.step_tiles = rs.chunk ? 0 : (group + tile_rows - 1) / tile_rows;
            h.cache = a.cache;
            h.part = part;
            ln.go("attn", mma, dim3(units, x.kv_heads, part.splits), dim3(kHmThreads), mma_smem, h);
        } else {
            ln.go("qkv_post", vec ? head_prep_kernel<float, KT, 4> : head_prep_kernel<float, KT, 1>, dim3(R, 3), prep_block, prep_smem, a, c->lat_q, x.dim);
            const RowAttnArgs ra{c->lat_q, x.heads, group, x.dim, x.kd, x.vdim, x.scale, a.rows, a.cache, part};
            ln.go("attn", pick_row_attn<KT, false>(x.vdim), dim3(x.heads, R, part.splits), dim3(256), row_attn_smem(ra.dk, ra.vw), ra);
        }
        const size_t smem = sizeof(float) * part.splits;
        if (fused) {
            ln.go("attn_merge", head_merge_kernel<float>, dim3(x.heads, R), dim3(128), smem, x.heads, x.vdim, part, x.sink, OutTail{}, c->attn_out, x.owp);
            output(x, one(c->attn_out, x.owp), x.vdim, 0, nullptr, in, ACT_NONE);
            return;
        }
        const OutTail tail = ff_tail(x, in);
        const dim3 grid(x.heads + tail.slices(), R);
        if (tc) ln.go("attn_merge", head_merge_kernel<uint16_t>, grid, dim3(128), smem, x.heads, x.vdim, part, x.sink, tail, (uint16_t*)c->mix_y, x.o.K);
        else ln.go("attn_merge", head_merge_kernel<float>, grid, dim3(128), smem, x.heads, x.vdim, part, x.sink, tail, (float*)c->mix_y, x.o.K);
        pend(project("o", x.o, c->mix_y, c->o_part), nullptr);
    }

    template <typename WT, typename KT>
    void attend(const MixPlan& x, int l, const SplitIn& in) {
        if (x.kind == MIX_LATENT) latent<WT, KT>(x, l, in);
        else attention<WT, KT>(x, l, in);
    }

    void feed_forward(const MixPlan& x) {
        if (!tc) {
            GemvArgs a{};
            a.W0 = x.gateup.w;
            a.W1 = x.gateup.w1;
            residual_args(a, x.norm2);
            a.act = m->ff_act;
            a.out = c->gu_part;
            launch_gemv(ln, "gateup", c, R, a, x.gateup.gp, PRO_NORM, EPI_GATEUP);
            advance();
            GemvArgs d{};
            d.W0 = x.down.w;
            d.in = c->gu_part;
            d.out = c->down_part;
            launch_gemv(ln, "down", c, R, d, x.down.gp, PRO_PLAIN, EPI_STORE);
            pend(one(c->down_part, H), x.norm2b);
            return;
        }
        close_rows(x.norm2, c->mix_x, nullptr);
        const SplitIn gu = project("gateup", x.gateup, c->mix_x, c->gu_part);
        ln.go("geglu", geglu_rows_kernel, dim3((x.ffp / 4 + kRowsThreads - 1) / kRowsThreads, R), dim3(kRowsThreads), 0, R, x.ffp,
              (const float*)c->gu_part, gu.splits, (uint16_t*)c->mix_y, m->ff_act);
        pend(project("down", x.down, c->mix_y, c->down_part), x.norm2b);
    }
};

}  // namespace

static Pending run_layered(oxg4_cache* c, Launcher& ln, const RowSet& rs, bool use_tc, const TraceCtx* tr) {
    oxg4_model* m = c->m;
    LayeredPass p{c, ln, rs, use_tc, !use_tc && rs.R == 1 && !rs.chunk, tr};
    for (int l = 0; l < m->cfg.num_hidden_layers && ln.status == OXG4_OK; ++l) {
        const MixPlan& x = m->layers[l].mix;
        const SplitIn in = p.input(x, l);
        if (x.kind != MIX_LATENT && x.kind != MIX_ATTENTION) p.recurrent(x, l, in);
        else if (m->es == 2) {
            if (c->kv_dtype == OXG4_BF16) p.attend<uint16_t, uint16_t>(x, l, in);
            else p.attend<uint16_t, float>(x, l, in);
        } else {
            if (c->kv_dtype == OXG4_BF16) p.attend<float, uint16_t>(x, l, in);
            else p.attend<float, float>(x, l, in);
        }
        if (x.ff > 0 && !m->parallel) p.feed_forward(x);
    }
    p.pd.h = p.cur;
    p.pd.h_out = p.nxt;
    return p.pd;
}
