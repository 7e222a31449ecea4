// Engine methods of the Fufipel family (see fufipel.cuh): weight upload, sequence memory of every layer, and the launch sequence of
// the stack.  The step function, step metadata, cache pages, slot / snapshot interface and CUDA graphs are the ones of
// kemirax_engine.cuh.  Included by engine.cu after it.
#pragma once

using namespace b200;

// places of the parts of a layer's stacked projection row.  `proj` (a multiple of four) is the length of the mixer's part; the
// feed-forward's interleaved (gate, up) rows follow it in the matrix and land, gated, in the row of heads' outputs
struct FfRow {
    int q = 0, k = 0, v = 0, g = 0;                // attention (left half of a parallel layer); g: output gate
    int rq = 0, rk = 0, rv = 0, rg = 0, ra = 0;    // gated linear attention; ra: low-rank decay input
    int proj = 0;
    int heads = 0, rheads = 0, out = 0;            // outputs of the (left) heads, of the right heads, with the feed-forward's units
    FfRow(const KxLayerCfg& c, int a_rank) {
        const bool par = c.mixer == KX_CHUNK_GLA, own = c.kv_from < 0;
        heads = c.heads * c.vdim;
        k = c.heads * c.dim;
        v = k + (own ? c.kv_heads * c.dim : 0);
        int n = v + (own ? c.kv_heads * c.vdim : 0);
        if (par) {
            rheads = c.mm_heads * c.mm_vdim;
            rq = n; rk = rq + c.mm_heads * c.mm_dim; rv = rk + c.mm_heads * c.mm_dim; rg = rv + rheads; ra = rg + rheads;
            n = ra + a_rank;
        } else {
            g = n; n += heads;
        }
        proj = rup(n, 4);
        out = heads + rheads + (c.has_mlp ? c.ff : 0);
    }
};

void b200rwkv_engine::ff_load(const StFile& st, KxSizes& z) {
    SeqModel& m = *kx;
    const int W = m.W, nl = (int)m.cfg.layers.size();
    auto plus_one = [](std::vector<float> v) { for (float& f : v) f += 1.f; return v; };     // norm weights are stored as offsets from one
    m.embed = kx_up16(kx_host_bf16(st, "embed", m.V, W));
    m.head = m.embed;                              // the embedding table is the output matrix
    {   // the factor on the logits rides on the last norm's weight
        std::vector<float> f = plus_one(kx_host_f32(st, "final.norm", W));
        for (float& v : f) v *= m.cfg.logit_scale;
        m.final_w = kx_up32(f);
    }
    if (m.cfg.pair_buckets > 0) m.pairs = kx_up16(kx_host_bf16(st, "bigram", (int64_t)m.cfg.pair_buckets + 1, W));
    m.layers.resize(nl);
    auto memory = [&](KxLayer& l, size_t per_slot) {
        float* d = (float*)dalloc(std::max<size_t>((size_t)S * per_slot, 1) * 4);
        l.fixed.push_back({d, per_slot});
        return d;
    };
    if (m.pairs) m.last_tok = memory(m.layers[0], 1);      // the previous token travels with the first layer's memory
    for (int i = 0; i < nl; ++i) {
        KxLayer& l = m.layers[i];
        l.c = m.cfg.layers[i];
        const KxLayerCfg& c = l.c;
        const std::string p = "l" + std::to_string(i) + ".";
        const int H_ = c.heads, G_ = c.kv_heads, dk = c.dim, dv = c.vdim;
        const bool par = c.mixer == KX_CHUNK_GLA;
        l.norm1_w = kx_up32(plus_one(kx_host_f32(st, p + "norm1", W)));
        if (par) {
            const StTensor* a1 = st.find(p + "mix.right.a1");
            REQUIRE(a1 && a1->shape.size() == 2, B200RWKV_ERR_INVALID, "missing tensor: " + p + "mix.right.a1");
            l.a_rank = (int)a1->shape[0];
        }
        const FfRow r(c, l.a_rank);
        std::vector<uint16_t> w;
        auto rows = [&](const std::string& name, int64_t n) { kx_cat(w, kx_host_bf16(st, p + "mix." + name, n, W)); };
        // output matrices side by side: one product over the concatenated inputs
        auto beside = [&](const std::vector<uint16_t>& a, int na, const std::vector<uint16_t>& b, int nb) {
            std::vector<uint16_t> o((size_t)(na + nb) * W);
            for (int n = 0; n < W; ++n) {
                memcpy(&o[(size_t)n * (na + nb)], &a[(size_t)n * na], (size_t)na * 2);
                if (nb) memcpy(&o[(size_t)n * (na + nb) + na], &b[(size_t)n * nb], (size_t)nb * 2);
            }
            return o;
        };
        std::vector<uint16_t> down;
        if (c.has_mlp) down = kx_host_bf16(st, p + "mlp.down", W, c.ff);
        if (par) {
            const int Hr = c.mm_heads, mk = c.mm_dim, mv = c.mm_vdim;
            REQUIRE(mk <= SCAN_MAX_DK, B200RWKV_ERR_UNSUPPORTED, "gla: dim must be <= 1024");
            rows("left.q", (int64_t)H_ * dk); rows("left.k", (int64_t)G_ * dk); rows("left.v", (int64_t)G_ * dv);
            rows("right.q", (int64_t)Hr * mk); rows("right.k", (int64_t)Hr * mk); rows("right.v", (int64_t)Hr * mv); rows("right.g", (int64_t)Hr * mv);
            rows("right.a1", l.a_rank);
            l.a2 = kx_up16(kx_host_bf16(st, p + "mix.right.a2", (int64_t)Hr * mk, l.a_rank));
            l.a2_b = kx_up32(kx_host_f32(st, p + "mix.right.a2.b", (int64_t)Hr * mk));
            l.norm_w = kx_up32(kx_host_f32(st, p + "mix.right.norm", mv));
            l.norm1b_w = kx_up32(kx_host_f32(st, p + "mix.left.out", W));
            l.norm2b_w = kx_up32(kx_host_f32(st, p + "mix.right.out", W));
            l.o = kx_up16(kx_host_bf16(st, p + "mix.left.o", W, r.heads));
            l.o2 = kx_up16(kx_host_bf16(st, p + "mix.right.o", W, r.rheads));
            if (c.has_mlp) l.sh_down = kx_up16(down);
            l.mag = kx_rot_mag(c.rot);
            l.gla_state = memory(l, (size_t)Hr * scan_state_floats(mk, mv));
            z.n_z = std::max(z.n_z, (size_t)Hr * mk);
        } else {
            rows("q", (int64_t)H_ * dk);
            l.qn_w = kx_up32(kx_host_f32(st, p + "mix.q.norm", (int64_t)H_ * dk));
            if (c.kv_from < 0) {
                rows("k", (int64_t)G_ * dk); rows("v", (int64_t)G_ * dv);
                l.kn_w = kx_up32(kx_host_f32(st, p + "mix.k.norm", (int64_t)G_ * dk));
            }
            rows("g", r.heads);
            l.o = kx_up16(beside(kx_host_bf16(st, p + "mix.o", W, r.heads), r.heads, down, c.has_mlp ? c.ff : 0));
            const StTensor* rt = st.find(p + "mix.rel");
            REQUIRE(rt && rt->shape.size() == 2 && (int)rt->shape[1] == H_, B200RWKV_ERR_INVALID, "tensor " + p + "mix.rel has an unexpected shape");
            const int B_ = (int)rt->shape[0];
            const std::vector<float> t = zf_bias_table(kx_host_f32(st, p + "mix.rel", (int64_t)B_ * H_), B_, H_, c.bias_max, l.rel_n);
            std::vector<float> th(t.size());       // head by head: a warp reads neighbouring distances
            for (int n = 0; n <= l.rel_n; ++n)
                for (int h = 0; h < H_; ++h) th[(size_t)h * (l.rel_n + 1) + n] = t[(size_t)n * H_ + h];
            l.rel_bias = kx_up32(th);
        }
        w.resize((size_t)r.proj * W, 0);
        if (c.has_mlp) kx_cat(w, kx_interleave(kx_host_bf16(st, p + "mlp.gate", c.ff, W), kx_host_bf16(st, p + "mlp.up", c.ff, W), c.ff, W));
        l.proj = kx_up16(w);
        l.proj_n = r.proj + (c.has_mlp ? 2 * c.ff : 0);
        const std::vector<double> fr = kx_rot_freqs(c.rot);
        l.freq_d = (double*)dalloc(fr.size() * 8, false);
        CK(cudaMemcpy(l.freq_d, fr.data(), fr.size() * 8, cudaMemcpyHostToDevice));
        if (c.kv_from < 0) {
            l.cache_D = G_ * (dk + dv);
            l.cache = (float*)dalloc((size_t)m.npages * m.page * l.cache_D * 4);
        } else {
            l.cache = m.layers[c.kv_from].cache;   // the lender's pool, the same page table
        }
        z.n_pr = std::max(z.n_pr, (size_t)r.proj); z.n_q = std::max(z.n_q, (size_t)H_ * dk); z.n_vout = std::max(z.n_vout, (size_t)r.out);
    }
    sa_plan_model(m);
    CK(cudaFuncSetAttribute(gla_scan_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SCAN_SMEM));
    REQUIRE((size_t)W * 8 <= 200 * 1024, B200RWKV_ERR_UNSUPPORTED, "width too large for the norm kernel");
    CK(cudaFuncSetAttribute(pre_norm_kernel<NORM_THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CK(cudaFuncSetAttribute(pre_norm_kernel<PRE_NORM_THREADS_FEW_ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CK(cudaStreamCreateWithFlags(&m.side_stream, cudaStreamNonBlocking));
    CK(cudaEventCreateWithFlags(&m.side_fork, cudaEventDisableTiming));
    CK(cudaEventCreateWithFlags(&m.side_join, cudaEventDisableTiming));
    m.side_lin = true;
}

// the whole stack and the last norm: every layer begins with one pre_norm launch (in front of it the residual sum of a parallel layer's
// two normed halves), then one product for all projections of mixer and feed-forward
void b200rwkv_engine::ff_enqueue_layers(cudaStream_t s, int rows, int nslot_grid, bool decode, int nsplit, Profiler* prof) {
    SeqModel& m = *kx;
    const int W = m.W;
    const float eps = m.cfg.eps, mul = m.cfg.residual_mul;
    MetaView mv{d_meta, maxT, S};
    const int* cntT = d_meta;
    auto lin = [&](const float* X, int ldx, const __nv_bfloat16* Wt, float* Y, int ldy, int N_, int K_, int epi = LE_STORE, const float* bias = nullptr) {
        LinParams p;
        memset(&p, 0, sizeof(p));
        p.X = X; p.ldx = ldx; p.W = Wt; p.Y = Y; p.ldy = ldy; p.N = N_; p.K = K_; p.cnt = cntT; p.epi = epi; p.bias = bias;
        p.limit = mul;                             // LE_ADD: the factor on a sublayer's contribution
        return p;
    };
    const KxLayer* halves = nullptr;               // a parallel layer whose two outputs wait in m.y and m.hs
    auto boundary = [&](float* snap, const float* weight, float* h, int compact, float* hidden) {
        PreNormParams pn{m.x, nullptr, nullptr, nullptr, 0, nullptr, snap, nullptr, nullptr, weight, eps, h, compact, hidden, W, mv};
        if (halves) { pn.y = m.y; pn.post_w = halves->norm1b_w; pn.y2 = m.hs; pn.post2_w = halves->norm2b_w; pn.post_mul = 0.5f * mul; }
        const size_t sm_b = (size_t)W * (halves ? 8 : 4);
        if (rows <= 32) launch_k(pre_norm_kernel<PRE_NORM_THREADS_FEW_ROWS>, dim3(rows), dim3(PRE_NORM_THREADS_FEW_ROWS), sm_b, pn, KC_LN, s, prof);
        else launch_k(pre_norm_kernel<NORM_THREADS>, dim3(rows), dim3(NORM_THREADS), sm_b, pn, KC_LN, s, prof);
        halves = nullptr;
    };
    const int chunks_grid = decode ? rows : cdiv(rows, m.qb_prompt) + nslot_grid;
    for (size_t li = 0; li < m.layers.size(); ++li) {
        KxLayer& l = m.layers[li];
        const KxLayerCfg& c = l.c;
        const int H_ = c.heads, G_ = c.kv_heads, dk = c.dim, dv = c.vdim;
        const bool par = c.mixer == KX_CHUNK_GLA;
        const FfRow r(c, l.a_rank);
        const int PN = r.proj, KO = r.out;
        boundary(nullptr, l.norm1_w, m.h, 0, nullptr);
        {   // mixer projections -> pr; the feed-forward's gated units -> the end of the row of heads' outputs
            LinParams p = lin(m.h, W, l.proj, m.pr, PN, l.proj_n, W, c.has_mlp ? LE_SPLIT_GLU_RELU : LE_STORE);
            p.split = PN; p.Y2 = m.vout + r.heads + r.rheads; p.ldy2 = KO;
            kx_lin(s, prof, p, rows, 1);
        }
        // a parallel layer's right half and its feed-forward run beside the attention
        const bool fork = par && prof == nullptr;
        cudaStream_t s2 = fork ? m.side_stream : s;
        if (fork) { CK(cudaEventRecord(m.side_fork, s)); CK(cudaStreamWaitEvent(s2, m.side_fork, 0)); }
        if (par) {
            const int Hr = c.mm_heads, mk = c.mm_dim, mvd = c.mm_vdim;
            kx_lin(s2, prof, lin(m.pr + r.ra, PN, l.a2, m.z, Hr * mk, Hr * mk, l.a_rank, LE_STORE, l.a2_b), rows, 1);
            kx_gla(s2, prof, l, Hr, mk, mvd, m.pr + r.rq, m.pr + r.rk, m.pr + r.rv, m.pr + r.rg, PN, m.vout + r.heads, KO, rows, nslot_grid, decode);
            kx_lin(s2, prof, lin(m.vout + r.heads, KO, l.o2, m.hs, W, W, r.rheads), rows, 1);
            if (c.has_mlp) kx_lin(s2, prof, lin(m.vout + r.heads + r.rheads, KO, l.sh_down, m.x, W, W, c.ff, LE_ADD), rows, 1);
        }
        const bool own = c.kv_from < 0;
        RotPrepParams rp{m.pr + r.q, own ? m.pr + r.k : nullptr, own ? m.pr + r.v : nullptr, PN, m.q, H_ * dk, l.cache, m.d_table, m.npages, m.page,
                         l.qn_w, l.kn_w, l.freq_d, H_, G_, dk, dv, c.rot.dims, eps, mv, m.sm, l.mag};
        launch_k(rot_prep_kernel, dim3(rows), dim3(ROT_PREP_THREADS), (size_t)std::max(c.rot.dims, 4) * 4, rp, KC_OTHER, s, prof);
        const SaPlan plan = sa_plan(l, m.qb_prompt, decode);
        SinkAttnParams sp;
        memset(&sp, 0, sizeof(sp));
        sp.q = m.q; sp.ldq = H_ * dk; sp.cache = l.cache; sp.table = m.d_table; sp.stride = m.npages; sp.page = m.page; sp.D = G_ * (dk + dv);
        sp.koff = 0; sp.voff = G_ * dk; sp.out = m.vout; sp.ldo = KO; sp.out_mul = 1.f; sp.scale = c.scale;
        sp.H = H_; sp.G = G_; sp.dk = dk; sp.dv = dv; sp.HB = plan.hb;
        if (par) {
            sp.win = 1 << 30; sp.chunk = c.chunk;
        } else {
            sp.win = c.window; sp.keep = c.keep_first; sp.bias = l.rel_bias; sp.nb = l.rel_n;
            sp.gate = m.pr + r.g; sp.ldg = PN;
        }
        sp.qb = plan.qb; sp.gt = plan.gt; sp.cl = nsplit; sp.nbuf = plan.nbuf; sp.ks = plan.ks;
        sp.nsub = decode ? 1 : m.qb_prompt / plan.qb;
        sp.meta = mv; sp.sm = m.sm;
        launch_cluster = nsplit;
        launch_k(plan.kern, dim3(chunks_grid * sp.nsub * nsplit, cdiv(H_, plan.hb)), dim3(plan.threads), plan.smem, sp, KC_WKV, s, prof);
        if (par) {
            kx_lin(s, prof, lin(m.vout, KO, l.o, m.y, W, W, r.heads), rows, 1);
            halves = &l;
        } else {                                   // attention and feed-forward in one product, straight into the residual
            kx_lin(s, prof, lin(m.vout, KO, l.o, m.x, W, W, KO, LE_ADD), rows, 1);
        }
        if (fork) { CK(cudaEventRecord(m.side_join, s2)); CK(cudaStreamWaitEvent(s, m.side_join, 0)); }
        if (m.dbg_layers && !use_graph)            // bring-up aid: the residual as this layer leaves it
            boundary(m.dbg_layers + li * (size_t)maxT * W, nullptr, nullptr, 0, nullptr);
    }
    boundary(nullptr, m.final_w, m.hn, 1, d_hidden);
}
