// Engine methods of the Panupel family (see panupel.cuh): weight upload, sequence memory of every layer run, and the launch
// sequence of the stack.  The step function, step metadata, cache pages, slot / snapshot interface and CUDA graphs are the ones
// of kemirax_engine.cuh.  Included by engine.cu after it.
#pragma once

using namespace b200;

// places of the parts of a parallel layer's stacked projection row; the last entry is the row's length
struct PnParallelRow {
    int q, k, v, mq, mk, mv, mg, g, mi, mf, n;
    explicit PnParallelRow(const KxLayerCfg& c) {
        q = 0; k = q + c.heads * c.dim; v = k + c.kv_heads * c.dim;
        mq = v + c.kv_heads * c.vdim; mk = mq + c.mm_heads * c.mm_dim; mv = mk + c.mm_heads * c.mm_dim; mg = mv + c.mm_heads * c.mm_vdim;
        g = mg + c.mm_heads * c.mm_vdim; mi = g + c.heads; mf = mi + c.mm_heads; n = mf + c.mm_heads;
    }
};
// the same for a delta-rule layer: convolved inputs [q; k; v], output gate, write strengths, decays
struct PnDeltaRow {
    int conv, g, b, a, n;
    explicit PnDeltaRow(const KxLayerCfg& c) {
        conv = 2 * c.kv_heads * c.dim + c.heads * c.vdim;
        g = conv; b = g + c.heads * c.vdim; a = b + c.heads; n = a + c.heads;
    }
};

void b200rwkv_engine::pn_load(const StFile& st, KxSizes& z) {
    SeqModel& m = *kx;
    const int W = m.W, nr = (int)m.cfg.layers.size();
    m.embed = kx_up16(kx_host_bf16(st, "embed", m.V, W));
    m.head = kx_up16(kx_host_bf16(st, "head", m.V, W));
    m.final_w = kx_up32(kx_host_f32(st, "final.norm", W));
    if (m.cfg.has_loop) m.pass_in = kx_up16(kx_host_bf16(st, "loop.in", W, 2 * (int64_t)W));
    int ntens = 0;
    for (const KxLayerCfg& c : m.cfg.layers) ntens = std::max(ntens, c.tensors_of + 1);
    // ---- tensors, once per layer of the file ----
    std::vector<KxLayer> own(ntens);
    std::vector<char> loaded(ntens, 0);
    for (const KxLayerCfg& c : m.cfg.layers) {
        const int i = c.tensors_of;
        if (loaded[i]) continue;
        loaded[i] = 1;
        KxLayer& l = own[i];
        l.c = c;
        const std::string p = "l" + std::to_string(i) + ".";
        const int H_ = c.heads, G_ = c.kv_heads, dk = c.dim, dv = c.vdim;
        l.norm1_w = kx_up32(kx_host_f32(st, p + "norm1", W));
        l.norm1b_w = kx_up32(kx_host_f32(st, p + "norm1b", W));
        std::vector<uint16_t> w;
        auto rows = [&](const std::string& name, int64_t n) { kx_cat(w, kx_host_bf16(st, p + "mix." + name, n, W)); };
        if (c.mixer == KX_PARALLEL) {
            const PnParallelRow r(c);
            const int Hm = c.mm_heads, mk = c.mm_dim, mv = c.mm_vdim;
            rows("left.q", (int64_t)H_ * dk); rows("left.k", (int64_t)G_ * dk); rows("left.v", (int64_t)G_ * dv);
            rows("right.q", (int64_t)Hm * mk); rows("right.k", (int64_t)Hm * mk); rows("right.v", (int64_t)Hm * mv); rows("right.g", (int64_t)Hm * mv);
            rows("left.g", H_); rows("right.i", Hm); rows("right.f", Hm);
            l.proj_n = r.n;
            std::vector<float> b((size_t)r.n, 0.f);            // only the memory's two gates have a bias
            auto bi = kx_host_f32(st, p + "mix.right.i.b", Hm), bf = kx_host_f32(st, p + "mix.right.f.b", Hm);
            std::copy(bi.begin(), bi.end(), b.begin() + r.mi);
            std::copy(bf.begin(), bf.end(), b.begin() + r.mf);
            l.proj_b = kx_up32(b);
            l.qn_w = kx_up32(kx_host_f32(st, p + "mix.left.q.norm", (int64_t)H_ * dk));
            l.kn_w = kx_up32(kx_host_f32(st, p + "mix.left.k.norm", (int64_t)G_ * dk));
            l.sink = kx_up32(kx_host_f32(st, p + "mix.left.sink", H_));
            l.mm_norm_w = kx_up32(kx_host_f32(st, p + "mix.right.norm", (int64_t)Hm * mv));
            const std::vector<double> fr = kx_rot_freqs(c.rot);
            l.freq_d = (double*)dalloc(fr.size() * 8, false);
            CK(cudaMemcpy(l.freq_d, fr.data(), fr.size() * 8, cudaMemcpyHostToDevice));
            // both output projections side by side: one product over [attention heads | memory heads]
            const auto oa = kx_host_bf16(st, p + "mix.left.o", W, (int64_t)H_ * dv), om = kx_host_bf16(st, p + "mix.right.o", W, (int64_t)Hm * mv);
            const size_t na = (size_t)H_ * dv, nm = (size_t)Hm * mv;
            std::vector<uint16_t> o((na + nm) * W);
            for (int n = 0; n < W; ++n) {
                memcpy(&o[n * (na + nm)], &oa[n * na], na * 2);
                memcpy(&o[n * (na + nm) + na], &om[n * nm], nm * 2);
            }
            l.o = kx_up16(o);
        } else {
            const PnDeltaRow r(c);
            rows("q", (int64_t)G_ * dk); rows("k", (int64_t)G_ * dk); rows("v", (int64_t)H_ * dv); rows("g", (int64_t)H_ * dv); rows("b", H_); rows("a", H_);
            l.conv_C = r.conv;
            l.proj_n = r.n;
            std::vector<float> b((size_t)r.n, 0.f);            // only the decays have a bias
            auto dt = kx_host_f32(st, p + "mix.dt_bias", H_);
            std::copy(dt.begin(), dt.end(), b.begin() + r.a);
            l.proj_b = kx_up32(b);
            l.a_log = kx_up32(kx_host_f32(st, p + "mix.A_log", H_));
            l.norm_w = kx_up32(kx_host_f32(st, p + "mix.norm", dv));
            std::vector<float> cw;
            auto taps = [&](const char* name, int64_t n) {
                auto t = kx_host_f32(st, p + "mix." + name + ".conv", n * c.taps);
                cw.insert(cw.end(), t.begin(), t.end());
            };
            taps("q", (int64_t)G_ * dk); taps("k", (int64_t)G_ * dk); taps("v", (int64_t)H_ * dv);
            l.conv_w = kx_up32(cw);
            l.o = kx_up16(kx_host_bf16(st, p + "mix.o", W, (int64_t)H_ * dv));
        }
        l.proj = kx_up16(w);
        if (c.has_mlp) {                           // one gated unit: kept where a routed layer keeps its always-on expert
            l.norm2_w = kx_up32(kx_host_f32(st, p + "norm2", W));
            l.norm2b_w = kx_up32(kx_host_f32(st, p + "norm2b", W));
            l.sh_gu = kx_up16(kx_interleave(kx_host_bf16(st, p + "mlp.gate", c.ff, W), kx_host_bf16(st, p + "mlp.up", c.ff, W), c.ff, W));
            l.sh_down = kx_up16(kx_host_bf16(st, p + "mlp.down", W, c.ff));
        }
    }
    // ---- the layer runs: the tensors of their layer, sequence memory of their own ----
    auto memory = [&](KxLayer& l, size_t per_slot) {
        float* d = (float*)dalloc(std::max<size_t>((size_t)S * per_slot, 1) * 4);
        l.fixed.push_back({d, per_slot});
        return d;
    };
    m.layers.resize(nr);
    for (int r = 0; r < nr; ++r) {
        KxLayer& l = m.layers[r];
        l = own[m.cfg.layers[r].tensors_of];
        l.c = m.cfg.layers[r];
        const KxLayerCfg& c = l.c;
        size_t heads_out = (size_t)c.heads * c.vdim;
        if (c.mixer == KX_PARALLEL) {
            REQUIRE(c.mm_dim <= SCAN_MAX_DK, B200RWKV_ERR_UNSUPPORTED, "matrix memory: dim must be <= 1024");
            l.cache_D = c.kv_heads * (c.dim + c.vdim);
            l.cache = (float*)dalloc((size_t)m.npages * m.page * l.cache_D * 4);
            l.mm_state = memory(l, (size_t)c.mm_heads * scan_state_floats(c.mm_dim, c.mm_vdim));
            l.mm_n = memory(l, (size_t)c.mm_heads * c.mm_dim);
            l.mm_m = memory(l, (size_t)c.mm_heads * c.mm_vdim);
            heads_out += (size_t)c.mm_heads * c.mm_vdim;
            z.n_q = std::max(z.n_q, (size_t)c.heads * c.dim); z.n_z = std::max(z.n_z, (size_t)c.mm_heads);
        } else {
            REQUIRE(c.dim <= SCAN_MAX_DK, B200RWKV_ERR_UNSUPPORTED, "delta rule: dim must be <= 1024");
            l.rec_state = memory(l, (size_t)c.heads * scan_state_floats(c.dim, c.vdim));
            l.conv_tail = memory(l, (size_t)(c.taps - 1) * l.conv_C);
            z.n_cv = std::max(z.n_cv, (size_t)rup(l.conv_C, 4));
        }
        z.n_pr = std::max(z.n_pr, (size_t)rup(l.proj_n, 4)); z.n_vout = std::max(z.n_vout, heads_out);
        if (c.has_mlp) z.n_ys = std::max(z.n_ys, (size_t)c.ff);
    }
    sa_plan_model(m);
    CK(cudaFuncSetAttribute(delta_scan_kernel<false, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SCAN_SMEM));
    CK(cudaFuncSetAttribute(matrix_memory_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SCAN_SMEM));
    REQUIRE((size_t)W * 4 <= 200 * 1024, B200RWKV_ERR_UNSUPPORTED, "width too large for the norm kernel");
    CK(cudaFuncSetAttribute(pre_norm_kernel<NORM_THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CK(cudaFuncSetAttribute(pre_norm_kernel<PRE_NORM_THREADS_FEW_ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    CK(cudaStreamCreateWithFlags(&m.side_stream, cudaStreamNonBlocking));
    CK(cudaEventCreateWithFlags(&m.side_fork, cudaEventDisableTiming));
    CK(cudaEventCreateWithFlags(&m.side_join, cudaEventDisableTiming));
}

// the whole stack and the last norm: every sublayer begins with one pre_norm launch (the norm on the output of the sublayer that
// just finished, the residual sum, the norm on the input of the next one)
void b200rwkv_engine::pn_enqueue_layers(cudaStream_t s, int rows, int nslot_grid, bool decode, int nsplit, Profiler* prof) {
    SeqModel& m = *kx;
    const int W = m.W;
    const float eps = m.cfg.eps;
    MetaView mv{d_meta, maxT, S};
    const int* cntT = d_meta;
    auto lin = [&](const float* X, int ldx, const __nv_bfloat16* Wt, float* Y, int ldy, int N_, int K_, int epi = LE_STORE, const float* bias = nullptr) {
        LinParams p;
        memset(&p, 0, sizeof(p));
        p.X = X; p.ldx = ldx; p.W = Wt; p.Y = Y; p.ldy = ldy; p.N = N_; p.K = K_; p.cnt = cntT; p.epi = epi; p.bias = bias;
        return p;
    };
    const float* post_w = nullptr;                 // norm weight of a finished sublayer whose output waits in m.y
    auto boundary = [&](float* snap, float* cat, const float* weight, float* h, int compact, float* hidden) {
        PreNormParams pn{m.x, nullptr, nullptr, nullptr, 0, nullptr, snap, cat ? m.embed : nullptr, nullptr, weight, eps, h, compact, hidden, W, mv,
                         post_w ? m.y : nullptr, post_w, m.cfg.residual_mul, cat};
        if (rows <= 32) launch_k(pre_norm_kernel<PRE_NORM_THREADS_FEW_ROWS>, dim3(rows), dim3(PRE_NORM_THREADS_FEW_ROWS), (size_t)W * 4, pn, KC_LN, s, prof);
        else launch_k(pre_norm_kernel<NORM_THREADS>, dim3(rows), dim3(NORM_THREADS), (size_t)W * 4, pn, KC_LN, s, prof);
        post_w = nullptr;
    };
    const int chunks_grid = decode ? rows : cdiv(rows, m.qb_prompt) + nslot_grid;
    for (size_t li = 0; li < m.layers.size(); ++li) {
        KxLayer& l = m.layers[li];
        const KxLayerCfg& c = l.c;
        const int H_ = c.heads, G_ = c.kv_heads, dk = c.dim, dv = c.vdim, PN = rup(l.proj_n, 4);
        if (c.opens_pass >= 0) {                   // x <- W_in [x; embedding row]
            boundary(nullptr, m.G, nullptr, nullptr, 0, nullptr);
            kx_lin(s, prof, lin(m.G, 2 * W, m.pass_in, m.x, W, W, 2 * W), rows, 1);
        }
        boundary(nullptr, nullptr, l.norm1_w, m.h, 0, nullptr);
        kx_lin(s, prof, lin(m.h, W, l.proj, m.pr, PN, l.proj_n, W, LE_STORE, l.proj_b), rows, 1);
        int KO = H_ * dv;                          // heads' outputs side by side, the input of the output projection
        if (c.mixer == KX_PARALLEL) {
            const PnParallelRow r(c);
            const int Hm = c.mm_heads, mk = c.mm_dim, mvd = c.mm_vdim;
            KO += Hm * mvd;
            // the memory runs beside the attention: both read the projection row and write their own columns of vout
            const bool fork = prof == nullptr;
            cudaStream_t s2 = fork ? m.side_stream : s;
            if (fork) { CK(cudaEventRecord(m.side_fork, s)); CK(cudaStreamWaitEvent(s2, m.side_fork, 0)); }
            {
                const ScanShape sh = scan_shape(mk, mvd, 2, decode);
                MatrixMemoryParams mp{m.pr + r.mq, m.pr + r.mk, m.pr + r.mv, PN, m.pr + r.mi, m.pr + r.mf, l.mm_state, l.mm_n, l.mm_m, m.z, Hm, mk, mvd,
                                      c.mm_cap, 1.f / sqrtf((float)mk), 1e-6f, sh,
                                      {m.vout + H_ * dv, KO, m.z, m.pr + r.mg, PN, l.mm_norm_w, mvd, Hm, mvd, eps, c.mm_mul, 0, mv}};
                launch_k(decode ? matrix_memory_kernel<true> : matrix_memory_kernel<false>, dim3(Hm * sh.ncta, nslot_grid), dim3(sh.threads), sh.smem_floats() * 4, mp, KC_WKV, s2, prof);
                if (sh.ncta > 1) launch_k(head_norm_kernel, dim3(rows, cdiv(Hm, 4)), dim3(128), 0, mp.norm, KC_LN, s2, prof);
            }
            RotPrepParams rp{m.pr + r.q, m.pr + r.k, m.pr + r.v, PN, m.q, H_ * dk, l.cache, m.d_table, m.npages, m.page, l.qn_w, l.kn_w, l.freq_d,
                             H_, G_, dk, dv, c.rot.dims, eps, mv, m.sm};
            launch_k(rot_prep_kernel, dim3(rows), dim3(ROT_PREP_THREADS), (size_t)std::max(c.rot.dims, 4) * 4, rp, KC_OTHER, s, prof);
            const SaPlan plan = sa_plan(l, m.qb_prompt, decode);
            SinkAttnParams sp;
            memset(&sp, 0, sizeof(sp));
            sp.q = m.q; sp.ldq = H_ * dk; sp.cache = l.cache; sp.table = m.d_table; sp.stride = m.npages; sp.page = m.page; sp.D = l.cache_D;
            sp.koff = 0; sp.voff = G_ * dk; sp.out = m.vout; sp.ldo = KO; sp.gate = m.pr + r.g; sp.ldg = PN; sp.gate_heads = 1;
            sp.out_mul = c.attn_mul; sp.sink = l.sink; sp.scale = c.scale; sp.H = H_; sp.G = G_; sp.dk = dk; sp.dv = dv; sp.HB = plan.hb;
            sp.win = 1 << 30;                      // the whole context
            sp.qb = plan.qb; sp.gt = plan.gt; sp.cl = nsplit; sp.nbuf = plan.nbuf; sp.ks = plan.ks;
            sp.nsub = decode ? 1 : m.qb_prompt / plan.qb;
            sp.meta = mv; sp.sm = m.sm;
            launch_cluster = nsplit;
            launch_k(plan.kern, dim3(chunks_grid * sp.nsub * nsplit, cdiv(H_, plan.hb)), dim3(plan.threads), plan.smem, sp, KC_WKV, s, prof);
            if (fork) { CK(cudaEventRecord(m.side_join, s2)); CK(cudaStreamWaitEvent(s, m.side_join, 0)); }
        } else {
            const PnDeltaRow r(c);
            const int C_ = l.conv_C, ldc = rup(C_, 4);
            ShortConvParams cp{m.pr, PN, m.cv, ldc, l.conv_w, l.conv_tail, C_, c.taps, mv};
            kx_short_conv(s, prof, cp, rows, nslot_grid, decode);
            const ScanShape sh = scan_shape(dk, dv, 2, decode);
            DeltaScanParams dp{m.cv, m.cv + G_ * dk, m.cv + 2 * G_ * dk, ldc, m.pr + r.a, PN, m.pr + r.b, PN, l.a_log, l.rec_state, H_, G_, dk, dv,
                               1.f / sqrtf((float)dk), 1e-6f, sh, {m.vout, KO, nullptr, m.pr + r.g, PN, l.norm_w, 0, H_, dv, eps, 1.f, 1, mv}};
            launch_k(decode ? delta_scan_kernel<false, true> : delta_scan_kernel<false, false>, dim3(H_ * sh.ncta, nslot_grid), dim3(sh.threads), sh.smem_floats() * 4, dp, KC_WKV, s, prof);
            if (sh.ncta > 1) launch_k(head_norm_kernel, dim3(rows, cdiv(H_, 4)), dim3(128), 0, dp.norm, KC_LN, s, prof);
        }
        kx_lin(s, prof, lin(m.vout, KO, l.o, m.y, W, W, KO), rows, 1);
        post_w = l.norm1b_w;
        if (c.has_mlp) {
            boundary(nullptr, nullptr, l.norm2_w, m.h, 0, nullptr);
            kx_lin(s, prof, lin(m.h, W, l.sh_gu, m.ys, c.ff, 2 * c.ff, W, LE_GLU_SILU), rows, 1);
            kx_lin(s, prof, lin(m.ys, c.ff, l.sh_down, m.y, W, W, c.ff), rows, 1);
            post_w = l.norm2b_w;
        }
        if (m.dbg_layers && !use_graph)            // bring-up aid: the residual as this run leaves it
            boundary(m.dbg_layers + li * (size_t)maxT * W, nullptr, nullptr, nullptr, 0, nullptr);
    }
    boundary(nullptr, nullptr, m.final_w, m.hn, 1, d_hidden);
}
