// Launch shapes of the sink-attention kernels (sink_attn.cuh) for the layers of a model: which form of the kernel, query heads and
// tokens per CTA, tile buffers, and the clusters the device can hold at once.  Included by engine.cu after kemirax_engine.cuh; the
// families whose layers attend through those kernels call sa_plan_model once their layers know their sizes.
#pragma once

using namespace b200;

typedef void (*SinkAttnKernel)(const SinkAttnParams);
static inline SinkAttnKernel sa_tile_kernel(int rb) {
    return rb >= 4 ? sink_attn_kernel<4> : (rb == 2 ? sink_attn_kernel<2> : sink_attn_kernel<1>);
}

// the attention launch sees every mixer as (H query heads, G key heads, key size, value size, value = leading part of the key?)
struct SaShape { int H, G, dk, dv; bool valias; };
static inline SaShape sa_shape(const KxLayerCfg& c) {
    if (c.mixer == KX_LATENT) return {c.heads, 1, c.kv_rank + c.rot_dim, c.kv_rank, true};        // absorbed form: one shared row
    return {c.heads, c.kv_heads, c.dim, c.vdim, false};
}

static inline bool sa_layer(const KxLayerCfg& c) { return c.mixer == KX_SINK || c.mixer == KX_LATENT || c.mixer == KX_PARALLEL ||
                                                         c.mixer == KX_BIAS_WINDOW || c.mixer == KX_CHUNK_GLA; }

// query heads per CTA: whole key heads, or a part of one key head's query heads; about `want`
static inline int sa_heads_per_cta(int H, int G, int want) {
    const int rep = H / G;
    want = std::max(1, std::min(want, H));
    if (G == 1) return want;
    if (rep >= want) {
        int d = want;
        while (rep % d) --d;
        return d;
    }
    return rep * (want / rep);
}

// the register form is built for key rows of one 512-byte piece per head.  (With three and five pieces, which the kernel's
// template allows, a decode step of a 576-float latent row took 120 us where the tile form takes 84: every piece's loads wait
// for the registers of the piece before it.)
static inline SinkAttnKernel sa_reg_kernel(int rb, bool decode) {
    if (decode) return rb >= 4 ? sink_attn_reg_kernel<4, 1, 1> : (rb == 2 ? sink_attn_reg_kernel<2, 1, 1> : sink_attn_reg_kernel<1, 1, 1>);
    return rb >= 4 ? sink_attn_reg_kernel<4, 1, 4> : (rb == 2 ? sink_attn_reg_kernel<2, 1, 4> : sink_attn_reg_kernel<1, 1, 4>);
}

// how one attention launch of a layer runs: which kernel, its block size and shared memory, and the tile parameters
struct SaPlan { SinkAttnKernel kern; int threads; size_t smem; int gt, nbuf, qb, ks, hb; };

static SaPlan sa_plan(const KxLayer& l, int qb_prompt, bool decode) {
    const SaShape a = sa_shape(l.c);
    const int rep = a.H / a.G, HB = decode ? l.sa_hb_decode : l.sa_hb;
    const int nhc = std::min(rep, HB), ncv = HB / nhc;
    SaPlan p;
    p.hb = HB;
    if (l.sa_reg) {
        const int qb = decode ? 1 : qb_prompt, rows = qb * nhc;              // rows of one key head in a full chunk
        const int rb = rows >= 4 ? 4 : (rows >= 2 ? 2 : 1);
        const int items = ncv * cdiv(rows, rb);
        int ks = 1;                                // few items (decode): the 8 warps share each item's key tiles
        while (ks < 8 && items * ks * 2 <= SAR_THREADS / 32) ks *= 2;
        p.kern = sa_reg_kernel(rb, decode); p.threads = SAR_THREADS; p.smem = sink_attn_reg_smem(qb, HB, rep, a.dv, rb, ks);
        p.gt = 1; p.nbuf = 1; p.qb = qb; p.ks = ks;
        return p;
    }
    const int qb = decode ? 1 : l.sa_qb, rows = qb * nhc;
    const int gt = decode ? l.sa_gt_decode : l.sa_gt, nbuf = decode ? l.sa_nbuf_decode : l.sa_nbuf;
    // rows per warp: every key float a lane reads from the tile feeds one product per row, and the tile loop is bound by
    // shared-memory reads, so as many rows as still leave 4 warps an item (8 in decode-shaped
    int rb = SA_RB;
    while (rb > 1 && std::min(gt, ncv) * cdiv(rows, rb) < (decode ? 8 : 4)) rb >>= 1;    // steps, whose CTAs have an SM to themselves)
    p.kern = sa_tile_kernel(rb);
    p.threads = std::min(gt, ncv) * cdiv(rows, rb) >= 16 ? SA_THREADS : 256;
    p.smem = sink_attn_smem(qb, HB, a.dk, a.dv, gt, nbuf, a.valias);
    p.gt = gt; p.nbuf = nbuf; p.qb = qb; p.ks = 1;
    return p;
}

// fills the launch shape of every attention layer (cache_D must be set) and the model's cluster limits
static void sa_plan_model(SeqModel& m) {
    const int qb = 4;                              // tokens per chunk of a prompt step; a layer whose rows do not fit takes a part of a chunk per CTA
    m.qb_prompt = qb;
    m.max_split = m.wa_ctas_prompt = m.wa_ctas_decode = 8;
    m.sa_ygroups = m.sa_ygroups_decode = 1 << 30;
    for (KxLayer& l : m.layers) {
        if (!sa_layer(l.c)) continue;
        const SaShape a = sa_shape(l.c);
        // launch shape of the attention kernel: about 16 query heads per CTA, fewer (and then shorter chunks) where the rows of a
        // chunk would not fit into shared memory beside one tile
        // the register form takes key / value sizes that are multiples of four up to 128; longer rows (a latent) and odd sizes
        // go through shared-memory tiles
        l.sa_reg = a.dk % 4 == 0 && a.dv % 4 == 0 && l.cache_D % 4 == 0 && a.dk <= 128 && a.dv <= 128;
        l.sa_hb = sa_heads_per_cta(a.H, a.G, 16);
        l.sa_qb = qb;
        // tile form: rows (tokens x heads) per CTA such that two CTAs fit an SM beside one tile each (one loads while the other
        // multiplies); where that would leave fewer than four rows, one CTA per SM
        const int hb0 = l.sa_hb;
        for (size_t target : {(size_t)112 * 1024, (size_t)160 * 1024}) {
            if (l.sa_reg) break;
            l.sa_qb = qb; l.sa_hb = hb0;
            while (sink_attn_smem(l.sa_qb, l.sa_hb, a.dk, a.dv, 1, 1, a.valias) > target) {
                if (l.sa_qb > 1) l.sa_qb /= 2;
                else if (l.sa_hb > 1 && sa_heads_per_cta(a.H, a.G, l.sa_hb / 2) < l.sa_hb) l.sa_hb = sa_heads_per_cta(a.H, a.G, l.sa_hb / 2);
                else break;
            }
            if (sink_attn_smem(l.sa_qb, l.sa_hb, a.dk, a.dv, 1, 1, a.valias) <= target && l.sa_qb * l.sa_hb >= 4) break;
        }
        REQUIRE(l.sa_reg || sink_attn_smem(l.sa_qb, l.sa_hb, a.dk, a.dv, 1, 1, a.valias) <= 160 * 1024, B200RWKV_ERR_UNSUPPORTED,
                "attention heads too large for shared memory");
        // decode-shaped steps have one row per head: the register form then takes one key head per CTA, so that a chunk's tiles
        // are spread over more warps
        l.sa_hb_decode = l.sa_reg ? sa_heads_per_cta(a.H, a.G, std::max(1, a.H / a.G)) : l.sa_hb;
        m.sa_ygroups = std::min(m.sa_ygroups, cdiv(a.H, l.sa_hb));
        m.sa_ygroups_decode = std::min(m.sa_ygroups_decode, cdiv(a.H, l.sa_hb_decode));
        for (int dec = 0; dec < 2; ++dec) {        // as many key heads per tile load, and two tile buffers, where they fit
            const int q = dec ? 1 : l.sa_qb;
            const int hb = dec ? l.sa_hb_decode : l.sa_hb, ncv = std::max(1, hb / std::max(1, a.H / a.G));
            int nbuf = 2, gt = ncv;
            if (sink_attn_smem(q, hb, a.dk, a.dv, 1, 2, a.valias) > (size_t)(dec ? 200 : 112) * 1024) nbuf = 1;
            while (gt > 1 && sink_attn_smem(q, hb, a.dk, a.dv, gt, nbuf, a.valias) > (dec ? 160 : 112) * 1024) gt = (gt + 1) / 2;
            (dec ? l.sa_gt_decode : l.sa_gt) = gt;
            (dec ? l.sa_nbuf_decode : l.sa_nbuf) = nbuf;
        }
    }
    if (m.sa_ygroups == 1 << 30) m.sa_ygroups = m.sa_ygroups_decode = 1;       // no attention layer
    for (int rb = 1; rb <= SA_RB; rb *= 2) {
        CK(cudaFuncSetAttribute(sa_tile_kernel(rb), cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        for (bool decode : {false, true}) CK(cudaFuncSetAttribute(sa_reg_kernel(rb, decode), cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    // the largest cluster the attention launch may ask for: what the device can co-schedule at this layer's shared memory
    for (const KxLayer& l : m.layers) {
        if (!sa_layer(l.c)) continue;
        const SaPlan pp = sa_plan(l, qb, false), pd = sa_plan(l, qb, true);
        REQUIRE(pp.smem <= 200 * 1024 && pd.smem <= 200 * 1024, B200RWKV_ERR_UNSUPPORTED, "attention heads too large for shared memory");
        int cl = 8, cl_ok = 0;
        for (; cl > 1; cl >>= 1) {
            bool ok = true;
            for (const SaPlan* a : {&pp, &pd}) {
                int lg = 0;
                while ((1 << lg) < cl) ++lg;
                cudaLaunchConfig_t cfg;
                memset(&cfg, 0, sizeof(cfg));
                cfg.gridDim = dim3(cl); cfg.blockDim = dim3(a->threads);
                cfg.dynamicSmemBytes = a->smem;
                cudaLaunchAttribute at;
                at.id = cudaLaunchAttributeClusterDimension;
                at.val.clusterDim.x = (unsigned)cl; at.val.clusterDim.y = 1; at.val.clusterDim.z = 1;
                cfg.attrs = &at; cfg.numAttrs = 1;
                int n = 0;
                if (cudaOccupancyMaxActiveClusters(&n, a->kern, &cfg) != cudaSuccess || n <= 0) { ok = false; n = 0; }
                cudaGetLastError();
                int& cap = (a == &pd ? m.cl_cap_decode : m.cl_cap_prompt)[lg];      // clusters of this size the GPU holds at once
                cap = std::min(cap, n);
            }
            if (ok && cl_ok == 0) cl_ok = cl;
        }
        m.max_split = std::min(m.max_split, std::max(cl_ok, 1));
        int np = 1, nd = 1;
        CK(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&np, pp.kern, pp.threads, pp.smem));
        CK(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&nd, pd.kern, pd.threads, pd.smem));
        m.wa_ctas_prompt = std::max(1, std::min(m.wa_ctas_prompt, np));
        m.wa_ctas_decode = std::max(1, std::min(m.wa_ctas_decode, nd));
    }
}
