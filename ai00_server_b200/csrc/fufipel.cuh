// Fufipel model family: blocks with one norm whose output both sublayers read,
//     h = N1(x);   x += r (Mixer(h) + FF(h))                              (r: residual_mult; RMS norms 1 + w; FF may be absent)
// The embedding row of a token is scaled and a row looked up by a hash of (previous token, token) is added (rmsnorm.cuh:
// embed_rows_kernel).  Mixers: "attention" = softmax attention with a norm over the whole query / key projection, no rotation, a
// learned bias per (distance bucket, head), a sliding window that keeps the first tokens and a sigmoid gate per output entry, on keys
// and values of its own or of an earlier layer (sink_attn.cuh);  "parallel" = rotary softmax attention inside fixed chunks of the
// sequence (sink_attn.cuh) beside gated linear attention (gla.cuh), each output normed over the width, the two averaged.
// Feed-forward: W_down (relu(W_gate h) * (W_up h)).  The embedding table is the output matrix.
// Every size and constant that can differ between models comes from config.json / the tensor shapes.  The family shares the
// sequence-model engine of the other config.json families (kemirax.cuh: configuration structs, slot / page / snapshot plumbing); this
// file reads its configuration.
#pragma once

namespace b200 {

static KxConfig ff_parse_config(const JVal& root) {
    KxConfig c;
    c.family = KX_FAMILY_FUFIPEL;
    c.vocab = root.integer("vocab");
    c.width = root.integer("width");
    c.eps = (float)root.at("norm").number("eps");
    c.residual_mul = root.has("residual_mult") ? (float)root.number("residual_mult") : 1.f;
    c.logit_scale = root.has("logit_scale") ? (float)root.number("logit_scale") : 1.f;
    if (root.has("embedding")) {
        const JVal& e = root.at("embedding");
        if (e.has("scale")) c.embed_scale = (float)e.number("scale");
        if (e.has("bigram")) {
            const JVal& b = e.at("bigram");
            c.pair_buckets = b.integer("buckets"); c.pair_mul_prev = b.integer("mul_prev"); c.pair_mul_cur = b.integer("mul_cur");
            REQUIRE(c.pair_buckets >= 1, B200RWKV_ERR_INVALID, "config: embedding.bigram.buckets must be >= 1");
            REQUIRE(c.vocab <= 1 << 24, B200RWKV_ERR_UNSUPPORTED, "config: vocab too large for pair embeddings");     // last tokens are kept as floats
        }
    }
    const JVal& ls = root.at("layers");
    REQUIRE(ls.kind == JVal::ARR && !ls.arr.empty(), B200RWKV_ERR_INVALID, "config: layers");
    for (const JVal& l : ls.arr) {
        KxLayerCfg k;
        REQUIRE(l.kind == JVal::OBJ && l.has("type") && l.at("type").kind == JVal::STR, B200RWKV_ERR_INVALID, "config: layer without a type");
        const std::string type = l.at("type").str;
        const JVal& m = l.at("mixer");
        auto heads = [&](const JVal& v) {
            k.heads = v.integer("heads"); k.dim = v.integer("dim");
            k.vdim = v.has("vdim") ? v.integer("vdim") : k.dim;
            k.kv_heads = v.has("kv_heads") ? v.integer("kv_heads") : k.heads;
            k.scale = (float)v.number("scale");
            REQUIRE(k.heads >= 1 && k.dim >= 1 && k.vdim >= 1, B200RWKV_ERR_INVALID, "config: bad mixer sizes");
            REQUIRE(k.kv_heads >= 1 && k.heads % k.kv_heads == 0, B200RWKV_ERR_INVALID, "config: heads must be a multiple of kv_heads");
        };
        if (type == "attention") {
            k.mixer = KX_BIAS_WINDOW;
            heads(m);
            k.bias_max = m.number("bias_max");
            k.window = m.at("mask").integer("size");
            k.keep_first = m.at("mask").has("keep_first") ? m.at("mask").integer("keep_first") : 0;
            REQUIRE(k.window >= 1, B200RWKV_ERR_INVALID, "config: mask.size must be >= 1");
            if (m.has("kv_from")) {
                k.kv_from = m.integer("kv_from");
                REQUIRE(k.kv_from < (int)c.layers.size(), B200RWKV_ERR_INVALID, "config: kv_from must name an earlier layer");
                const KxLayerCfg& s = c.layers[k.kv_from];
                REQUIRE(s.mixer == KX_BIAS_WINDOW && s.kv_from < 0 && s.kv_heads == k.kv_heads && s.dim == k.dim && s.vdim == k.vdim, B200RWKV_ERR_INVALID,
                        "config: kv_from must name an attention layer with keys and values of its own and the same sizes");
            }
        } else if (type == "parallel") {
            k.mixer = KX_CHUNK_GLA;
            const JVal &a = m.at("left"), &b = m.at("right");
            heads(a);
            k.chunk = a.at("mask").integer("size");
            REQUIRE(k.chunk >= 1, B200RWKV_ERR_INVALID, "config: mask.size must be >= 1");
            if (a.has("rot")) {
                const JVal& r = a.at("rot");
                k.rot.dims = r.integer("dims"); k.rot.base = r.number("base");
                REQUIRE(k.rot.dims % 2 == 0 && k.rot.dims <= k.dim, B200RWKV_ERR_INVALID, "config: rot.dims must be even and <= dim");
                if (r.has("scaling")) {
                    const JVal& s = r.at("scaling");
                    k.rot.scaled = true;
                    k.rot.factor = s.number("factor"); k.rot.original = s.number("original");
                    k.rot.fast = s.number("fast"); k.rot.slow = s.number("slow");
                    REQUIRE(k.rot.factor > 0 && k.rot.original > 0 && k.rot.fast > 0 && k.rot.slow > 0, B200RWKV_ERR_INVALID,
                            "config: rot.scaling entries must be positive");
                }
            }
            k.mm_heads = b.integer("heads"); k.mm_dim = b.integer("dim");
            k.mm_vdim = b.has("vdim") ? b.integer("vdim") : k.mm_dim;
            k.tau = (float)b.number("tau");
            REQUIRE(k.mm_heads >= 1 && k.mm_dim >= 1 && k.mm_vdim >= 1 && k.tau > 0.f, B200RWKV_ERR_INVALID, "config: bad mixer sizes");
        } else {
            throw Error(B200RWKV_ERR_UNSUPPORTED, "config: unknown layer type '" + type + "'");
        }
        if (l.has("mlp")) {
            const JVal& f = l.at("mlp");
            REQUIRE(f.at("kind").str == "dense", B200RWKV_ERR_UNSUPPORTED, "config: unknown mlp kind '" + f.at("kind").str + "'");
            k.has_mlp = k.mlp_dense = true;
            k.ff = f.integer("ff");
            REQUIRE(k.ff >= 1, B200RWKV_ERR_INVALID, "config: mlp.ff must be >= 1");
        }
        c.layers.push_back(k);
    }
    return c;
}

}  // namespace b200
