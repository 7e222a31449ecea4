// Panupel model family: blocks with a norm on both sides of every sublayer,
//     x += r N1b(Mixer(N1(x)));   x += r N2b(FF(N2(x)))          (r: residual_mult; RMS norms with plain weights; FF may be absent)
// A run of consecutive layers (`loop`: start, stop, times) is executed `times` times with the same tensors and sequence memory of
// its own per pass; every pass begins with x <- W_in [x; embedding row of the token].
// Mixers: "parallel" = two mixers on the same input, their outputs added with two constants: causal softmax attention over the
// whole context (norm of the whole query / key projection, half-split rotation with banded frequencies, a sink term per head, one
// sigmoid gate per head; sink_attn.cuh) beside a matrix memory (matrix_memory.cuh);  "delta" = gated delta rule with one decay per
// head behind short causal convolutions, silu output gate (delta_rule.cuh).
// Feed-forward: W_down (silu(W_gate h) * (W_up h)).
// Every size and constant that can differ between models comes from config.json / the tensor shapes.  The family shares the
// sequence-model engine of the Kemirax family (kemirax.cuh: configuration structs, slot / page / snapshot plumbing); this file
// reads its configuration.
#pragma once

namespace b200 {

static KxConfig pn_parse_config(const JVal& root) {
    KxConfig c;
    c.family = KX_FAMILY_PANUPEL;
    c.vocab = root.integer("vocab");
    c.width = root.integer("width");
    c.eps = (float)root.at("norm").number("eps");
    c.residual_mul = root.has("residual_mult") ? (float)root.number("residual_mult") : 1.f;
    const JVal& ls = root.at("layers");
    REQUIRE(ls.kind == JVal::ARR && !ls.arr.empty(), B200RWKV_ERR_INVALID, "config: layers");
    std::vector<KxLayerCfg> own;
    for (const JVal& l : ls.arr) {
        KxLayerCfg k;
        REQUIRE(l.kind == JVal::OBJ && l.has("type") && l.at("type").kind == JVal::STR, B200RWKV_ERR_INVALID, "config: layer without a type");
        const std::string type = l.at("type").str;
        const JVal& m = l.at("mixer");
        auto heads = [&](const JVal& v) {
            k.heads = v.integer("heads"); k.dim = v.integer("dim");
            k.vdim = v.has("vdim") ? v.integer("vdim") : k.dim;
            k.kv_heads = v.has("kv_heads") ? v.integer("kv_heads") : k.heads;
            REQUIRE(k.heads >= 1 && k.dim >= 1 && k.vdim >= 1, B200RWKV_ERR_INVALID, "config: bad mixer sizes");
            REQUIRE(k.kv_heads >= 1 && k.heads % k.kv_heads == 0, B200RWKV_ERR_INVALID, "config: heads must be a multiple of kv_heads");
        };
        if (type == "parallel") {
            k.mixer = KX_PARALLEL;
            const JVal &a = m.at("left"), &b = m.at("right");
            heads(a);
            k.scale = (float)a.number("scale");
            if (a.has("rot")) {
                const JVal& r = a.at("rot");
                k.rot.dims = r.integer("dims"); k.rot.base = r.number("base");
                REQUIRE(k.rot.dims % 2 == 0 && k.rot.dims <= k.dim, B200RWKV_ERR_INVALID, "config: rot.dims must be even and <= dim");
                if (r.has("scaling")) {
                    const JVal& s = r.at("scaling");
                    k.rot.banded = true;
                    k.rot.factor = s.number("factor"); k.rot.original = s.number("original");
                    k.rot.low = s.number("low"); k.rot.high = s.number("high");
                    REQUIRE(k.rot.factor > 0 && k.rot.original > 0 && k.rot.low > 0 && k.rot.high > 0, B200RWKV_ERR_INVALID,
                            "config: rot.scaling entries must be positive");
                }
            }
            k.mm_heads = b.integer("heads"); k.mm_dim = b.integer("dim");
            k.mm_vdim = b.has("vdim") ? b.integer("vdim") : k.mm_dim;
            k.mm_cap = (float)b.number("gate_cap");
            REQUIRE(k.mm_heads >= 1 && k.mm_dim >= 1 && k.mm_vdim >= 1 && k.mm_cap > 0.f, B200RWKV_ERR_INVALID, "config: bad mixer sizes");
            k.attn_mul = (float)m.number("left_scale"); k.mm_mul = (float)m.number("right_scale");
        } else if (type == "delta") {
            k.mixer = KX_DELTA;
            k.head_decay = true;
            heads(m);
            k.taps = m.integer("conv");
            REQUIRE(k.taps >= 1, B200RWKV_ERR_INVALID, "config: conv must be >= 1");
        } else {
            throw Error(B200RWKV_ERR_UNSUPPORTED, "config: unknown layer type '" + type + "'");
        }
        if (l.has("mlp")) {
            const JVal& f = l.at("mlp");
            REQUIRE(f.at("kind").str == "dense", B200RWKV_ERR_UNSUPPORTED, "config: unknown mlp kind '" + f.at("kind").str + "'");
            k.has_mlp = k.mlp_dense = true;
            k.ff = f.integer("ff");
        }
        own.push_back(k);
    }
    kx_unroll_loop(root, own, c);
    return c;
}

}  // namespace b200
