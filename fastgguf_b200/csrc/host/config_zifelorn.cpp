// The Zifelorn decoder's config.json, and the model it describes as data.
//
// Keys: "architecture": "Zifelorn"; "vocab", "width"; "embedding": {"scale"}; "norm": {"eps"}; "logit_scale"; "layers": a list, each
// {"type": "latent_attention" | "rglru", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | {"kind": "moe", "expert": {"ff"},
// "router": {"experts", "top"}} | null}.
//   latent_attention mixer  {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {"base", "dims"}, "kv_from": j}
//                           - with kv_from the layer has no key/value latent of its own and reads layer j's
//   rglru mixer             {"width", "blocks", "conv": taps}
// Every size and constant above comes from the file.  What the design itself fixes is written here once: a layer is
// x += norm1(mixer(x)), x += norm2(ff(x)), no norm in front; norms multiply by their weight as stored; latent attention rotates
// adjacent pairs, has an ordinary softmax and a sigmoid gate per number on the heads' outputs; the recurrent unit's rate is
// 8 softplus(lam); the dense feed-forward gates with the tanh form of gelu; experts are W_down max(W_up x, 0)^2, the router's
// weights the softmax over the chosen logits; the head is the embedding table without its scale, the logits times logit_scale.
// Tensor names: embed, final.norm, l<i>.norm1 / norm2, l<i>.mix.*, l<i>.mlp.gate / up / down, l<i>.mlp.router (+ .b),
// l<i>.mlp.e<k>.up / down.
#include <cmath>

#include "config.hpp"

namespace fg {

static const std::string kZifelornName = "Zifelorn";
static const double kZifelornGain = 8.0;             // log a = -8 r softplus(lam)

static const Json *zifelorn_object(const Json &d, const std::string &key, const std::string &where, bool required) {
    const Json *v = d.find(key);
    if (!v || v->is_null()) {
        if (required) fail(FG_E_CONFIG, where + ": '" + key + "' must be an object");
        return nullptr;
    }
    if (!v->is_object()) fail(FG_E_CONFIG, where + ": '" + key + "' must be an object");
    return v;
}

class ZifelornConfig : public ModelConfig {
public:
    struct Layer {
        bool latent = false;
        long long heads = 0, dim = 0, vdim = 0, rot_dim = 0, kv_rank = 0, q_rank = 0, kv_from = -1;      // latent attention
        double scale = 0, base = 0;
        long long width = 0, blocks = 1, taps = 1;                                                       // recurrent block
        long long ff = 0, experts = 0, top = 0;          // experts 0: dense; ff 0: no feed-forward
    };
    Json source;
    long long vocab = 0, width = 0;
    double eps = 0.0, embed_scale = 1.0, logit_scale = 1.0;
    std::vector<Layer> layers;

    static std::unique_ptr<ModelConfig> from_json(const Json &d) {
        auto cfg = std::make_unique<ZifelornConfig>();
        ZifelornConfig &c = *cfg;
        c.source = d;
        c.vocab = take_int(d, "vocab");
        c.width = take_int(d, "width");
        const Json *norm = zifelorn_object(d, "norm", "config.json", true);
        c.eps = take_float(*norm, "eps", "config.json norm");
        if (c.vocab <= 0 || c.width <= 0) fail(FG_E_CONFIG, "config.json: vocab and width must be positive");
        if (!(c.eps > 0.0)) fail(FG_E_CONFIG, format("config.json: norm.eps must be positive, got %g", c.eps));
        if (const Json *e = zifelorn_object(d, "embedding", "config.json", false)) c.embed_scale = take_float(*e, "scale", 1.0, "config.json embedding");
        c.logit_scale = take_float(d, "logit_scale", 1.0);
        if (!std::isfinite(c.embed_scale) || !std::isfinite(c.logit_scale)) fail(FG_E_CONFIG, "config.json: embedding.scale and logit_scale must be finite");
        const Json *ls = d.find("layers");
        if (!ls || !ls->is_array() || ls->size() == 0) fail(FG_E_CONFIG, "config.json: 'layers' must be a non-empty list");
        for (size_t i = 0; i < ls->size(); i++) {
            const Json &l = (*ls)[i];
            const std::string w = format("config.json layers[%zu]", i);
            if (!l.is_object()) fail(FG_E_CONFIG, w + " must be an object");
            Layer y;
            const std::string type = take_string(l, "type", "", w.c_str());
            const Json &m = *zifelorn_object(l, "mixer", w, true);
            const std::string wm = w + ".mixer";
            if (type == "latent_attention") {
                y.latent = true;
                y.heads = take_int(m, "heads", wm.c_str());
                y.dim = take_int(m, "dim", wm.c_str());
                y.vdim = take_int(m, "vdim", y.dim, wm.c_str());
                y.rot_dim = take_int(m, "rot_dim", wm.c_str());
                y.kv_rank = take_int(m, "kv_rank", wm.c_str());
                y.q_rank = take_int(m, "q_rank", wm.c_str());
                if (y.heads <= 0 || y.dim <= 0 || y.vdim <= 0) fail(FG_E_CONFIG, wm + ": heads, dim and vdim must be positive");
                if (y.rot_dim <= 0 || y.rot_dim % 2 || y.kv_rank <= 0 || y.q_rank <= 0)
                    fail(FG_E_CONFIG, wm + ": rot_dim (even), kv_rank and q_rank must be positive");
                y.scale = take_float(m, "scale", 1.0 / std::sqrt((double)(y.dim + y.rot_dim)), wm.c_str());
                const Json &rot = *zifelorn_object(m, "rot", wm, true);
                y.base = take_float(rot, "base", (wm + ".rot").c_str());
                if (!(y.base > 0.0)) fail(FG_E_CONFIG, wm + ".rot: base must be positive");
                const long long dims = take_int(rot, "dims", y.rot_dim, (wm + ".rot").c_str());
                if (dims != y.rot_dim) fail(FG_E_CONFIG, wm + format(".rot: dims (%lld) must equal rot_dim (%lld)", dims, y.rot_dim));
                const Json *from = m.find("kv_from");
                if (from && !from->is_null()) {
                    y.kv_from = take_int(m, "kv_from", wm.c_str());
                    if (y.kv_from < 0 || y.kv_from >= (long long)i) fail(FG_E_CONFIG, wm + format(": kv_from must name an earlier layer, got %lld", y.kv_from));
                    const Layer &o = c.layers[(size_t)y.kv_from];
                    if (!o.latent || o.kv_from >= 0) fail(FG_E_CONFIG, wm + format(": kv_from names layer %lld, which keeps no latent of its own", y.kv_from));
                    if (o.kv_rank != y.kv_rank || o.rot_dim != y.rot_dim || o.base != y.base)
                        fail(FG_E_CONFIG, wm + format(": kv_rank, rot_dim and rot of layer %lld must equal this layer's", y.kv_from));
                }
            } else if (type == "rglru") {
                y.width = take_int(m, "width", wm.c_str());
                y.blocks = take_int(m, "blocks", 1, wm.c_str());
                y.taps = take_int(m, "conv", 1, wm.c_str());
                if (y.width <= 0 || y.blocks <= 0 || y.taps <= 0) fail(FG_E_CONFIG, wm + ": width, blocks and conv must be positive");
                if (y.width % y.blocks) fail(FG_E_CONFIG, wm + format(": width (%lld) must be a multiple of blocks (%lld)", y.width, y.blocks));
            } else {
                fail(FG_E_CONFIG, w + ": type '" + type + "' is not known (known: latent_attention, rglru)");
            }
            if (const Json *mlp = zifelorn_object(l, "mlp", w, false)) {
                const std::string wf = w + ".mlp";
                const std::string kind = take_string(*mlp, "kind", "dense", wf.c_str());
                if (kind == "dense") {
                    y.ff = take_int(*mlp, "ff", wf.c_str());
                } else if (kind == "moe") {
                    const Json &r = *zifelorn_object(*mlp, "router", wf, true);
                    y.ff = take_int(*zifelorn_object(*mlp, "expert", wf, true), "ff", (wf + ".expert").c_str());
                    y.experts = take_int(r, "experts", (wf + ".router").c_str());
                    y.top = take_int(r, "top", (wf + ".router").c_str());
                    if (y.experts <= 0 || y.top <= 0 || y.top > y.experts)
                        fail(FG_E_CONFIG, wf + format(".router: experts and top must be positive and top (%lld) at most experts (%lld)", y.top, y.experts));
                } else fail(FG_E_CONFIG, wf + ": kind '" + kind + "' is not known (known: dense, moe)");
                if (y.ff <= 0) fail(FG_E_CONFIG, wf + ": ff must be positive");
            }
            c.layers.push_back(std::move(y));
        }
        return cfg;
    }

    long long layer_parameters(const Layer &y) const {
        long long n = width + (y.ff ? width : 0);
        if (y.experts) n += y.experts * (2 * width * y.ff + width + 1);
        else n += 3 * width * y.ff;
        if (y.latent) {
            n += width * y.q_rank + y.q_rank + y.q_rank * y.heads * (y.dim + y.rot_dim) + y.kv_rank * y.heads * (y.dim + y.vdim) + 2 * width * y.heads * y.vdim;
            if (y.kv_from < 0) n += width * (y.kv_rank + y.rot_dim) + y.kv_rank;
        } else {
            n += 3 * width * y.width + 2 * y.width + y.width * (y.taps + 1) + 2 * y.width * (y.width / y.blocks) + 2 * y.width + y.width;
        }
        return n;
    }
    long long parameter_count() const {
        long long n = vocab * width + width;
        for (auto &y : layers) n += layer_parameters(y);
        return n;
    }

    const std::string &architecture() const override { return kZifelornName; }
    Json to_json() const override { return source; }

    Json describe() const override {
        Json d = Json::object();
        d.set("vocab_size", vocab);
        d.set("hidden_size", width);
        d.set("num_hidden_layers", (long long)layers.size());
        d.set("layer_runs", (long long)layers.size());
        d.set("norm_eps", eps);
        long long kv_numbers = 0, state_floats = 0;
        Json kinds = Json::array();
        for (auto &y : layers) {
            kinds.push(std::string(y.latent ? "latent_attention" : "rglru") + "+" + (y.experts ? "experts" : y.ff ? "dense" : "none"));
            if (y.latent) kv_numbers += y.kv_from < 0 ? y.kv_rank + y.rot_dim : 0;
            else state_floats += (y.taps > 1 ? y.taps + 1 : 1) * y.width;
        }
        d.set("layer_kinds", kinds);
        d.set("parameters", parameter_count());
        Json kvb = Json::object(), pb = Json::object();
        kvb.set("bfloat16", kv_numbers * 2);
        kvb.set("float32", kv_numbers * 4);
        pb.set("bfloat16", parameter_count() * 2);
        pb.set("float32", parameter_count() * 4);
        d.set("kv_bytes_per_token", kvb);
        d.set("parameter_bytes", pb);
        d.set("state_bytes_per_sequence", state_floats * 4);
        d.set("eos_token_ids", Json::array());
        d.set("defaulted", Json::array());
        return d;
    }

    Json spec() const override;
};

static Json zifelorn_part(const char *kind, Json params, Json tensors = Json::object()) {
    Json p = Json::object();
    p.set("kind", kind);
    p.set("params", std::move(params));
    p.set("tensors", std::move(tensors));
    return p;
}

Json ZifelornConfig::spec() const {
    auto norm = [&](const std::string &name, double gain) {
        Json p = Json::object();
        p.set("size", width);
        p.set("eps", eps);
        if (gain != 1.0) p.set("gain", gain);
        Json t = Json::object();
        t.set("weight", name);
        return zifelorn_part("rmsnorm", p, t);
    };
    Json ls = Json::array(), schedule = Json::array();
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        const std::string pre = format("l%zu.", i), mx = pre + "mix.", fx = pre + "mlp.";
        Json layer = Json::object(), mp = Json::object(), mt = Json::object();
        layer.set("block", "postnorm");
        mp.set("hidden_size", width);
        if (y.latent) {
            Json rp = Json::object();
            rp.set("head_dim", y.rot_dim);
            rp.set("theta", y.base);
            rp.set("rotary_dim", y.rot_dim);
            rp.set("layout", "adjacent");
            rp.set("scaling", Json());
            mp.set("n_heads", y.heads);
            mp.set("head_dim", y.dim);
            mp.set("v_head_dim", y.vdim);
            mp.set("eps", eps);
            mp.set("rot_dim", y.rot_dim);
            mp.set("kv_rank", y.kv_rank);
            mp.set("q_rank", y.q_rank);
            mp.set("scale", y.scale);
            mp.set("sink", false);
            mp.set("gate", true);
            mp.set("shared_kv", y.kv_from >= 0);
            mp.set("position", zifelorn_part("rope", rp));
            mt.set("q_down.weight", mx + "dq");
            mt.set("q_down_norm.weight", mx + "dq.norm");
            mt.set("q_up.weight", mx + "uq");
            if (y.kv_from < 0) {
                mt.set("kv_down.weight", mx + "dkv");
                mt.set("kv_down_norm.weight", mx + "dkv.norm");
            }
            mt.set("k_up.weight", mx + "uk");
            mt.set("v_up.weight", mx + "uv");
            mt.set("g_proj.weight", mx + "g");
            mt.set("o_proj.weight", mx + "o");
            layer.set("mixer", zifelorn_part("latent_attention", mp, mt));
        } else {
            mp.set("width", y.width);
            mp.set("n_blocks", y.blocks);
            mp.set("conv_taps", y.taps);
            mp.set("gain", kZifelornGain);
            for (const char *n : {"y", "x"}) {
                mt.set(std::string(n) + "_proj.weight", mx + n);
                mt.set(std::string(n) + "_proj.bias", mx + n + ".b");
            }
            mt.set("conv.weight", mx + "conv");
            mt.set("conv.bias", mx + "conv.b");
            for (const char *n : {"r", "i"}) {
                mt.set(std::string(n) + "_gate.weight", mx + "r" + (n[0] == 'r' ? "a" : "i"));
                mt.set(std::string(n) + "_gate.bias", mx + "r" + (n[0] == 'r' ? "a" : "i") + ".b");
            }
            mt.set("lam", mx + "lam");
            mt.set("o_proj.weight", mx + "o");
            layer.set("mixer", zifelorn_part("rglru", mp, mt));
        }
        layer.set("mixer_norm", Json());
        layer.set("mixer_post_norm", norm(pre + "norm1", 1.0));
        if (y.ff > 0) {
            Json fp = Json::object(), ft = Json::object();
            fp.set("hidden_size", width);
            fp.set("d_ff", y.ff);
            if (y.experts) {
                fp.set("n_experts", y.experts);
                fp.set("top_k", y.top);
                fp.set("router", "softmax_chosen");
                fp.set("activation", "relu2");
                ft.set("router.weight", fx + "router");
                ft.set("router.bias", fx + "router.b");
                for (long long e = 0; e < y.experts; e++)
                    for (const char *n : {"up", "down"}) ft.set(format("experts.%lld.%s_proj.weight", e, n), fx + format("e%lld.%s", e, n));
                layer.set("feed_forward", zifelorn_part("moe", fp, ft));
            } else {
                fp.set("activation", "gelu_tanh");
                for (const char *n : {"gate", "up", "down"}) ft.set(std::string(n) + "_proj.weight", fx + n);
                layer.set("feed_forward", zifelorn_part("swiglu", fp, ft));
            }
            layer.set("feed_forward_post_norm", norm(pre + "norm2", 1.0));
        } else layer.set("feed_forward", Json());
        ls.push(layer);
        Json r = Json::object();
        r.set("layer", (long long)i);
        r.set("cache_from", y.kv_from >= 0 ? Json(y.kv_from) : Json());
        schedule.push(r);
    }
    Json ep = Json::object(), hp = Json::object(), et = Json::object(), ht = Json::object();
    ep.set("vocab_size", vocab);
    ep.set("hidden_size", width);
    ep.set("scale", embed_scale);
    hp.set("vocab_size", vocab);
    hp.set("hidden_size", width);
    et.set("weight", "embed");
    ht.set("weight", "embed");
    Json s = Json::object();
    s.set("hidden_size", width);
    s.set("vocab_size", vocab);
    s.set("max_positions", 1LL << 20);          // the design has no longest sequence; tables are built for what the cache holds
    s.set("embedding", zifelorn_part("embedding", ep, et));
    s.set("layers", ls);
    s.set("schedule", schedule);
    s.set("final_norm", norm("final.norm", logit_scale));       // the logits' scale rides in the norm in front of the head
    s.set("head", zifelorn_part("lm_head", hp, ht));
    s.set("stop_token_ids", Json::array());
    s.set("ignored_tensors", Json::array());
    return s;
}

std::unique_ptr<ModelConfig> zifelorn_config_from_json(const Json &d) { return ZifelornConfig::from_json(d); }

}  // namespace fg
