// The Buguzen decoder's config.json, and the model it describes as data.
//
// Keys: "architecture": "Buguzen"; "vocab", "width"; "norm": {"eps"}; "layers": a list, each {"type": "attention" | "attention_2" |
// "lightning", "mixer": {...}, "mlp": {...} | null}; optional "loop": {"start", "stop", "times"}; optional "token_side": {"dim"}.
//   attention mixer    {"heads", "kv_heads", "dim", "vdim", "scale", "diff", "mask": {"size"}, "rot": {"base", "dims", "scaling": {"factor"}}}
//   attention_2 mixer  {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims", "scaling": {"factor", "low",
//                      "high", "original"}}}
//   lightning mixer    {"heads", "dim", "vdim", "decay": [per head]}
//   mlp                {"kind": "dense", "ff"}
// mask, rot, rot.scaling, mlp, loop and token_side are each left out (or null) by a model that has none.
// Every size and constant above comes from the file.  What the design itself fixes is written here once: layers are pre-norm,
// x += mixer(norm1(x)), x += ff(norm2(x)), with plain RMS norms, and then add a token input (a slice of a second embedding table,
// gated by the stream, projected and normalised); "attention" is differential (two maps over the same values, subtracted and
// normalised), with biases on q, k and v and adjacent rotary pairs whose frequencies may be divided by a factor; "attention_2" takes its
// keys, as projected, for values, normalises q and k per head, rotates pairs (i, i + dims / 2), whose frequencies may be slowed between
// two wavelengths (llama3), and has a learned sink per head; "lightning" is linear attention with a fixed decay per head, silu on
// q, k and v, one norm over all heads and a sigmoid gate; the feed-forward is gated by max(., 0); the head is a matrix of its own.
// With "loop", layers start .. stop - 1 run `times` times in a row, every pass with caches and states of its own, and in front of
// pass t (the first too) row t of a table is added to the stream.
// Tensor names: embed, head, final.norm, loop.step, side.embed, l<i>.norm1, l<i>.norm2, l<i>.mix.{q,k,v,g,o}(.b), l<i>.mix.{lq1,lk1,lq2,
// lk2}, l<i>.mix.{q,k}.norm, l<i>.mix.sink, l<i>.mix.norm, l<i>.mlp.{gate,up,down}, l<i>.side.{gate,proj,norm}.
#include <cmath>

#include "config.hpp"

namespace fg {

static const std::string kBuguzenName = "Buguzen";

static const Json *object_or_absent(const Json &d, const std::string &key, const std::string &where) {
    const Json *v = d.find(key);
    if (!v || v->is_null()) return nullptr;
    if (!v->is_object()) fail(FG_E_CONFIG, where + ": '" + key + "' must be an object");
    return v;
}

class BuguzenConfig : public ModelConfig {
public:
    enum Kind { Differential, KeysAsValues, Lightning };
    struct Layer {
        Kind kind = Differential;
        std::string type;
        long long heads = 0, kv_heads = 0, dim = 0, vdim = 0, window = 0;
        double scale = 0.0, diff = 0.0;
        bool rotates = false, scaled = false;
        double rot_base = 0.0, factor = 1.0, low = 0.0, high = 0.0, original = 0.0;
        long long rot_dims = 0;
        std::vector<double> decay;
        long long ff = 0;                       // 0: no feed-forward
    };
    struct Run {
        long long layer;
        long long pass;                         // >= 0: the pass that begins in front of this entry
    };
    Json source;
    long long vocab = 0, width = 0, side_dim = 0;
    double eps = 0.0;
    bool loops = false;
    long long loop_start = 0, loop_stop = 0, loop_times = 1;
    std::vector<Layer> layers;

    static void read_attention(const Json &m, Layer &y, const std::string &wm) {
        y.kv_heads = take_int(m, "kv_heads", y.heads, wm.c_str());
        if (y.kv_heads <= 0 || y.heads % y.kv_heads)
            fail(FG_E_CONFIG, wm + format(": heads (%lld) must be a multiple of kv_heads (%lld)", y.heads, y.kv_heads));
        y.scale = take_float(m, "scale", 1.0 / std::sqrt((double)y.dim), wm.c_str());
        if (!(y.scale > 0.0)) fail(FG_E_CONFIG, wm + format(": scale must be positive, got %g", y.scale));
        if (y.kind == Differential) y.diff = take_float(m, "diff", wm.c_str());
        if (y.kind == KeysAsValues && y.vdim != y.dim)
            fail(FG_E_CONFIG, wm + format(": the values are the keys, so vdim (%lld) must be dim (%lld)", y.vdim, y.dim));
        if (const Json *mask = object_or_absent(m, "mask", wm)) {
            y.window = take_int(*mask, "size", (wm + ".mask").c_str());
            if (y.window <= 0) fail(FG_E_CONFIG, wm + ".mask: size must be positive");
        }
        const Json *rot = object_or_absent(m, "rot", wm);
        if (!rot) return;
        const std::string wr = wm + ".rot", ws = wr + ".scaling";
        y.rotates = true;
        y.rot_base = take_float(*rot, "base", wr.c_str());
        if (!(y.rot_base > 0.0)) fail(FG_E_CONFIG, wr + ": base must be positive");
        y.rot_dims = take_int(*rot, "dims", y.dim, wr.c_str());
        if (y.rot_dims <= 0 || y.rot_dims % 2 || y.rot_dims > y.dim)
            fail(FG_E_CONFIG, wr + format(": dims must be even, positive and at most dim, got %lld", y.rot_dims));
        if (y.dim % 2) fail(FG_E_CONFIG, wm + format(": a rotated head needs an even dim, got %lld", y.dim));
        const Json *sc = object_or_absent(*rot, "scaling", wr);
        if (!sc) return;
        y.scaled = true;
        y.factor = take_float(*sc, "factor", ws.c_str());
        if (!(y.factor > 0.0)) fail(FG_E_CONFIG, ws + ": factor must be positive");
        if (y.kind != KeysAsValues) return;
        y.low = take_float(*sc, "low", ws.c_str());
        y.high = take_float(*sc, "high", ws.c_str());
        y.original = take_float(*sc, "original", ws.c_str());
        if (!(y.low > 0.0) || !(y.high > 0.0) || !(y.original > 0.0)) fail(FG_E_CONFIG, ws + ": every number must be positive");
    }

    static Layer read_layer(const Json &l, const std::string &w) {
        if (!l.is_object()) fail(FG_E_CONFIG, w + " must be an object");
        Layer y;
        y.type = take_string(l, "type", "", w.c_str());
        if (y.type == "attention") y.kind = Differential;
        else if (y.type == "attention_2") y.kind = KeysAsValues;
        else if (y.type == "lightning") y.kind = Lightning;
        else fail(FG_E_CONFIG, w + ": type '" + y.type + "' is not known (known: attention, attention_2, lightning)");
        const Json *m = object_or_absent(l, "mixer", w);
        if (!m) fail(FG_E_CONFIG, w + ": 'mixer' must be an object");
        const std::string wm = w + ".mixer";
        y.heads = take_int(*m, "heads", wm.c_str());
        y.dim = take_int(*m, "dim", wm.c_str());
        y.vdim = take_int(*m, "vdim", y.dim, wm.c_str());
        if (y.heads <= 0 || y.dim <= 0 || y.vdim <= 0) fail(FG_E_CONFIG, wm + ": heads, dim and vdim must be positive");
        if (y.kind == Lightning) {
            const Json *dl = m->find("decay");
            if (!dl || !dl->is_array() || (long long)dl->size() != y.heads)
                fail(FG_E_CONFIG, wm + format(": 'decay' must list one number for each of the %lld heads", y.heads));
            for (auto &v : dl->items()) {
                if (!v.is_number() || v.is_bool() || !(v.as_double() >= 0.0) || !(v.as_double() <= 1.0))
                    fail(FG_E_CONFIG, wm + ": a decay must be a number in [0, 1], got " + json_repr(v));
                y.decay.push_back(v.as_double());
            }
        } else read_attention(*m, y, wm);
        if (const Json *mlp = object_or_absent(l, "mlp", w)) {
            const std::string wf = w + ".mlp", kind = take_string(*mlp, "kind", "dense", wf.c_str());
            if (kind != "dense") fail(FG_E_CONFIG, wf + ": kind '" + kind + "' is not known (known: dense)");
            y.ff = take_int(*mlp, "ff", wf.c_str());
            if (y.ff <= 0) fail(FG_E_CONFIG, wf + ": ff must be positive");
        }
        return y;
    }

    static std::unique_ptr<ModelConfig> from_json(const Json &d) {
        auto cfg = std::make_unique<BuguzenConfig>();
        BuguzenConfig &c = *cfg;
        c.source = d;
        c.vocab = take_int(d, "vocab");
        c.width = take_int(d, "width");
        const Json *norm = object_or_absent(d, "norm", "config.json");
        if (!norm) fail(FG_E_CONFIG, "config.json: 'norm' must be an object");
        c.eps = take_float(*norm, "eps", "config.json norm");
        if (c.vocab <= 0 || c.width <= 0) fail(FG_E_CONFIG, "config.json: vocab and width must be positive");
        if (!(c.eps > 0.0)) fail(FG_E_CONFIG, format("config.json: norm.eps must be positive, got %g", c.eps));
        if (const Json *side = object_or_absent(d, "token_side", "config.json")) {
            c.side_dim = take_int(*side, "dim", "config.json token_side");
            if (c.side_dim <= 0) fail(FG_E_CONFIG, "config.json token_side: dim must be positive");
        }
        const Json *ls = d.find("layers");
        if (!ls || !ls->is_array() || ls->size() == 0) fail(FG_E_CONFIG, "config.json: 'layers' must be a non-empty list");
        for (size_t i = 0; i < ls->size(); i++) c.layers.push_back(read_layer((*ls)[i], format("config.json layers[%zu]", i)));
        if (const Json *loop = object_or_absent(d, "loop", "config.json")) {
            c.loops = true;
            c.loop_start = take_int(*loop, "start", "config.json loop");
            c.loop_stop = take_int(*loop, "stop", "config.json loop");
            c.loop_times = take_int(*loop, "times", "config.json loop");
            if (c.loop_start < 0 || c.loop_stop <= c.loop_start || c.loop_stop > (long long)c.layers.size() || c.loop_times < 1)
                fail(FG_E_CONFIG, format("config.json loop: need 0 <= start < stop <= %zu and times >= 1", c.layers.size()));
        }
        return cfg;
    }

    // the layers in the order they run
    std::vector<Run> order() const {
        std::vector<Run> o;
        const long long n = (long long)layers.size(), a = loops ? loop_start : n, b = loops ? loop_stop : n;
        for (long long i = 0; i < a; i++) o.push_back({i, -1});
        for (long long t = 0; loops && t < loop_times; t++)
            for (long long i = a; i < b; i++) o.push_back({i, i == a ? t : -1});
        for (long long i = b; i < n; i++) o.push_back({i, -1});
        return o;
    }
    long long layer_parameters(const Layer &y) const {
        const long long Q = y.heads * y.dim, V = y.heads * y.vdim;
        long long n = width;                                                        // norm1
        if (y.kind == Differential) n += (2 * Q + y.kv_heads * (2 * y.dim + y.vdim)) * (width + 1) + 4 * y.dim + V * width;
        if (y.kind == KeysAsValues) n += (Q + y.kv_heads * y.dim) * (width + 1) + 2 * y.dim + y.heads + V * width;
        if (y.kind == Lightning) n += (2 * Q + 2 * V) * width + V + V * width;
        if (y.ff > 0) n += width + 3 * width * y.ff;
        if (side_dim > 0) n += 2 * width * side_dim + width;
        return n;
    }
    long long parameter_count() const {
        long long n = 2 * vocab * width + width + (loops ? loop_times * width : 0) + vocab * side_dim * (long long)layers.size();
        for (auto &y : layers) n += layer_parameters(y);
        return n;
    }

    const std::string &architecture() const override { return kBuguzenName; }
    Json to_json() const override { return source; }

    Json describe() const override {
        Json d = Json::object();
        d.set("vocab_size", vocab);
        d.set("hidden_size", width);
        d.set("num_hidden_layers", (long long)layers.size());
        d.set("layer_runs", (long long)order().size());
        d.set("norm_eps", eps);
        long long kv_numbers = 0, state_floats = 0;
        Json kinds = Json::array();
        for (auto &y : layers) kinds.push(y.type + "+" + (y.ff > 0 ? "dense" : "none"));
        for (auto &run : order()) {
            const Layer &y = layers[(size_t)run.layer];
            if (y.kind == Lightning) state_floats += y.heads * y.dim * y.vdim;
            else kv_numbers += y.kv_heads * ((y.kind == Differential ? 2 : 1) * y.dim + y.vdim);
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

static Json part(const char *kind, Json params, Json tensors = Json::object()) {
    Json p = Json::object();
    p.set("kind", kind);
    p.set("params", std::move(params));
    p.set("tensors", std::move(tensors));
    return p;
}

static Json rotation(const BuguzenConfig::Layer &y) {
    if (!y.rotates) return Json();
    Json rp = Json::object();
    rp.set("head_dim", y.dim);
    rp.set("theta", y.rot_base);
    rp.set("rotary_dim", y.rot_dims);
    rp.set("layout", y.kind == BuguzenConfig::Differential ? "adjacent" : "halves");
    Json sc;
    if (y.scaled) {
        sc = Json::object();
        sc.set("rope_type", y.kind == BuguzenConfig::Differential ? "linear" : "llama3");
        sc.set("factor", y.factor);
        if (y.kind == BuguzenConfig::KeysAsValues) {
            sc.set("low_freq_factor", y.low);
            sc.set("high_freq_factor", y.high);
            sc.set("original_max_position_embeddings", y.original);
        }
    }
    rp.set("scaling", sc);
    return part("rope", rp);
}

Json BuguzenConfig::spec() const {
    auto norm = [&](const std::string &name) {
        Json p = Json::object();
        p.set("size", width);
        p.set("eps", eps);
        Json t = Json::object();
        t.set("weight", name);
        return part("rmsnorm", p, t);
    };
    auto mixer = [&](const Layer &y, const std::string &mx) {
        Json mp = Json::object(), mt = Json::object();
        mp.set("hidden_size", width);
        mp.set("n_heads", y.heads);
        mp.set("head_dim", y.dim);
        mp.set("v_head_dim", y.vdim);
        mp.set("eps", eps);
        for (const char *n : {"q", "k", "o"}) mt.set(std::string(n) + "_proj.weight", mx + n);
        if (y.kind != KeysAsValues) mt.set("v_proj.weight", mx + "v");
        if (y.kind == Lightning) {
            Json dl = Json::array();
            for (double v : y.decay) dl.push(Json(v));
            mp.set("decay", dl);
            mp.set("k_scale", 1.0);
            mp.set("position", Json());
            mp.set("qkv_activation", "silu");
            mp.set("norm", "whole");
            mp.set("gate_activation", "sigmoid");
            mt.set("g_proj.weight", mx + "g");
            mt.set("norm.weight", mx + "norm");
            return part("retention", mp, mt);
        }
        mp.set("n_kv_heads", y.kv_heads);
        mp.set("scale", y.scale);
        mp.set("window", y.window);
        mp.set("bias", true);
        mp.set("position", rotation(y));
        for (const char *n : {"q", "k", "v"})
            if (n[0] != 'v' || y.kind == Differential) mt.set(std::string(n) + "_proj.bias", mx + n + ".b");
        if (y.kind == Differential) {
            mp.set("differential", y.diff);
            for (const char *n : {"q1", "k1", "q2", "k2"}) mt.set(std::string("lambda_") + n, mx + "l" + n);
        } else {
            mp.set("values", "keys");
            mp.set("qk_norm", "head");
            mp.set("sink", true);
            mt.set("q_norm.weight", mx + "q.norm");
            mt.set("k_norm.weight", mx + "k.norm");
            mt.set("sinks", mx + "sink");
        }
        return part("sink_attention", mp, mt);
    };
    Json ls = Json::array(), schedule = Json::array();
    for (size_t i = 0; i < layers.size(); i++) {
        const Layer &y = layers[i];
        const std::string pre = format("l%zu.", i);
        Json layer = Json::object();
        layer.set("block", "prenorm");
        layer.set("mixer", mixer(y, pre + "mix."));
        layer.set("mixer_norm", norm(pre + "norm1"));
        if (y.ff > 0) {
            Json fp = Json::object(), ft = Json::object();
            fp.set("hidden_size", width);
            fp.set("d_ff", y.ff);
            fp.set("activation", "relu");
            for (const char *n : {"gate", "up", "down"}) ft.set(std::string(n) + "_proj.weight", pre + "mlp." + n);
            layer.set("feed_forward", part("swiglu", fp, ft));
            layer.set("feed_forward_norm", norm(pre + "norm2"));
        } else layer.set("feed_forward", Json());
        if (side_dim > 0) {
            Json sp = Json::object(), st = Json::object();
            sp.set("hidden_size", width);
            sp.set("vocab_size", vocab);
            sp.set("dim", side_dim);
            sp.set("column", side_dim * (long long)i);
            sp.set("table_dim", side_dim * (long long)layers.size());
            sp.set("eps", eps);
            st.set("table", "side.embed");
            st.set("gate", pre + "side.gate");
            st.set("proj", pre + "side.proj");
            st.set("norm", pre + "side.norm");
            layer.set("token_input", part("gated_token_embedding", sp, st));
        }
        ls.push(layer);
    }
    for (auto &run : order()) {
        Json r = Json::object();
        r.set("layer", run.layer);
        r.set("cache_from", Json());
        if (run.pass >= 0) {
            r.set("reenter", true);
            r.set("pass", run.pass);
        }
        schedule.push(r);
    }
    Json ep = Json::object(), hp = Json::object(), et = Json::object(), ht = Json::object();
    ep.set("vocab_size", vocab);
    ep.set("hidden_size", width);
    hp.set("vocab_size", vocab);
    hp.set("hidden_size", width);
    et.set("weight", "embed");
    ht.set("weight", "head");
    Json s = Json::object();
    s.set("hidden_size", width);
    s.set("vocab_size", vocab);
    s.set("max_positions", 1LL << 20);          // the design has no longest sequence; tables are built for what the cache holds
    s.set("embedding", part("embedding", ep, et));
    s.set("layers", ls);
    s.set("schedule", schedule);
    if (loops) {
        Json rp = Json::object(), rt = Json::object();
        rp.set("hidden_size", width);
        rp.set("rows", loop_times);
        rt.set("table", "loop.step");
        s.set("reentry", part("add_row", rp, rt));
    }
    s.set("final_norm", norm("final.norm"));
    s.set("head", part("lm_head", hp, ht));
    s.set("stop_token_ids", Json::array());
    s.set("ignored_tensors", Json::array());
    return s;
}

std::unique_ptr<ModelConfig> buguzen_config_from_json(const Json &d) { return BuguzenConfig::from_json(d); }

}  // namespace fg
