/* vb_lm_config.cpp - config.json of the decoder language models (vb_lm_config.h). */
#include "vb_lm_config.h"

#include <math.h>

#include <algorithm>

namespace vb {

std::vector<double> LmRope::frequencies() const {
    std::vector<double> f((size_t)dims / 2);
    double lo = 0.0, hi = 0.0;
    if (yarn) {
        /* pair index whose wave makes t turns over the original context */
        auto pair_of = [&](double t) { return dims * log(original / (2.0 * M_PI * t)) / (2.0 * log(base)); };
        lo = std::max(floor(pair_of(fast)), 0.0);
        hi = std::min(ceil(pair_of(slow)), (double)dims - 1.0);
    }
    for (size_t i = 0; i < f.size(); i++) {
        f[i] = pow(base, -2.0 * (double)i / dims);
        if (yarn) {
            const double r = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            f[i] = f[i] / factor * r + f[i] * (1.0 - r);
        }
    }
    return f;
}

double LmRope::magnitude() const { return yarn ? 0.1 * log(factor) + 1.0 : 1.0; }

std::vector<LmConfig::Run> LmConfig::runs() const {
    std::vector<Run> r;
    const int n = (int)layers.size();
    const int a = loop_times > 0 ? loop_start : n, b = loop_times > 0 ? loop_stop : n;
    for (int i = 0; i < a; i++) r.push_back({i, false});
    for (int t = 0; t < loop_times; t++)
        for (int i = a; i < b; i++) r.push_back({i, i == a});
    for (int i = b; i < n; i++) r.push_back({i, false});
    return r;
}

int LmConfig::cache_window(int i) const {
    int w = layers[i].mixer.mask.window;
    for (const LmLayer &l : layers)
        if (l.mixer.kv_from == i) w = w > 0 && l.mixer.mask.window > 0 ? std::max(w, l.mixer.mask.window) : 0;
    return w;
}

namespace {

/* Reads members of one JSON object and keeps the first complaint. */
struct Fields {
    const Json *o;
    std::string where, *err;
    bool ok = true;

    bool complain(const char *key, const char *what) {
        if (ok && err->empty()) *err = "config.json: " + where + "." + key + " " + what;
        return ok = false;
    }
    double number(const char *key, bool required = true, double fallback = 0.0) {
        const Json *v = o ? o->get(key) : nullptr;
        if (!v) {
            if (required) complain(key, "is missing");
            return fallback;
        }
        if (v->kind != Json::NUMBER || !std::isfinite(v->number)) { complain(key, "is not a number"); return fallback; }
        return v->number;
    }
    int integer(const char *key, int lo, int hi, bool required = true, int fallback = 0) {
        const double v = number(key, required, fallback);
        if (!ok) return fallback;
        if (v != floor(v) || v < lo || v > hi) { complain(key, "is out of range"); return fallback; }
        return (int)v;
    }
};

constexpr int kMaxSize = 1 << 20;

bool read_mask(const Json *mix, const std::string &where, LmMask *mask, std::string *err) {
    const Json *o = mix->get("mask");
    if (!o) return true;
    Fields g{o, where + ".mixer.mask", err};
    mask->window = g.integer("size", 1, 1 << 30);
    mask->keep_first = g.integer("keep_first", 0, 1 << 30, false, 0);
    return g.ok;
}

bool read_rope(const Json *mix, const std::string &where, int dim, LmRope *rope, std::string *err) {
    const Json *rot = mix->get("rot");
    if (!rot) return true;
    Fields g{rot, where + ".mixer.rot", err};
    rope->dims = g.integer("dims", 0, dim);
    rope->base = g.number("base");
    if (g.ok && (rope->dims & 1)) g.complain("dims", "is odd");
    if (g.ok && rope->base <= 1.0) g.complain("base", "is not above 1");
    if (const Json *sc = rot->get("scaling")) {
        Fields s{sc, where + ".mixer.rot.scaling", err};
        rope->yarn = true;
        rope->factor = s.number("factor");
        rope->original = s.number("original");
        rope->fast = s.number("fast");
        rope->slow = s.number("slow");
        if (s.ok && !(rope->factor > 0 && rope->original > 0 && rope->fast > 0 && rope->slow > 0))
            s.complain("factor", "and its companions have to be positive");
        if (!s.ok) return false;
    }
    return g.ok;
}

bool mixer_of(const Json &layer, const std::string &where, const Json **type, const Json **mix, std::string *err) {
    *type = layer.get("type");
    *mix = layer.get("mixer");
    if (*type && (*type)->kind == Json::STRING && *mix && (*mix)->kind == Json::OBJECT) return true;
    *err = "config.json: " + where + " needs 'type' and 'mixer'";
    return false;
}

bool read_mixer(const Json &layer, const std::string &where, LmMixer *m, std::string *err) {
    const Json *type, *mix;
    if (!mixer_of(layer, where, &type, &mix, err)) return false;
    Fields f{mix, where + ".mixer", err};
    m->heads = f.integer("heads", 1, 65535);
    m->kv_heads = f.integer("kv_heads", 1, 65535, false, m->heads);
    m->dim = f.integer("dim", 1, kMaxSize);
    m->vdim = f.integer("vdim", 1, kMaxSize, false, m->dim);
    if (f.ok && m->heads % m->kv_heads) f.complain("kv_heads", "does not divide heads");
    if (type->text == "delta") {
        m->kind = LM_MIXER_DELTA;
        m->taps = f.integer("conv", 1, 64);
        return f.ok;
    }
    if (type->text != "attention") {
        *err = "config.json: " + where + ".type '" + type->text + "' is not a known mixer";
        return false;
    }
    m->kind = LM_MIXER_ATTENTION;
    m->scale = f.number("scale");
    m->softcap = f.number("softcap", false, 0.0);
    if (f.ok && m->softcap < 0.0) f.complain("softcap", "is negative");
    return read_mask(mix, where, &m->mask, err) && read_rope(mix, where, m->dim, &m->rope, err) && f.ok;
}

/* vocab, width, norm.eps and the list of layers, each read by `layer`. */
bool read_stack(const Json &c, LmConfig *out, std::string *err,
                bool (*layer)(const Json &, const std::string &where, LmLayer *, std::string *err)) {
    Fields f{&c, "model", err};
    out->vocab = f.integer("vocab", 1, 1 << 26);
    out->width = f.integer("width", 1, kMaxSize);
    const Json *norm = c.get("norm");
    Fields n{norm, "norm", err};
    out->eps = n.number("eps");
    const Json *layers = c.get("layers");
    if (!f.ok || !n.ok) return false;
    if (!layers || layers->kind != Json::ARRAY || layers->items.empty()) {
        *err = "config.json: 'layers' has to list at least one layer";
        return false;
    }
    for (size_t i = 0; i < layers->items.size(); i++) {
        LmLayer l;
        if (!layer(layers->items[i], "layers[" + std::to_string(i) + "]", &l, err)) return false;
        out->layers.push_back(l);
    }
    return true;
}

bool read_kegizen_layer(const Json &layer, const std::string &where, LmLayer *l, std::string *err) {
    if (!read_mixer(layer, where, &l->mixer, err)) return false;
    const Json *mlp = layer.get("mlp");
    if (!mlp) return true;
    const Json *kind = mlp->get("kind");
    if (kind && (kind->kind != Json::STRING || kind->text != "dense")) {
        *err = "config.json: " + where + ".mlp.kind is not known";
        return false;
    }
    Fields m{mlp, where + ".mlp", err};
    l->mlp.kind = LM_MLP_SWIGLU;
    l->mlp.ff = m.integer("ff", 1, kMaxSize);
    return m.ok;
}

bool read_kegizen(const Json &c, LmConfig *out, std::string *err) {
    if (!read_stack(c, out, err, read_kegizen_layer)) return false;
    if (const Json *loop = c.get("loop")) {
        Fields l{loop, "loop", err};
        const int nl = (int)out->layers.size();
        out->loop_start = l.integer("start", 0, nl - 1);
        out->loop_stop = l.integer("stop", out->loop_start + 1, nl);
        out->loop_times = l.integer("times", 1, 4096);
        if (!l.ok) return false;
    }
    return true;
}

bool read_bupozen_layer(const Json &layer, const std::string &where, LmLayer *l, std::string *err) {
    const Json *type, *mix;
    if (!mixer_of(layer, where, &type, &mix, err)) return false;
    if (type->text != "latent_attention") {
        *err = "config.json: " + where + ".type '" + type->text + "' is not a known mixer";
        return false;
    }
    LmMixer *m = &l->mixer;
    Fields f{mix, where + ".mixer", err};
    m->kind = LM_MIXER_LATENT;
    m->heads = f.integer("heads", 1, 65535);
    m->kv_heads = m->heads;
    m->dim = f.integer("dim", 1, kMaxSize);
    m->rot_dim = f.integer("rot_dim", 0, kMaxSize);
    m->vdim = f.integer("vdim", 1, kMaxSize);
    m->q_rank = f.integer("q_rank", 1, kMaxSize);
    m->kv_rank = f.integer("kv_rank", 1, kMaxSize);
    m->scale = f.number("scale");
    if (mix->get("kv_from")) m->kv_from = f.integer("kv_from", 0, kMaxSize);
    if (!f.ok || !read_mask(mix, where, &m->mask, err) || !read_rope(mix, where, m->rot_dim, &m->rope, err)) return false;
    const Json *mlp = layer.get("mlp");
    if (!mlp) return true;
    const Json *kind = mlp->get("kind");
    const bool moe = kind && kind->kind == Json::STRING && kind->text == "moe";
    if (!moe && !(kind && kind->kind == Json::STRING && kind->text == "dense")) {
        *err = "config.json: " + where + ".mlp.kind is not known";
        return false;
    }
    l->mlp.kind = LM_MLP_RELU2;
    Fields s{moe ? mlp->get("expert") : mlp, where + (moe ? ".mlp.expert" : ".mlp"), err};
    l->mlp.ff = s.integer("ff", 1, kMaxSize);
    if (!moe) return s.ok;
    Fields r{mlp->get("router"), where + ".mlp.router", err};
    l->mlp.experts = r.integer("experts", 1, 1 << 16);
    l->mlp.top = r.integer("top", 1, l->mlp.experts > 0 ? l->mlp.experts : 1);
    return s.ok && r.ok;
}

bool read_bupozen(const Json &c, LmConfig *out, std::string *err) {
    out->block = LM_BLOCK_PARALLEL;
    out->norm = LM_NORM_RMS;
    if (!read_stack(c, out, err, read_bupozen_layer)) return false;
    for (size_t i = 0; i < out->layers.size(); i++) {
        const LmMixer &m = out->layers[i].mixer;
        if (m.kv_from < 0) continue;
        const LmMixer *o = m.kv_from < (int)i ? &out->layers[m.kv_from].mixer : nullptr;
        if (!o || o->kv_from >= 0 || o->kv_rank != m.kv_rank || o->rot_dim != m.rot_dim || o->rope.dims != m.rope.dims ||
            o->rope.base != m.rope.base) {
            *err = "config.json: layers[" + std::to_string(i) + "].mixer.kv_from has to name an earlier layer with a latent of its own, of equal "
                   "kv_rank, rot_dim and rotation";
            return false;
        }
    }
    return true;
}

const LmArchitecture kArchitectures[] = {
    {"Kegizen", read_kegizen},
    {"Bupozen", read_bupozen},
};

} // namespace

const LmArchitecture *lm_architecture(const std::string &name) {
    for (const LmArchitecture &a : kArchitectures)
        if (name == a.name) return &a;
    return nullptr;
}

bool lm_config_from_text(const std::string &text, LmConfig *out, std::string *err) {
    Json c;
    std::string je;
    err->clear();
    *out = LmConfig();
    if (!json_parse(text.data(), text.size(), &c, &je)) {
        *err = "config.json: " + je;
        return false;
    }
    const Json *name = c.get("architecture");
    const LmArchitecture *a = name && name->kind == Json::STRING ? lm_architecture(name->text) : nullptr;
    if (!a) {
        *err = "config.json: architecture '" + (name ? name->text : std::string("(none)")) + "' is not registered";
        return false;
    }
    out->architecture = a->name;
    return a->read(c, out, err);
}

} // namespace vb
