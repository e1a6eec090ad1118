// config.json of the config-driven decoder, and its entry in the architecture table.
#include "decoder.h"
#include "safetensors.h"

#include <cmath>
#include <new>

namespace tmb {
namespace {

thread_local std::string g_open_error;

struct Reader {
    std::string* why;
    bool         ok = true;

    void fail(const std::string& what)
    {
        if (ok) *why = what;
        ok = false;
    }
    double number(const Json& j, const char* key, const double* dflt = nullptr)
    {
        const Json* v = j.find(key);
        if (!v || v->is_null()) {
            if (dflt) return *dflt;
            fail(std::string("missing: ") + key);
            return 0;
        }
        if (v->kind != Json::kNumber || !std::isfinite(v->number)) fail(std::string("not a number: ") + key);
        return v->number;
    }
    int integer(const Json& j, const char* key, int lo, const double* dflt = nullptr)
    {
        const double x = number(j, key, dflt);
        if (x != std::floor(x) || x < lo || x > 2147483647.0) fail(std::string("out of range: ") + key);
        return ok ? (int)x : lo;
    }
    const Json* object(const Json& j, const char* key, bool optional)
    {
        const Json* v = j.find(key);
        if (!v || v->is_null()) {
            if (!optional) fail(std::string("missing: ") + key);
            return nullptr;
        }
        if (v->kind != Json::kObject) {
            fail(std::string("not an object: ") + key);
            return nullptr;
        }
        return v;
    }
};

bool read_text(const std::string& path, std::string* out)
{
    std::FILE* f = std::fopen(path.c_str(), "rb");
    if (!f) return false;
    char   buf[4096];
    size_t n;
    while ((n = std::fread(buf, 1, sizeof(buf), f)) > 0) out->append(buf, n);
    std::fclose(f);
    return true;
}

bool read_rumazen_config(const Json& j, DecoderConfig* c, std::string* why)
{
    Reader       r{why};
    const double one = 1.0, zero = 0.0;
    const Json * norm = r.object(j, "norm", false), *emb = r.object(j, "embedding", true), *layers = j.find("layers");
    c->vocab = r.integer(j, "vocab", 1);
    c->width = r.integer(j, "width", 1);
    if (norm) c->norm_eps = r.number(*norm, "eps");
    if (emb) c->embedding_scale = r.number(*emb, "scale", &one);
    if (!layers || layers->kind != Json::kArray || layers->items.empty()) r.fail("missing: layers");
    if (!r.ok) return false;
    for (const Json& l : layers->items) {
        LayerSpec   s;
        const Json *type = l.find("type"), *mixer = r.object(l, "mixer", false), *mlp = r.object(l, "mlp", true);
        if (!mixer || !type) return r.fail("a layer without type or mixer"), false;
        MixerSpec& m = s.mixer;
        m.heads      = r.integer(*mixer, "heads", 1);
        m.dim        = r.integer(*mixer, "dim", 1);
        if (type->text == "attention") {
            const double dim = m.dim, heads = m.heads, dflt_scale = 1.0 / std::sqrt(dim > 0 ? dim : 1.0);
            m.type           = MixerType::kAttention;
            m.kv_heads       = r.integer(*mixer, "kv_heads", 1, &heads);
            m.vdim           = r.integer(*mixer, "vdim", 1, &dim);
            m.scale          = r.number(*mixer, "scale", &dflt_scale);
            m.softcap        = r.number(*mixer, "softcap", &zero);
            if (const Json* rot = r.object(*mixer, "rot", true)) {
                m.rot_dims = r.integer(*rot, "dims", 0, &dim);
                m.rot_base = r.number(*rot, "base");
                if (const Json* sc = r.object(*rot, "scaling", true)) m.rot_factor = r.number(*sc, "factor", &one);
            }
            if (const Json* mask = r.object(*mixer, "mask", true)) {
                m.window = r.integer(*mask, "size", 1);
                m.pool   = r.integer(*mask, "pool", 0, &zero);
            }
            if (r.ok && (m.heads % m.kv_heads || m.rot_dims > m.dim || m.rot_dims % 2 || m.dim > 256 || m.vdim > 256 || m.softcap < 0)) {
                r.fail("attention sizes that do not fit together");
            }
        }
        else if (type->text == "general_delta") {
            const double rank = 16;
            m.type            = MixerType::kGeneralDelta;
            m.rank            = r.integer(*mixer, "rank", 1, &rank);
            if (m.dim > 256) r.fail("delta-rule heads larger than 256");
        }
        else {
            r.fail("unknown layer type: " + type->text);
        }
        if (mlp) {
            const Json* kind = mlp->find("kind");
            if (!kind || kind->text != "dense") r.fail("unknown feed-forward kind");
            s.ff = r.integer(*mlp, "ff", 1);
        }
        if (!r.ok) return false;
        c->layers.push_back(s);
    }
    return true;
}

bool read_fopinex_config(const Json& j, DecoderConfig* c, std::string* why)
{
    Reader       r{why};
    const double one = 1.0, zero = 0.0;
    const Json * norm = r.object(j, "norm", false), *layers = j.find("layers");
    c->form  = LayerForm::kGatedBranches;
    c->vocab = r.integer(j, "vocab", 1);
    c->width = r.integer(j, "width", 1);
    if (norm) c->norm_eps = r.number(*norm, "eps");
    c->residual_mult = r.number(j, "residual_mult", &one);
    if (!layers || layers->kind != Json::kArray || layers->items.empty()) r.fail("missing: layers");
    if (!r.ok) return false;
    for (const Json& l : layers->items) {
        LayerSpec   s;
        const Json *type = l.find("type"), *mixer = r.object(l, "mixer", false), *mlp = r.object(l, "mlp", true);
        if (!mixer || !type) return r.fail("a layer without type or mixer"), false;
        MixerSpec& m = s.mixer;
        m.heads      = r.integer(*mixer, "heads", 1);
        m.dim        = r.integer(*mixer, "dim", 1);
        const double dim = m.dim, heads = m.heads, dflt_scale = 1.0 / std::sqrt(dim > 0 ? dim : 1.0);
        m.vdim = r.integer(*mixer, "vdim", 1, &dim);
        if (m.dim > 256 || m.vdim > 256) r.fail("heads larger than 256");
        if (type->text == "attention") {
            const double own = -1;
            m.type     = MixerType::kChunkAttention;
            m.kv_heads = r.integer(*mixer, "kv_heads", 1, &heads);
            m.scale    = r.number(*mixer, "scale", &dflt_scale);
            m.kv_from  = r.integer(*mixer, "kv_from", -1, &own);
            if (const Json* mask = r.object(*mixer, "mask", true)) m.chunk = r.integer(*mask, "size", 1);
            if (r.ok && m.heads % m.kv_heads) r.fail("kv_heads does not divide heads");
            if (r.ok && m.kv_from >= 0) {
                const MixerSpec* o = m.kv_from < (int)c->layers.size() ? &c->layers[m.kv_from].mixer : nullptr;
                if (!o || o->type != MixerType::kChunkAttention || o->kv_from >= 0 || o->kv_heads != m.kv_heads || o->dim != m.dim || o->vdim != m.vdim) {
                    r.fail("kv_from: not an earlier attention layer with keys and values of the same shape");
                }
            }
        }
        else if (type->text == "gla") {
            const double rank = 16;
            m.type            = MixerType::kGatedLinear;
            m.tau             = r.number(*mixer, "tau");
            m.rank            = r.integer(*mixer, "rank", 1, &rank);
            if (r.ok && m.tau <= 0) r.fail("out of range: tau");
        }
        else {
            r.fail("unknown layer type: " + type->text);
        }
        if (mlp) {
            const Json *kind = mlp->find("kind"), *expert = r.object(*mlp, "expert", false), *router = r.object(*mlp, "router", false);
            if (!kind || kind->text != "moe") r.fail("unknown feed-forward kind");
            if (expert && router) {
                MoeSpec& e = s.moe;
                e.ff       = r.integer(*expert, "ff", 1);
                e.limit    = r.number(*expert, "limit");
                e.experts  = r.integer(*router, "experts", 1);
                e.identity = r.integer(*router, "identity", 0, &zero);
                e.top      = r.integer(*router, "top", 1);
                if (const Json* groups = r.object(*router, "groups", true)) {
                    e.groups = r.integer(*groups, "count", 1);
                    e.keep   = r.integer(*groups, "keep", 1);
                }
                const int n = e.experts + e.identity;
                if (r.ok && (n > kMaxRouterOutputs || e.top > kMaxRouterTop || n % e.groups || e.keep > e.groups || e.top > e.keep * (n / e.groups))) {
                    r.fail("router sizes that do not fit together");
                }
            }
        }
        if (!r.ok) return false;
        c->layers.push_back(s);
    }
    return true;
}

struct DecoderArchitecture {
    const char* name;
    bool (*read)(const Json& j, DecoderConfig* c, std::string* why);
    const char* decay_rank;  // tensor of a recurrent mixer whose rows are the rank of its decay projection
};
const DecoderArchitecture kArchitectures[] = {{"Rumazen", read_rumazen_config, "w1"}, {"Fopinex", read_fopinex_config, "a1"}};

const DecoderArchitecture* architecture_of(const Json& j)
{
    const Json* a = j.find("architecture");
    for (const DecoderArchitecture& d : kArchitectures) {
        if (a && a->text == d.name) return &d;
    }
    return nullptr;
}

}  // namespace

bool read_decoder_config(const Json& j, DecoderConfig* c, std::string* why)
{
    const DecoderArchitecture* a = architecture_of(j);
    if (!a) {
        *why = "unknown architecture";
        return false;
    }
    c->architecture = a->name;
    return a->read(j, c, why);
}

namespace {

bool read_config_file(const std::string& dir, Json* j)
{
    std::string text;
    return read_text(dir + "/config.json", &text) && Json::parse(text, j) && j->kind == Json::kObject;
}

template<int I>
bool claims(const std::string& dir)
{
    Json j;
    return read_config_file(dir, &j) && architecture_of(j) == &kArchitectures[I];
}

int decoder_open(tm_model** out, tm_handle* h, const std::string& dir, const tm_model_options& opt)
{
    Json          j;
    DecoderConfig c;
    g_open_error.clear();
    if (!read_config_file(dir, &j)) return TM_ERR_IO;
    if (!read_decoder_config(j, &c, &g_open_error)) return TM_ERR_INVALID_ARG;
    const std::string path = dir + "/model.safetensors";
    {
        // the ranks of the decay projections are given by their tensors
        SafeTensors st;
        if (!st.open(path)) {
            g_open_error = "cannot read " + path;
            return TM_ERR_IO;
        }
        for (size_t i = 0; i < c.layers.size(); ++i) {
            MixerSpec& m = c.layers[i].mixer;
            if (m.type != MixerType::kGeneralDelta && m.type != MixerType::kGatedLinear) continue;
            const std::string name = "l" + std::to_string(i) + ".mix." + architecture_of(j)->decay_rank;
            const SafeTensor* t    = st.find(name);
            if (!t || t->shape.size() != 2 || t->shape[0] < 1 || t->shape[0] > 65536) {
                g_open_error = "missing: " + name;
                return TM_ERR_IO;
            }
            m.rank = (int)t->shape[0];
        }
    }
    tm_decoder* m = new (std::nothrow) tm_decoder();
    if (!m) return TM_ERR_CUDA;
    int rc = m->init(h, c, opt);
    if (rc == TM_OK) rc = m->load(path, &g_open_error);
    if (rc != TM_OK) {
        tm_model_close(m);
        return rc;
    }
    *out = m;
    return TM_OK;
}

const ArchitectureRegistration g_rumazen({kArchitectures[0].name, claims<0>, decoder_open});
const ArchitectureRegistration g_fopinex({kArchitectures[1].name, claims<1>, decoder_open});

}  // namespace
}  // namespace tmb

using namespace tmb;

extern "C" const char* tm_model_last_error(void)
{
    return g_open_error.c_str();
}

extern "C" int tm_decoder_create_random(tm_model** out, tm_handle* h, const char* config_json, const tm_model_options* opt,
                                        unsigned long long seed)
{
    if (!out || !h || !config_json || !opt || opt->max_batch_size <= 0 || opt->session_len <= 1) return TM_ERR_INVALID_ARG;
    *out = nullptr;
    Json          j;
    DecoderConfig c;
    g_open_error.clear();
    if (!Json::parse(config_json, &j) || !read_decoder_config(j, &c, &g_open_error)) return TM_ERR_INVALID_ARG;
    tm_decoder* m = new (std::nothrow) tm_decoder();
    if (!m) return TM_ERR_CUDA;
    int rc = m->init(h, c, *opt);
    if (rc == TM_OK) rc = m->random_weights(seed);
    if (rc != TM_OK) {
        tm_model_close(m);
        return rc;
    }
    *out = m;
    return TM_OK;
}
