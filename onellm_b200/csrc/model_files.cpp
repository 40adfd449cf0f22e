// config.json and .safetensors readers, the model registry and the entry points that open a model folder.
#include "model_files.h"

#include <errno.h>
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include "engine.h"

namespace onellm {

// ---- JSON --------------------------------------------------------------------------------------------------
namespace {
struct Parser {
    const char* p;
    const char* end;
    const char* start;
    bool fail = false;

    void space()
    {
        while (p < end && (*p == ' ' || *p == '\t' || *p == '\n' || *p == '\r')) p++;
    }
    bool take(char c)
    {
        space();
        if (p < end && *p == c) {
            p++;
            return true;
        }
        return false;
    }
    bool word(const char* w)
    {
        const size_t n = strlen(w);
        if ((size_t)(end - p) >= n && memcmp(p, w, n) == 0) {
            p += n;
            return true;
        }
        return false;
    }
    static void utf8(std::string& s, uint32_t c)
    {
        if (c < 0x80) s += (char)c;
        else if (c < 0x800) {
            s += (char)(0xC0 | (c >> 6));
            s += (char)(0x80 | (c & 63));
        } else if (c < 0x10000) {
            s += (char)(0xE0 | (c >> 12));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        } else {
            s += (char)(0xF0 | (c >> 18));
            s += (char)(0x80 | ((c >> 12) & 63));
            s += (char)(0x80 | ((c >> 6) & 63));
            s += (char)(0x80 | (c & 63));
        }
    }
    uint32_t hex4()
    {
        uint32_t v = 0;
        for (int i = 0; i < 4; i++) {
            if (p >= end) {
                fail = true;
                return 0;
            }
            const char c = *p++;
            v <<= 4;
            if (c >= '0' && c <= '9') v |= c - '0';
            else if (c >= 'a' && c <= 'f') v |= c - 'a' + 10;
            else if (c >= 'A' && c <= 'F') v |= c - 'A' + 10;
            else fail = true;
        }
        return v;
    }
    std::string string()
    {
        std::string s;
        if (!take('"')) {
            fail = true;
            return s;
        }
        while (p < end && *p != '"') {
            if (*p != '\\') {
                s += *p++;
                continue;
            }
            if (++p >= end) break;
            const char c = *p++;
            switch (c) {
                case 'n': s += '\n'; break;
                case 't': s += '\t'; break;
                case 'r': s += '\r'; break;
                case 'b': s += '\b'; break;
                case 'f': s += '\f'; break;
                case 'u': {
                    uint32_t u = hex4();
                    if (u >= 0xD800 && u < 0xDC00 && word("\\u")) u = 0x10000 + ((u - 0xD800) << 10) + (hex4() - 0xDC00);
                    utf8(s, u);
                    break;
                }
                default: s += c;
            }
        }
        if (p >= end) fail = true;
        else p++;
        return s;
    }
    Json value(int depth)
    {
        Json j;
        space();
        if (fail || p >= end || depth > 64) {
            fail = true;
            return j;
        }
        if (*p == '{') {
            p++;
            j.kind = Json::OBJECT;
            if (take('}')) return j;
            do {
                space();
                const std::string k = string();
                if (fail || !take(':')) {
                    fail = true;
                    return j;
                }
                j.fields[k] = value(depth + 1);
            } while (!fail && take(','));
            if (!take('}')) fail = true;
        } else if (*p == '[') {
            p++;
            j.kind = Json::ARRAY;
            if (take(']')) return j;
            do j.items.push_back(value(depth + 1));
            while (!fail && take(','));
            if (!take(']')) fail = true;
        } else if (*p == '"') {
            j.kind = Json::STRING;
            j.text = string();
        } else if (word("true")) {
            j.kind = Json::BOOL;
            j.boolean = true;
        } else if (word("false")) {
            j.kind = Json::BOOL;
        } else if (word("null")) {
        } else {
            j.kind = Json::NUMBER;
            const char* q = p;
            while (q < end && strchr("+-0123456789.eE", *q)) q++;
            const std::string s(p, q);
            char* stop = nullptr;
            j.number = strtod(s.c_str(), &stop);
            if (s.empty() || stop != s.c_str() + s.size()) fail = true;
            p = q;
        }
        return j;
    }
};
}  // namespace

int json_parse(const std::string& text, Json* out)
{
    Parser ps{text.data(), text.data() + text.size(), text.data()};
    *out = ps.value(0);
    ps.space();
    ONELLM_REQUIRE(!ps.fail && ps.p == ps.end, ONELLM_ERR_IO, "not JSON (near byte %zu)", (size_t)(ps.p - ps.start));
    return ONELLM_OK;
}

int read_text_file(const std::string& path, std::string* out)
{
    FILE* f = fopen(path.c_str(), "rb");
    ONELLM_REQUIRE(f, ONELLM_ERR_IO, "cannot open %s: %s", path.c_str(), strerror(errno));
    char buf[65536];
    size_t n;
    out->clear();
    while ((n = fread(buf, 1, sizeof(buf), f)) > 0) out->append(buf, n);
    fclose(f);
    return ONELLM_OK;
}

int json_object(const Json& j, const char* key, const char* where, const Json** out)
{
    const Json* v = j.find(key);
    ONELLM_REQUIRE(v && v->kind == Json::OBJECT, ONELLM_ERR_IO, "config: %s.%s is missing or not an object", where, key);
    *out = v;
    return ONELLM_OK;
}

int json_int(const Json& j, const char* key, const char* where, int* out)
{
    const Json* v = j.find(key);
    ONELLM_REQUIRE(v && v->kind == Json::NUMBER && v->number == floor(v->number) && fabs(v->number) < 2147483647.0, ONELLM_ERR_IO,
                   "config: %s.%s is missing or not an integer", where, key);
    *out = (int)v->number;
    return ONELLM_OK;
}

int json_float(const Json& j, const char* key, const char* where, double* out)
{
    const Json* v = j.find(key);
    ONELLM_REQUIRE(v && v->kind == Json::NUMBER, ONELLM_ERR_IO, "config: %s.%s is missing or not a number", where, key);
    *out = v->number;
    return ONELLM_OK;
}

// ---- safetensors -------------------------------------------------------------------------------------------
SafeTensors::~SafeTensors()
{
    if (f_) fclose(f_);
}

int SafeTensors::open(const std::string& path)
{
    path_ = path;
    f_ = fopen(path.c_str(), "rb");
    ONELLM_REQUIRE(f_, ONELLM_ERR_IO, "cannot open %s: %s", path.c_str(), strerror(errno));
    fseeko(f_, 0, SEEK_END);
    const size_t size = (size_t)ftello(f_);
    fseeko(f_, 0, SEEK_SET);
    unsigned char b[8];
    ONELLM_REQUIRE(size >= 8 && fread(b, 1, 8, f_) == 8, ONELLM_ERR_IO, "%s: no header", path.c_str());
    uint64_t n = 0;
    for (int i = 7; i >= 0; i--) n = (n << 8) | b[i];
    ONELLM_REQUIRE(n <= size - 8, ONELLM_ERR_IO, "%s: header of %llu bytes in a file of %zu", path.c_str(), (unsigned long long)n, size);
    std::string head(n, '\0');
    ONELLM_REQUIRE(fread(&head[0], 1, n, f_) == n, ONELLM_ERR_IO, "%s: short read", path.c_str());
    data_start_ = 8 + n;
    data_bytes_ = size - data_start_;
    Json j;
    RC(json_parse(head, &j));
    for (const auto& kv : j.fields) {
        if (kv.first == "__metadata__") continue;
        const Json *d = kv.second.find("dtype"), *s = kv.second.find("shape"), *o = kv.second.find("data_offsets");
        ONELLM_REQUIRE(d && s && o && o->items.size() == 2, ONELLM_ERR_IO, "%s: entry of %s", path.c_str(), kv.first.c_str());
        SafeTensor t;
        t.dtype = d->text;
        for (const auto& x : s->items) t.shape.push_back((int64_t)x.number);
        t.begin = (size_t)o->items[0].number;
        t.end = (size_t)o->items[1].number;
        ONELLM_REQUIRE(t.begin <= t.end && t.end <= data_bytes_, ONELLM_ERR_IO, "%s: %s lies outside the file", path.c_str(), kv.first.c_str());
        tensors_[kv.first] = t;
    }
    return ONELLM_OK;
}

const SafeTensor* SafeTensors::find(const std::string& name) const
{
    const auto it = tensors_.find(name);
    return it == tensors_.end() ? nullptr : &it->second;
}

int SafeTensors::read(const SafeTensor& t, std::vector<char>* out)
{
    out->resize(t.end - t.begin);
    ONELLM_REQUIRE(fseeko(f_, (off_t)(data_start_ + t.begin), SEEK_SET) == 0 && fread(out->data(), 1, out->size(), f_) == out->size(),
                   ONELLM_ERR_IO, "%s: short read", path_.c_str());
    return ONELLM_OK;
}

// ---- registry ----------------------------------------------------------------------------------------------
static std::map<std::string, ModelFactory>& registry()
{
    static std::map<std::string, ModelFactory> r;
    return r;
}

ModelRegistration::ModelRegistration(const char* architecture, ModelFactory make) { registry()[architecture] = make; }

static int make_model(const Json& config, const std::string& folder, int dtype, int max_batch, int max_seq_len, onellm_llama** out)
{
    const Json* name = config.find("architecture");
    ONELLM_REQUIRE(name && name->kind == Json::STRING, ONELLM_ERR_IO, "config: no \"architecture\"");
    const auto it = registry().find(name->text);
    ONELLM_REQUIRE(it != registry().end(), ONELLM_ERR_IO, "config: unknown architecture \"%s\"", name->text.c_str());
    ModelOptions opt;
    opt.dtype = dtype;
    opt.max_batch = max_batch;
    opt.max_seq_len = max_seq_len;
    Engine* m = nullptr;
    RC(it->second(config, folder, opt, &m));
    *out = reinterpret_cast<onellm_llama*>(m);
    return ONELLM_OK;
}

}  // namespace onellm

using namespace onellm;

extern "C" int onellm_model_open(const char* folder, int dtype, int max_batch, int max_seq_len, onellm_llama** out)
{
    ONELLM_REQUIRE(folder && out, ONELLM_ERR_ARG, "model_open: null pointer");
    ONELLM_REQUIRE(dtype == ONELLM_BF16 || dtype == ONELLM_F32, ONELLM_ERR_UNSUPPORTED, "model_open: dtype must be BF16 or F32");
    std::string text;
    RC(read_text_file(std::string(folder) + "/config.json", &text));
    Json config;
    RC(json_parse(text, &config));
    return make_model(config, folder, dtype, max_batch, max_seq_len, out);
}

extern "C" int onellm_model_create(const char* config_json, int dtype, int max_batch, int max_seq_len, onellm_llama** out)
{
    ONELLM_REQUIRE(config_json && out, ONELLM_ERR_ARG, "model_create: null pointer");
    ONELLM_REQUIRE(dtype == ONELLM_BF16 || dtype == ONELLM_F32, ONELLM_ERR_UNSUPPORTED, "model_create: dtype must be BF16 or F32");
    Json config;
    RC(json_parse(config_json, &config));
    return make_model(config, "", dtype, max_batch, max_seq_len, out);
}
