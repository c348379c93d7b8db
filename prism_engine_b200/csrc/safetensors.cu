// Reader of .safetensors checkpoints for the layered engine:
//   u64 LE header length | JSON header {name: {"dtype", "shape", "data_offsets": [begin, end]}, ...} | data
// Every tensor goes to its place in the engine by name; weights are bf16.
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstring>

#include "json.hpp"
#include "layered.hpp"

namespace prism {

struct MappedFile {
    const uint8_t *p = nullptr;
    size_t n = 0;
    ~MappedFile() {
        if (p) munmap(const_cast<uint8_t *>(p), n);
    }
    bool open(const char *path) {
        const int fd = ::open(path, O_RDONLY);
        if (fd < 0) return false;
        struct stat st;
        if (fstat(fd, &st) == 0 && st.st_size > 0) {
            void *m = mmap(nullptr, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
            if (m != MAP_FAILED) {
                p = static_cast<const uint8_t *>(m);
                n = (size_t)st.st_size;
            }
        }
        ::close(fd);
        return p != nullptr;
    }
};

struct SafeTensor {
    std::string name, dtype;
    std::vector<uint64_t> shape;
    uint64_t begin = 0, end = 0;
};

static bool parse_numbers(Json &j, std::vector<uint64_t> &out) {
    out.clear();
    if (!j.eat('[')) return false;
    if (j.eat(']')) return true;
    while (j.ok) {
        out.push_back(j.num());
        if (j.eat(',')) continue;
        return j.ok && j.eat(']');
    }
    return false;
}

static bool parse_safetensors(const char *p, size_t n, std::vector<SafeTensor> &out) {
    Json j{p, p + n};
    if (!j.eat('{')) return false;
    if (j.eat('}')) return true;
    while (j.ok) {
        SafeTensor t;
        t.name = j.str();
        if (!j.eat(':')) return false;
        if (t.name == "__metadata__") {
            j.skip();
        } else {
            if (!j.eat('{')) return false;
            while (j.ok) {
                const std::string f = j.str();
                std::vector<uint64_t> v;
                if (!j.eat(':')) return false;
                if (f == "dtype") t.dtype = j.str();
                else if (f == "shape") { if (!parse_numbers(j, t.shape)) return false; }
                else if (f == "data_offsets") {
                    if (!parse_numbers(j, v) || v.size() != 2) return false;
                    t.begin = v[0];
                    t.end = v[1];
                } else j.skip();
                if (j.eat(',')) continue;
                if (j.eat('}')) break;
                return false;
            }
            out.push_back(t);
        }
        if (j.eat(',')) continue;
        return j.ok && j.eat('}');
    }
    return false;
}

}  // namespace prism

using namespace prism;

extern "C" int prism_cuda_engine_load_safetensors(prism_cuda_engine *e, const char *path) {
    if (!e || !path) return fail(e ? e->ctx : nullptr, PRISM_E_NULL, "null argument");
    prism_cuda_ctx *ctx = e->ctx;
    if (!e->lm) return fail(ctx, PRISM_E_STATE, "palettized models load .cimage containers");
    MappedFile f;
    if (!f.open(path)) return fail(ctx, PRISM_E_IO, std::string("cannot open ") + path);
    uint64_t hlen = 0;
    if (f.n < 8) return fail(ctx, PRISM_E_IO, "safetensors: short file");
    memcpy(&hlen, f.p, 8);
    if (hlen > f.n - 8) return fail(ctx, PRISM_E_IO, "safetensors: header longer than the file");
    std::vector<SafeTensor> ts;
    if (!parse_safetensors(reinterpret_cast<const char *>(f.p) + 8, hlen, ts)) return fail(ctx, PRISM_E_IO, "safetensors: header does not parse");
    const uint8_t *data = f.p + 8 + hlen;
    const uint64_t n = f.n - 8 - hlen;
    for (const SafeTensor &t : ts) {
        uint64_t count = 1;
        bool sane = !t.shape.empty() && t.shape.size() <= 2;
        for (uint64_t d : t.shape) {
            sane = sane && d > 0 && d <= 0xFFFFFFFFull;
            count *= sane ? d : 0;
        }
        if (t.dtype != "BF16") return fail(ctx, PRISM_E_IO, "safetensors: tensor " + t.name + " is " + t.dtype + ", expected BF16");
        if (!sane || t.end < t.begin || t.end > n || t.end - t.begin != 2 * count)
            return fail(ctx, PRISM_E_IO, "safetensors: tensor " + t.name + " has a bad shape or range");
        std::vector<uint16_t> aligned;  // the data section may start at an odd address
        const uint16_t *src = reinterpret_cast<const uint16_t *>(data + t.begin);
        if (reinterpret_cast<uintptr_t>(src) & 1) {
            aligned.resize(count);
            memcpy(aligned.data(), data + t.begin, count * 2);
            src = aligned.data();
        }
        PRISM_TRY(prism_cuda_engine_set_tensor(e, t.name.c_str(), src, t.shape[0], t.shape.size() == 2 ? t.shape[1] : 1));
    }
    return layered_check_bound(e);
}
