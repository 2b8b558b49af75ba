// A model folder (config.json + model.safetensors) into a decode driver (b200_model_load_dir).
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <fstream>
#include <iterator>

#include "decode_ctx.h"

using namespace b200;

namespace {

struct Mapped {
    const uint8_t *p = nullptr;
    size_t n = 0;
    int open(const std::string &path) {
        const int fd = ::open(path.c_str(), O_RDONLY);
        B200_REQUIRE(fd >= 0, "model_load: cannot open %s", path.c_str());
        struct stat st;
        const bool ok = fstat(fd, &st) == 0 && st.st_size > 0;
        void *m = ok ? mmap(nullptr, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0) : MAP_FAILED;
        ::close(fd);
        B200_REQUIRE(m != MAP_FAILED, "model_load: cannot map %s", path.c_str());
        p = (const uint8_t *)m;
        n = (size_t)st.st_size;
        return B200_STATUS_SUCCESS;
    }
    ~Mapped() {
        if (p) munmap((void *)p, n);
    }
};

struct FileTensor {
    std::string name;
    int type = -1;
    int64_t ne0 = 1, ne1 = 1;
    const uint8_t *data = nullptr;
    size_t nbytes = 0;
};

// The tensors of a safetensors file.  Layout: u64 header size, a JSON object with one member per tensor, the bytes the members'
// data_offsets refer to.
int read_table(const Mapped &f, std::vector<FileTensor> *out) {
    uint64_t len = 0;
    B200_REQUIRE(f.n >= 8, "model_load: the safetensors file is too short");
    memcpy(&len, f.p, 8);
    B200_REQUIRE(len <= f.n - 8, "model_load: the safetensors header is longer than the file");
    Json h;
    B200_REQUIRE(Json::parse((const char *)f.p + 8, (size_t)len, &h) && h.kind == Json::OBJ, "model_load: the safetensors header is not a JSON object");
    const uint8_t *data = f.p + 8 + len;
    const size_t room = f.n - 8 - (size_t)len;
    for (const auto &m : h.members) {
        if (m.first == "__metadata__") continue;
        FileTensor t;
        t.name = m.first;
        const Json *dt = m.second.find("dtype"), *shape = m.second.find("shape"), *at = m.second.find("data_offsets");
        B200_REQUIRE(dt && shape && at && at->items.size() == 2, "model_load: tensor %s has no dtype, shape or place", t.name.c_str());
        t.type = dt->str == "BF16" ? B200_TYPE_BF16 : dt->str == "F32" ? B200_TYPE_F32 : dt->str == "I32" ? B200_TYPE_I32 : -1;
        B200_REQUIRE(t.type >= 0, "model_load: tensor %s is of type %s", t.name.c_str(), dt->str.c_str());
        const size_t nd = shape->items.size();
        for (size_t d = 0; d < nd; d++) {
            const int64_t e = (int64_t)shape->items[d].num;
            B200_REQUIRE(e > 0 && e < ((int64_t)1 << 40), "model_load: tensor %s has an empty dimension", t.name.c_str());
            if (d + 1 == nd) t.ne0 = e;
            else t.ne1 *= e;
        }
        const double a = at->items[0].num, b = at->items[1].num;
        B200_REQUIRE(a >= 0 && b >= a && b <= (double)room, "model_load: tensor %s lies outside the file", t.name.c_str());
        t.data = data + (size_t)a;
        t.nbytes = (size_t)(b - a);
        out->push_back(t);
    }
    return B200_STATUS_SUCCESS;
}

}  // namespace

extern "C" int b200_model_load_dir(const char *dir, int dtype, int device, int32_t n_ctx, int32_t n_batch, int32_t n_seq, b200_llama **out) {
    B200_REQUIRE(dir != nullptr && out != nullptr, "model_load: null argument");
    *out = nullptr;
    const std::string d(dir);
    std::ifstream cf(d + "/config.json", std::ios::binary);
    B200_REQUIRE(cf.good(), "model_load: cannot open %s/config.json", dir);
    const std::string config((std::istreambuf_iterator<char>(cf)), std::istreambuf_iterator<char>());
    Mapped f;
    int rc = f.open(d + "/model.safetensors");
    if (rc != B200_STATUS_SUCCESS) return rc;
    std::vector<FileTensor> tensors;
    rc = read_table(f, &tensors);
    if (rc != B200_STATUS_SUCCESS) return rc;
    b200_llama *c = nullptr;
    rc = b200_model_new(config.c_str(), dtype, device, n_ctx, n_batch, n_seq, &c);
    if (rc != B200_STATUS_SUCCESS) return rc;
    for (const FileTensor &t : tensors)
        if (rc == B200_STATUS_SUCCESS) rc = b200_llama_learn_shape(c, t.name.c_str(), t.ne0, t.ne1);
    std::vector<uint8_t> aligned;
    for (const FileTensor &t : tensors) {
        if (rc != B200_STATUS_SUCCESS) break;
        const void *p = t.data;
        if ((uintptr_t)p & 3) {   // the data section starts wherever the header ends
            aligned.assign(t.data, t.data + t.nbytes);
            p = aligned.data();
        }
        rc = b200_llama_set_tensor(c, t.name.c_str(), t.type, t.ne0, t.ne1, p, t.nbytes);
    }
    if (rc != B200_STATUS_SUCCESS) {
        b200_llama_free(c);
        return rc;
    }
    *out = c;
    return B200_STATUS_SUCCESS;
}
