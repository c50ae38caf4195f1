// The .vlt weight file, read into one device buffer, and the model's tensor table.
// Layout: tools/convert.py:117-133 (writer), engine/src/weights.rs:37-74 (reader).
#pragma once
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <algorithm>
#include <cstring>
#include <map>
#include <string>
#include <vector>

#include "common.h"
#include "json.h"

namespace vlt {

enum class DType : uint32_t { F32 = 0, Bf16 = 1, I8 = 2 };

struct Tensor {
    DType dtype;
    std::vector<uint32_t> shape;
    size_t offset, nbytes;  // offset into the weight buffer
};

struct Weights {
    Buffer buffer;
    std::map<std::string, Tensor> tensors;
    std::vector<uint8_t> host;  // small f32 tensors are also read on the host from here
    std::string path;

    // engine/src/weights.rs:38-74 `load`.
    void load(const std::string& p, bool host_only) {
        path = p;
        FILE* f = std::fopen(p.c_str(), "rb");
        if (!f) throw Error(p + ": cannot open");
        struct Closer { FILE* f; ~Closer() { std::fclose(f); } } closer{f};
        uint8_t head[32];
        if (std::fread(head, 1, 32, f) != 32) throw Error(p + ": short header");
        auto u32 = [](const uint8_t* b) { uint32_t v; std::memcpy(&v, b, 4); return v; };
        auto u64 = [](const uint8_t* b) { uint64_t v; std::memcpy(&v, b, 8); return v; };
        if (std::memcmp(head, "VIOLETTO", 8) != 0 || u32(head + 8) != 1) throw Error(p + ": not a version-1 violetto weight file");
        const uint32_t n = u32(head + 12);
        const uint64_t data_offset = u64(head + 16);
        std::vector<uint8_t> rec(size_t(128) * n);
        if (std::fread(rec.data(), 1, rec.size(), f) != rec.size()) throw Error(p + ": short tensor records");
        size_t end = 0;
        for (uint32_t i = 0; i < n; i++) {
            const uint8_t* r = rec.data() + size_t(128) * i;
            size_t len = 0;
            while (len < 64 && r[len]) len++;
            std::string name(reinterpret_cast<const char*>(r), len);
            const uint32_t d = u32(r + 64);
            if (d > 2) throw Error(name + ": unknown dtype " + std::to_string(d));
            Tensor t;
            t.dtype = DType(d);
            const uint32_t ndim = u32(r + 68);
            if (ndim > 4) throw Error(name + ": more than 4 dimensions");
            for (uint32_t j = 0; j < ndim; j++) t.shape.push_back(u32(r + 72 + 4 * j));
            t.offset = u64(r + 88);
            t.nbytes = u64(r + 96);
            end = std::max(end, t.offset + t.nbytes);
            tensors[name] = t;
        }
        // One buffer for everything (weights.rs:64-72), staged through pinned memory in slices.
        if (std::fseek(f, long(data_offset), SEEK_SET) != 0) throw Error(p + ": cannot seek to the data region");
        buffer.alloc(end, host_only);
        const size_t SLICE = size_t(64) << 20;
        std::vector<uint8_t> stage(std::min(end, SLICE));
        for (size_t at = 0; at < end; at += SLICE) {
            const size_t nb = std::min(SLICE, end - at);
            if (std::fread(stage.data(), 1, nb, f) != nb) throw Error(p + ": short data region");
            buffer.write(at, stage.data(), nb);
        }
        // Keep the small f32 tensors on the host too.
        for (auto& [name, t] : tensors)
            if (t.dtype == DType::F32 && t.nbytes <= (1u << 20)) {
                if (host.size() < t.offset + t.nbytes) host.resize(t.offset + t.nbytes);
                buffer.read(t.offset, host.data() + t.offset, t.nbytes);
            }
    }

    bool has(const std::string& name) const { return tensors.count(name) != 0; }
    const Tensor& tensor(const std::string& name) const {
        auto it = tensors.find(name);
        if (it == tensors.end()) throw Error("weight file has no tensor " + name);
        return it->second;
    }
    // engine/src/weights.rs:83-89 `get`.
    const Tensor& get(const std::string& name, DType dtype, const std::vector<uint32_t>& shape) const {
        const Tensor& t = tensor(name);
        if (t.dtype != dtype || t.shape != shape) {
            auto fmt = [](const std::vector<uint32_t>& s) { std::string o = "["; for (size_t i = 0; i < s.size(); i++) o += (i ? ", " : "") + std::to_string(s[i]); return o + "]"; };
            throw Error(name + ": expected dtype " + std::to_string(uint32_t(dtype)) + " " + fmt(shape) + ", found dtype " + std::to_string(uint32_t(t.dtype)) + " " + fmt(t.shape));
        }
        return t;
    }
    // engine/src/weights.rs:91-95 `f32s`.
    std::vector<float> f32s(const std::string& name) const {
        const Tensor& t = tensor(name);
        if (t.dtype != DType::F32) throw Error(name + ": expected f32");
        std::vector<float> v(t.nbytes / 4);
        if (t.offset + t.nbytes <= host.size()) std::memcpy(v.data(), host.data() + t.offset, t.nbytes);
        else buffer.read(t.offset, v.data(), t.nbytes);
        return v;
    }
};

// A safetensors file (8-byte little-endian header length, JSON header name -> dtype, shape, data_offsets, then the data),
// mapped read-only; `place` copies tensors into the device buffer in whatever order and stacking the model wants them.
struct SafeTensors {
    struct Entry { std::string dtype; std::vector<uint32_t> shape; const uint8_t* data; size_t nbytes; };
    std::map<std::string, Entry> entries;
    Buffer buffer;
    size_t used = 0;
    std::string path;

    SafeTensors() = default;
    SafeTensors(const SafeTensors&) = delete;
    ~SafeTensors() { unmap(); }
    void unmap() {
        if (map) munmap(map, map_bytes);
        map = nullptr;
        entries.clear();
    }

    void open(const std::string& p) {
        path = p;
        const int fd = ::open(p.c_str(), O_RDONLY);
        if (fd < 0) throw Error(p + ": cannot open");
        struct stat st;
        const bool ok = fstat(fd, &st) == 0 && st.st_size >= 8;
        map_bytes = ok ? size_t(st.st_size) : 0;
        void* m = ok ? mmap(nullptr, map_bytes, PROT_READ, MAP_PRIVATE, fd, 0) : MAP_FAILED;
        ::close(fd);
        if (m == MAP_FAILED) throw Error(p + ": not a safetensors file");
        map = m;
        const uint8_t* base = static_cast<const uint8_t*>(m);
        uint64_t n;
        std::memcpy(&n, base, 8);
        if (n > map_bytes - 8) throw Error(p + ": the header is longer than the file");
        const Json head = Json::parse(reinterpret_cast<const char*>(base + 8), n, p);
        const size_t left = map_bytes - 8 - n;
        size_t total = 0;
        for (const auto& [name, t] : head.fields) {
            if (name == "__metadata__") continue;
            Entry e;
            e.dtype = t.at("dtype").text("dtype");
            size_t count = 1;
            for (const Json& d : t.at("shape").items) {
                e.shape.push_back(d.count(name + " shape"));
                count *= e.shape.back();
            }
            const std::vector<Json>& off = t.at("data_offsets").items;
            if (off.size() != 2) throw Error(name + ": bad data_offsets");
            const double a = off[0].number("data_offsets"), b = off[1].number("data_offsets");
            if (!(a >= 0 && b >= a && b <= double(left))) throw Error(name + ": its data lies outside the file");
            e.data = base + 8 + n + size_t(a);
            e.nbytes = size_t(b - a);
            const size_t size = e.dtype == "BF16" || e.dtype == "F16" ? 2 : e.dtype == "F32" || e.dtype == "I32" ? 4 : 0;
            if (size && e.nbytes != count * size) throw Error(name + ": its data does not fit its shape");
            total += e.nbytes + 256;
            if (e.shape.size() == 2) total += size_t(128) * e.shape[1] * 2 + size_t(126) * e.shape[0];  // (room for `zeros` and `place_wide`; untouched pages of it cost nothing)
            if (e.shape.size() == 1) total += 256;
            entries[name] = e;
        }
        buffer.alloc(total + 256, true);  // (filled on the host, then moved to the device in one copy: see to_device)
    }
    bool has(const std::string& name) const { return entries.count(name) != 0; }
    const Entry& get(const std::string& name, const std::vector<uint32_t>& shape) const {
        auto it = entries.find(name);
        if (it == entries.end()) throw Error(path + ": no tensor " + name);
        const Entry& e = it->second;
        if (e.dtype != "BF16" || e.shape != shape) {
            auto fmt = [](const std::vector<uint32_t>& s) { std::string o = "["; for (size_t i = 0; i < s.size(); i++) o += (i ? ", " : "") + std::to_string(s[i]); return o + "]"; };
            throw Error(name + ": expected BF16 " + fmt(shape) + ", found " + e.dtype + " " + fmt(e.shape));
        }
        return e;
    }
    // Appends a bf16 tensor; returns its offset. `fresh` starts a new 256-byte-aligned block, else it follows the tensor
    // placed before it without a gap (a stack of rows).
    size_t place(const std::string& name, const std::vector<uint32_t>& shape, bool fresh = true) {
        const Entry& e = get(name, shape);
        const size_t at = room(e.nbytes, fresh);
        std::memcpy(buffer.as<uint8_t>() + at, e.data, e.nbytes);
        return at;
    }
    // Two matrices of one shape with their rows (two vectors: their entries) in turn: a, b, a, b, ...
    size_t place_pairs(const std::string& a, const std::string& b, const std::vector<uint32_t>& shape, bool fresh = true) {
        const Entry &ea = get(a, shape), &eb = get(b, shape);
        const size_t row = size_t(shape.size() > 1 ? shape[1] : 1) * 2, at = room(2 * ea.nbytes, fresh);
        uint8_t* dst = buffer.as<uint8_t>() + at;
        for (size_t r = 0; r < shape[0]; r++) {
            std::memcpy(dst + 2 * r * row, ea.data + r * row, row);
            std::memcpy(dst + (2 * r + 1) * row, eb.data + r * row, row);
        }
        return at;
    }
    // A stack of `blocks` matrices [rows][k], each as its transpose [k][rows].
    size_t place_transposed(const std::string& name, uint32_t blocks, uint32_t rows, uint32_t k) {
        const Entry& e = get(name, {blocks * rows, k});
        const size_t at = room(e.nbytes, true);
        uint16_t* dst = reinterpret_cast<uint16_t*>(buffer.as<uint8_t>() + at);
        for (size_t b = 0; b < blocks; b++)
            for (size_t r = 0; r < rows; r++)
                for (size_t c = 0; c < k; c++) std::memcpy(dst + (b * k + c) * rows + r, e.data + ((b * rows + r) * k + c) * 2, 2);
        return at;
    }
    // A matrix [rows][k] with columns of zeros up to `wide`, fewer than 64 of them.
    size_t place_wide(const std::string& name, uint32_t rows, uint32_t k, uint32_t wide) {
        const Entry& e = get(name, {rows, k});
        const size_t at = room(size_t(rows) * wide * 2, true);
        for (size_t r = 0; r < rows; r++) std::memcpy(buffer.as<uint8_t>() + at + r * wide * 2, e.data + r * k * 2, size_t(k) * 2);
        return at;
    }
    // Zero bytes after the tensor placed last.
    void zeros(size_t nbytes) {
        if (used + nbytes > buffer.bytes) throw Error(path + ": no room for padding");
        used += nbytes;  // (the buffer starts as zeros)
    }
    // The rows of a matrix whose number nothing but its shape says.
    uint32_t rows(const std::string& name) const {
        auto it = entries.find(name);
        if (it == entries.end()) throw Error(path + ": no tensor " + name);
        if (it->second.shape.size() != 2 || it->second.shape[0] == 0) throw Error(name + ": not a matrix");
        return it->second.shape[0];
    }
    // The placed tensors' final home; offsets stay as they are.
    void to_device(bool host_only) {
        if (host_only) return;
        Buffer dev;
        dev.alloc(std::max<size_t>(used, 256), false);
        const size_t SLICE = size_t(64) << 20;
        for (size_t at = 0; at < used; at += SLICE) dev.write(at, buffer.as<uint8_t>() + at, std::min(SLICE, used - at));
        buffer = std::move(dev);
    }

  private:
    size_t room(size_t nbytes, bool fresh) {
        if (fresh) used = (used + 255) / 256 * 256;
        const size_t at = used;
        if (at + nbytes > buffer.bytes) throw Error(path + ": a tensor is placed twice");
        used += nbytes;
        return at;
    }
    void* map = nullptr;
    size_t map_bytes = 0;
};

// engine/src/model.rs:22-47 `Matrix`, `Int8`: [m][k] row-major at `w`; int8 has bf16 scales
// [m][k / group] at `scales`; bf16 may have a bias [m], which goes onto its products first thing.
struct Matrix {
    const uint8_t* w = nullptr;
    const uint16_t *scales = nullptr, *bias = nullptr;
    uint32_t m = 0, k = 0, group = 0;
    bool int8 = false;
    size_t bytes() const { return int8 ? size_t(m) * k + size_t(2) * m * (k / group) : size_t(2) * m * k; }
};

// engine/src/model.rs:81-103 `matrix`. The reference takes scale groups of 8..256; one scale per
// output row (group = k) is taken as well.
inline Matrix load_matrix(const Weights& w, const std::string& name, uint32_t m, uint32_t k) {
    const uint8_t* base = w.buffer.as<uint8_t>();
    Matrix out;
    out.m = m;
    out.k = k;
    if (w.tensor(name).dtype != DType::I8) {
        out.w = base + w.get(name, DType::Bf16, {m, k}).offset;
        return out;
    }
    out.w = base + w.get(name, DType::I8, {m, k}).offset;
    const std::string sn = name + ".scale";
    const Tensor& st = w.tensor(sn);
    const uint32_t groups = st.shape.size() > 1 ? st.shape[1] : 0;
    const uint32_t group = k / std::max(groups, 1u);
    // Groups of a power of two, or one scale per row whatever k is.
    if (group < 8 || (groups > 1 && (group & (group - 1))) || group * groups != k) throw Error(sn + ": " + std::to_string(groups) + " groups per row of " + std::to_string(k));
    out.scales = reinterpret_cast<const uint16_t*>(base + w.get(sn, DType::Bf16, {m, groups}).offset);
    out.group = group;
    out.int8 = true;
    return out;
}

struct ModelDesc {
    uint32_t n_layers = 0, d = 0, n_heads = 0, n_kv = 0, hd = 0, ffn = 0, vocab = 0, vocab_real = 0, page = 0;
    float eps = 0, attn_scale = 0;
    uint32_t qkv_w() const { return (n_heads + 2 * n_kv) * hd; }
    uint32_t group() const { return n_heads / n_kv; }
};

struct Layer {
    Matrix qkv, o, gate_up, down;
};

// What a layer of the reference's own architecture has beyond the four projections (engine/src/model.rs:49-67): device
// pointers into the weight buffer, and the scalars of tools/convert.py:104.
struct LimiteLayer {
    const float* attn_gate = nullptr;  // [n_heads][128]
    const float* ve_gate = nullptr;    // [n_kv][12]; layers with value embeddings only
    const float* xsa = nullptr;        // [n_heads]
    float qkv_scale = 1, o_scale = 1, resid_attn = 1, post_attn = 1, resid_mlp = 1, post_mlp = 1;
    bool global = false;
    uint32_t kv_index = 0;  // among the global or among the local layers
};

}  // namespace vlt
