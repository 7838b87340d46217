// Reader of safetensors files: an 8-byte little-endian length, that many bytes of JSON (name -> dtype, shape, data_offsets), then the
// tensors' bytes.
#include "dl/dl.h"
#include "dl/internal.h"
#include "dl/json.h"

#include <fstream>
#include <stdexcept>

namespace dl::io {

StateDict load_safetensors(const std::filesystem::path& path) {
    std::ifstream in;
    in.exceptions(std::ios::failbit | std::ios::badbit | std::ios::eofbit);
    in.open(path, std::ios::binary);
    const std::uint64_t file_bytes = std::filesystem::file_size(path);
    unsigned char raw[8];
    in.read(reinterpret_cast<char*>(raw), 8);
    std::uint64_t header_bytes = 0;
    for (int i = 7; i >= 0; --i) header_bytes = (header_bytes << 8) | raw[i];
    if (header_bytes > file_bytes - 8) throw std::runtime_error("corrupt safetensors file: the header exceeds the file");
    std::string text(static_cast<std::size_t>(header_bytes), '\0');
    in.read(text.data(), static_cast<std::streamsize>(header_bytes));
    const Json header = Json::parse(text);
    const std::uint64_t data_start = 8 + header_bytes, data_bytes = file_bytes - data_start;
    StateDict result;
    for (const auto& [name, entry] : header.members()) {
        if (name == "__metadata__") continue;
        const std::string& type = entry.at("dtype").text();
        const bool int32 = type == "I32";   // integer tables; held as i64, the library's index type
        DType dtype;
        if (type == "BF16") dtype = DType::bf16;
        else if (type == "F32") dtype = DType::f32;
        else if (type == "F64") dtype = DType::f64;
        else if (type == "I64" || int32) dtype = DType::i64;
        else throw std::runtime_error("safetensors: '" + name + "' has dtype " + type + ", which this library does not hold");
        Shape shape;
        std::uint64_t elements = 1;
        for (const auto& extent : entry.at("shape").items()) {
            const Index n = extent.integer();
            if (n < 0 || (n > 0 && elements > data_bytes / static_cast<std::uint64_t>(n) + 1)) throw std::runtime_error("corrupt safetensors file: extents of '" + name + "'");
            elements *= static_cast<std::uint64_t>(n);
            shape.push_back(n);
        }
        const auto& offsets = entry.at("data_offsets").items();
        if (offsets.size() != 2) throw std::runtime_error("corrupt safetensors file: offsets of '" + name + "'");
        const auto begin = static_cast<std::uint64_t>(offsets[0].integer()), end = static_cast<std::uint64_t>(offsets[1].integer());
        const std::uint64_t size = elements * (int32 ? 4 : element_size(dtype));
        if (end > data_bytes || begin > end || end - begin != size) throw std::runtime_error("corrupt safetensors file: offsets of '" + name + "'");
        Tensor tensor = empty(shape, {dtype, Device::cpu()});
        in.seekg(static_cast<std::streamoff>(data_start + begin));
        if (int32) {
            std::vector<std::int32_t> narrow(static_cast<std::size_t>(elements));
            in.read(reinterpret_cast<char*>(narrow.data()), static_cast<std::streamsize>(size));
            std::copy(narrow.begin(), narrow.end(), static_cast<Index*>(tensor.mutable_data()));
        } else if (size > 0) {
            in.read(static_cast<char*>(tensor.mutable_data()), static_cast<std::streamsize>(size));
        }
        result.emplace_back(name, std::move(tensor));
    }
    return result;
}

}  // namespace dl::io
