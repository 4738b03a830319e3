// Registry of decoder designs and the safetensors reader.
#include "model.cuh"

#include <cstring>
#include <fstream>
#include <sstream>

namespace lb {

std::unique_ptr<DecoderModel> make_gobesun(const Json &config, Precision precision);
std::unique_ptr<DecoderModel> make_mitilix(const Json &config, Precision precision);

namespace {

struct Design {
  const char *architecture;
  std::unique_ptr<DecoderModel> (*make)(const Json &, Precision);
};
const Design kDesigns[] = {
    {"Mitilix", &make_mitilix},
    {"Gobesun", &make_gobesun},
};

}  // namespace

std::unique_ptr<DecoderModel> make_model(const Json &config, Precision precision) {
  const std::string &name = config.at("architecture").as_string();
  for (const Design &d : kDesigns)
    if (name == d.architecture) return d.make(config, precision);
  throw std::runtime_error("unknown architecture \"" + name + "\" (known: " + registered_architectures() + ")");
}

const char *registered_architectures() {
  static const std::string names = [] {
    std::string s;
    for (const Design &d : kDesigns) s += (s.empty() ? "" : ",") + std::string(d.architecture);
    return s;
  }();
  return names.c_str();
}

std::string read_text_file(const std::string &path) {
  std::ifstream in(path, std::ios::binary);
  if (!in) throw std::runtime_error("cannot open " + path);
  std::stringstream ss;
  ss << in.rdbuf();
  return ss.str();
}

TensorFile::TensorFile(const std::string &path) : path_(path) {
  std::ifstream in(path, std::ios::binary | std::ios::ate);
  if (!in) throw std::runtime_error("cannot open " + path);
  const uint64_t size = (uint64_t)in.tellg();
  in.seekg(0);
  unsigned char len[8];
  if (size < 8 || !in.read(reinterpret_cast<char *>(len), 8)) throw std::runtime_error(path + ": no safetensors header");
  uint64_t n = 0;
  for (int i = 7; i >= 0; --i) n = n << 8 | len[i];
  if (n > size - 8) throw std::runtime_error(path + ": the header is longer than the file");
  std::string text((size_t)n, '\0');
  if (!in.read(&text[0], (std::streamsize)n)) throw std::runtime_error(path + ": truncated header");
  data_offset_ = 8 + n;
  data_bytes_ = size - data_offset_;
  const Json header = Json::parse(text);
  if (header.kind != Json::Object) throw std::runtime_error(path + ": the header is not an object");
  for (const auto &m : header.members) {
    if (m.first == "__metadata__") continue;
    Entry e;
    e.name = m.first;
    e.dtype = m.second.at("dtype").as_string();
    for (const Json &d : m.second.at("shape").as_array()) e.shape.push_back(d.as_int());
    const auto &off = m.second.at("data_offsets").as_array();
    if (off.size() != 2) throw std::runtime_error(path + ": bad data_offsets of " + e.name);
    e.begin = (uint64_t)off[0].as_int();
    e.end = (uint64_t)off[1].as_int();
    if (e.begin > e.end || e.end > data_bytes_) throw std::runtime_error(path + ": " + e.name + " lies outside the file");
    entries_.push_back(std::move(e));
  }
}

const TensorFile::Entry *TensorFile::lookup(const std::string &name) const {
  for (const Entry &e : entries_)
    if (e.name == name) return &e;
  return nullptr;
}

const std::vector<long long> &TensorFile::shape(const std::string &name) const {
  const Entry *e = lookup(name);
  if (e == nullptr) throw std::runtime_error(path_ + ": no tensor \"" + name + "\"");
  return e->shape;
}

const TensorFile::Entry &TensorFile::bf16(const std::string &name, const std::vector<long long> &shape) const {
  const Entry *e = lookup(name);
  if (e == nullptr) throw std::runtime_error(path_ + ": no tensor \"" + name + "\"");
  if (e->dtype != "BF16") throw std::runtime_error(path_ + ": " + name + " is " + e->dtype + ", expected BF16");
  long long count = 1;
  for (long long d : shape) count *= d;
  if (e->shape != shape || (uint64_t)count * 2 != e->end - e->begin) {
    auto show = [](const std::vector<long long> &v) {
      std::string s = "[";
      for (size_t i = 0; i < v.size(); ++i) s += (i ? ", " : "") + std::to_string(v[i]);
      return s + "]";
    };
    throw std::runtime_error(path_ + ": " + name + " has shape " + show(e->shape) + ", expected " + show(shape));
  }
  return *e;
}

float TensorFile::scalar_bf16(const std::string &name) const {
  const Entry *found = lookup(name);
  const Entry &e = bf16(name, found != nullptr && found->shape.size() == 1 ? std::vector<long long>{1} : std::vector<long long>{});
  std::ifstream in(path_, std::ios::binary);
  in.seekg((std::streamoff)(data_offset_ + e.begin));
  unsigned char b[2];
  if (!in.read(reinterpret_cast<char *>(b), 2)) throw std::runtime_error(path_ + ": cannot read " + name);
  const uint32_t bits = (uint32_t)b[0] << 16 | (uint32_t)b[1] << 24;
  float v;
  std::memcpy(&v, &bits, 4);
  if ((bits & 0x7f800000u) == 0x7f800000u) throw std::runtime_error(path_ + ": " + name + " is not finite");
  return v;
}

}  // namespace lb
