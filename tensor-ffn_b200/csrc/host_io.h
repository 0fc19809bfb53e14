// Host-side file formats of the inference path: config.json, *.safetensors, expert .bin,
// tokenizer.json. No CUDA in here, so all of it is unit-testable without a GPU.
#pragma once
#include <cstdint>
#include <cstdio>
#include <initializer_list>
#include <stdexcept>
#include <string>
#include <unordered_map>
#include <vector>

namespace tffn {

struct JsonValue;

struct Error : std::runtime_error {
    int code;
    Error(int c, const std::string& m) : std::runtime_error(m), code(c) {}
};
// status codes shared with the C ABI (include/tffn.h)
enum { kOk = 0, kErrInvalid = -1, kErrIO = -2, kErrFormat = -3, kErrShape = -4, kErrCuda = -5, kErrCapacity = -6,
       kErrUnsupported = -7, kErrDevice = -8 };

// Mirrors QwenConfig (inference/include/model/qwen.h:9-23) and qwen_config_from_json
// (inference/src/model/qwen.cu:21-63): same keys, same defaults, head_dim = hidden / heads,
// eos/bos given as a number or as an array whose first element counts.
// A model whose layers are listed one by one (`layers` not empty) is described by LayerSpec entries instead of
// the uniform Qwen2 fields; the uniform fields then hold what is common (width, vocabulary, layer count, eps) or
// the first layer's value.
struct RopeSpec {
    int dims = 0;         // rotated leading dimensions of a head (0: none)
    bool halves = false;  // pairs are (i, i + dims / 2) instead of the neighbours (2i, 2i + 1)
    double base = 10000.0;
    bool scaled = false;  // wavelength-dependent frequency scaling: long waves / factor, short ones kept, a ramp between
    double factor = 1.0, low = 1.0, high = 1.0, original = 1.0;
    bool operator==(const RopeSpec& o) const {
        return dims == o.dims && halves == o.halves && base == o.base && scaled == o.scaled && factor == o.factor && low == o.low && high == o.high &&
               original == o.original;
    }
};
// frequency of pair i (radians per position)
double rope_frequency(const RopeSpec& r, int i);

// ChannelDelta and Delta: gated delta rule with one decay per head and key channel, or per head.
// LatentAttention: keys and values of all heads are projections of one cached latent per token, and one rotated key part
// is shared by the heads. Rglru: a recurrence with one real decay per channel behind a short convolution.
enum class Mixer { Attention, ChannelDelta, Delta, LatentAttention, Rglru };
inline bool is_delta(Mixer m) { return m == Mixer::ChannelDelta || m == Mixer::Delta; }
struct LayerSpec {
    Mixer mixer = Mixer::Attention;
    int heads = 0, kv_heads = 0;  // query (value) heads; key/value (query/key) heads they share
    int dim = 0, vdim = 0;        // query/key size and value size of a head
    // attention
    int chunk = 0;                // a position sees the keys of its own chunk of this many positions (0: every earlier key)
    float scale = 0.f;            // factor of the scores
    RopeSpec rope;
    // latent attention (dim: the unrotated part of a head's query and key)
    int rot_dim = 0, kv_rank = 0, q_rank = 0;
    int kv_from = -1;             // >= 0: reads what that earlier layer cached instead of caching rows of its own
    // recurrent mixers
    int conv = 0;                 // taps of the short causal convolution
    // real-gated linear recurrence
    int lru_width = 0, lru_blocks = 0;  // channels; equal parts of them that share a gate matrix
    // feed-forward of `ff` columns (0: none): dense and SiLU-gated, or (experts > 0) a mixture of squared-ReLU experts
    int experts = 0, identity = 0, top = 0, ff = 0;
    // channels that go into the mixer's output projection
    int out_cols() const { return mixer == Mixer::Rglru ? lru_width : heads * vdim; }
};
// How a layer puts its sublayers on the residual stream.
enum class Block {
    PostNorm,  // x += norm(mixer(norm(x))), then x += norm(ff(norm(x)))
    Parallel,  // x += residual_mult * (mixer(norm1(x)) + ff(norm2(x))), both of the same x
};

struct Config {
    std::string family = "Qwen2";   // name in the model registry (model_families)
    std::vector<LayerSpec> layers;  // empty: the uniform Qwen2 stack
    int hidden_size = 896, intermediate_size = 4864, num_layers = 24, num_heads = 14, num_kv_heads = 2;
    int head_dim = 64, vocab_size = 151936, max_seq_len = 131072;
    float rms_norm_eps = 1e-6f, rope_theta = 1e6f;
    int eos_token_id = 151645, bos_token_id = 151643;
    bool tie_embeddings = true;
    // layer lists
    Block block = Block::PostNorm;
    float residual_mult = 1.f, logit_scale = 1.f;
    bool embed_norm = false;        // the residual stream starts with the normed embedding
};
Config read_config(const std::string& model_dir);

// The model registry: which families exist, how a config.json is recognised and read. Loading the weights is
// Model::load's table of the same names (engine.cu).
struct ModelFamily {
    const char* name;
    bool (*claims)(const JsonValue& config);
    Config (*read)(const JsonValue& config);
};
const std::vector<ModelFamily>& model_families();

// What one tensor-parallel rank owns. The reference is single-GPU; these are the slices of its matrices
// (q/k/v rows by head: inference/src/model/qwen.cu:317-319; o_proj columns: :413-415; gate/up rows and down
// columns on the intermediate dimension for the base FFN: :431-437 and for the expert:
// inference/src/model/expert.cu:51-58; LM-head rows on the vocabulary: qwen.cu:450-454).
// Heads are kept together with their kv head: with tp_size <= kv heads every rank takes whole kv groups;
// with more ranks than kv heads, tp_size / kv_heads ranks share a kv head (each computes its K/V row
// itself) and split its query heads as evenly as they go (7 heads over 2 ranks: 3 + 4).
struct TpPartition {
    int tp_rank = 0, tp_size = 1;
    int q_head0 = 0, n_q_heads = 0;    // first global query head, count (all of one kv group when kv heads are shared)
    int kv_head0 = 0, n_kv_heads = 0;  // first global kv head, count
    int i0 = 0, n_i = 0;               // rows of gate/up and columns of down (multiples of 64)
    int v0 = 0, n_v = 0;               // rows of the LM head (multiples of 8)
};
TpPartition tp_partition(const Config& c, int tp_rank, int tp_size);  // kErrUnsupported if the shape does not split

// One memory-mapped .safetensors file: u64 LE header length, JSON header, raw data
// (inference/src/io/safetensors.cpp:41-78). "__metadata__" is skipped.
struct TensorInfo {
    std::string dtype;
    std::vector<int64_t> shape;
    const uint8_t* data = nullptr;
    size_t nbytes = 0;
};
class SafeTensorsFile {
public:
    explicit SafeTensorsFile(const std::string& path);
    ~SafeTensorsFile();
    SafeTensorsFile(const SafeTensorsFile&) = delete;
    SafeTensorsFile& operator=(const SafeTensorsFile&) = delete;
    std::unordered_map<std::string, TensorInfo> tensors;
    std::string path;

private:
    void* map_ = nullptr;
    size_t size_ = 0;
    int fd_ = -1;
};
// Every *.safetensors of a directory, shards in sorted-name order; a name resolves to the
// first shard that holds it (inference/src/io/safetensors.cpp:104-131).
class SafeTensorsDir {
public:
    explicit SafeTensorsDir(const std::string& dir);
    ~SafeTensorsDir();
    bool has(const std::string& name) const;
    const TensorInfo& get(const std::string& name) const;  // throws kErrFormat "Missing tensor"
    // BF16 tensor with exactly `elems` elements, else throws (the reference checks the byte
    // size only: inference/src/model/qwen.cu:69-78)
    const uint16_t* bf16(const std::string& name, size_t elems) const;
    // the same with every dimension checked
    const uint16_t* bf16(const std::string& name, std::initializer_list<int64_t> shape) const;
    size_t num_shards() const { return shards_.size(); }
    size_t num_tensors() const;

private:
    std::vector<SafeTensorsFile*> shards_;
};

// Expert checkpoint (trainer/include/io/checkpoint.h:12-24; reader inference/src/io/checkpoint.cpp:11-65):
// u32 magic 0x45585054, u32 version, u32 layers, u32 hidden, u32 intermediate, then per layer
// gate[I*H], up[I*H], down[H*I] as little-endian fp32.
constexpr uint32_t kExpertMagic = 0x45585054u;
constexpr uint32_t kExpertVersion = 1u;
struct ExpertHeader {
    uint32_t magic = 0, version = 0, num_layers = 0, hidden = 0, intermediate = 0;
};
class ExpertFile {
public:
    explicit ExpertFile(const std::string& path);  // validates magic and that the file holds every matrix
    ~ExpertFile();
    ExpertHeader hdr;
    // fp32 matrix m (0 gate, 1 up, 2 down) of layer l, memory-mapped
    const float* matrix(int layer, int m) const;
    size_t matrix_elems() const { return (size_t)hdr.hidden * hdr.intermediate; }

private:
    void* map_ = nullptr;
    size_t size_ = 0;
    int fd_ = -1;
};
// Writer of the same format (trainer/src/io/checkpoint.cpp:15-52). mats[l*3+m] -> fp32 [I*H].
void write_expert(const std::string& path, uint32_t layers, uint32_t hidden, uint32_t inter,
                  const float* const* mats);

// Round-to-nearest-even fp32 -> bf16 (what __float2bfloat16 does in the reference's loader).
inline uint16_t f32_to_bf16(float f) {
    uint32_t u;
    __builtin_memcpy(&u, &f, 4);
    if ((u & 0x7fffffffu) > 0x7f800000u) return 0x7fff;
    u += 0x7fffu + ((u >> 16) & 1u);
    return (uint16_t)(u >> 16);
}
inline float bf16_to_f32(uint16_t v) {
    uint32_t u = (uint32_t)v << 16;
    float f;
    __builtin_memcpy(&f, &u, 4);
    return f;
}

// Reference-compatible tokenizer (inference/src/io/tokenizer.cpp:16-153): vocab + merges +
// added_tokens from tokenizer.json, eos/bos from generation_config.json, per-byte lookup with
// "<0xNN>" fallback, greedy lowest-rank merge loop, decode with the byte-level space marker
// turned back into ' '. It deliberately keeps the reference's behaviour (bytes with no vocab
// entry are dropped).
class Tokenizer {
public:
    void load(const std::string& model_dir);
    std::vector<uint32_t> encode(const std::string& text) const;
    std::string decode(const std::vector<uint32_t>& ids) const;
    // The tokenisation Qwen2's tokenizer.json actually specifies, which the reference's encode() above does not
    // implement (it has no pre-tokenizer and no byte-to-unicode map, so spaces and newlines are dropped:
    // inference/src/io/tokenizer.cpp:86-108; the authors work around it with HF in tools/tokenize_correctly.py):
    // added tokens are cut out verbatim, the rest is split by the Qwen2 pre-tokenizer pattern
    //   (?i:'s|'t|'re|'ve|'m|'ll|'d)|[^\r\n\p{L}\p{N}]?\p{L}+|\p{N}| ?[^\s\p{L}\p{N}]+[\r\n]*|\s*[\r\n]+|\s+(?!\S)|\s+
    // every piece's UTF-8 bytes go through GPT-2's byte-to-unicode map, and the merges are applied lowest
    // rank first. decode_bpe maps the characters back to bytes.
    std::vector<uint32_t> encode_bpe(const std::string& text) const;
    std::string decode_bpe(const std::vector<uint32_t>& ids) const;
    uint32_t get_id(const std::string& token) const;  // 0 and a warning on stderr when absent
    uint32_t eos_id = 151645, bos_id = 151643, pad_id = 151643;
    size_t vocab_size() const { return token_to_id_.size(); }

private:
    std::unordered_map<std::string, uint32_t> token_to_id_;
    std::unordered_map<uint32_t, std::string> id_to_token_;
    std::vector<std::pair<uint32_t, uint32_t>> merges_;
    std::unordered_map<uint64_t, uint32_t> merge_rank_;
    std::vector<std::string> added_;  // added tokens, longest first
    void bpe_piece(const std::string& bytes, std::vector<uint32_t>& out) const;
};

std::string read_text_file(const std::string& path, bool* ok);

}  // namespace tffn
