// Interfaces and registries of the parts that a layer is put together from.
//
// A part is built from a PartSpec (its sizes and constants) and a Runtime (device, compute dtype,
// which kernels run the products); it never learns which model it is in.  It declares the tensors it
// needs under names of its own (tensors()), receives them (load()), and runs on the tokens of one
// step (forward()).  The kinds are looked up by name in the registries below, so a mixer,
// feed-forward, norm, position encoding, block arrangement, embedding or head is added without
// touching this library:
//
//     struct MyMixer : illm::Mixer { ... };
//     illm::register_mixer("my_mixer", [](const PartSpec& s, Runtime* rt) { return std::unique_ptr<Mixer>(new MyMixer(s, rt)); });
//
// (or through the C entry points of binding/c_api.h, which let a part be written in another language).
// The reference has the same seam one level lower: modules take their sizes as constructor arguments
// and own their weights by name (AttentionModule, LlamaFFNModule, src/core/graph.h:84-123,
// src/core/graph.cpp:57-79).
#pragma once
#include <functional>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "cache/cache.h"
#include "config/config.h"
#include "kernels/ops.h"

namespace illm {

struct PositionTable;

// Where and in which precision a model runs.  `dtype` is the dtype of activations, matrices and
// cache pages: bfloat16 (serving) or float32 (everything in true 32-bit).
struct Runtime {
    Device* dev = nullptr;
    DType dtype = DType::BF16;
    int page_size = 64;
    ops::GemmBackend gemm = ops::GemmBackend::Auto;
    bool is_f32() const { return dtype == DType::F32; }
    // cos/sin tables of rotary encodings, one per distinct (theta, rot_dim, positions) of the model:
    // layers with the same encoding share a table
    std::map<std::string, std::shared_ptr<PositionTable>> position_tables;
};

// A tensor that a part needs.  init: "matrix" -> N(0, 0.02); "norm" -> 1 + N(0, 0.02); "int" -> an
// integer table (kept int32).  Used by the loader to check shapes and by the random-weights writer.
struct TensorDecl {
    std::vector<long long> shape;      // a size of -1 is whatever the weight file has (the part reads it at load)
    std::string init = "matrix";
    // true: a weight file may leave the tensor out (the part then does without it); random models have none
    bool optional = false;
    long long numel() const { long long n = 1; for (long long s : shape) n *= s; return n; }
};
using TensorDecls = std::vector<std::pair<std::string, TensorDecl>>;     // in the part's own order

// Persistent device memory owned by a part.
class DeviceBuffer {
public:
    DeviceBuffer() {}
    DeviceBuffer(Device* dev, size_t bytes, const char* what) : dev_(dev), p_(dev->alloc_persistent(bytes, what)), bytes_(bytes) {}
    ~DeviceBuffer() { reset(); }
    DeviceBuffer(DeviceBuffer&& o) noexcept : dev_(o.dev_), p_(o.p_), bytes_(o.bytes_) { o.p_ = nullptr; }
    DeviceBuffer& operator=(DeviceBuffer&& o) noexcept {
        if (this != &o) { reset(); dev_ = o.dev_; p_ = o.p_; bytes_ = o.bytes_; o.p_ = nullptr; }
        return *this;
    }
    void reset() { if (p_ && dev_) dev_->free_persistent(p_); p_ = nullptr; }
    void* get() const { return p_; }
    size_t bytes() const { return bytes_; }
private:
    Device* dev_ = nullptr;
    void* p_ = nullptr;
    size_t bytes_ = 0;
};

// Where a part's tensors come from at load: a weight file or the random generator.  Names are the
// part's own (the model adds the prefix).
class TensorSource {
public:
    virtual ~TensorSource() {}
    // The dtype the tensor is kept in by the storage rule: 16-bit floats -> bfloat16, a tensor stored
    // in 32-bit stays so, integers -> int32; in the float32 mode every float is widened to float32.
    virtual DType kept_dtype(const std::string& name) = 0;
    // Bring the tensor to the device as `want` (float32 or bfloat16 for floats, int32 for integer
    // tables) into dst, whose rows are `dst_row_elems` elements apart (0: contiguous).
    virtual void fetch_into(const std::string& name, void* dst, DType want, long long dst_row_elems = 0) = 0;
    virtual std::vector<long long> shape(const std::string& name) = 0;
    // whether the source has the tensor at all (asked for tensors that were declared optional)
    virtual bool has(const std::string& name) { return true; }
};

// A matrix owned by a part: a fresh persistent buffer filled from the source.
struct OwnedMat {
    DeviceBuffer buf;
    Mat m;
};
OwnedMat fetch_owned(Runtime* rt, TensorSource& src, const std::string& name, DType want, const char* what);

class Part {
public:
    Part(PartSpec s, Runtime* runtime) : spec(std::move(s)), rt(runtime) {}
    virtual ~Part() {}
    virtual TensorDecls tensors() const { return {}; }
    // Receive the declared tensors and bring them into the form the kernels want.
    virtual void load(TensorSource&) {}
    PartSpec spec;
    Runtime* rt;      // nullptr: the part only declares its tensors (checking a folder, writing a random one)
};

// The step as the parts see it: the device-side arrays (StepView) and, for parts that need them on
// the host, the step's lengths.  A part that reads the host fields cannot be replayed from a graph
// (see Mixer::graph_safe).
struct StepContext : StepView {
    Device* dev = nullptr;
    Runtime* rt = nullptr;
    std::vector<int> q_lens, host_slots;
    std::vector<long long> past;
    // What a layer keeps for later layers of the same step, by name: `keep` makes a float32 matrix in memory that outlives
    // the layers' own activations (lane 0 of the step arena).  Emptied when a step's forward pass begins.
    mutable std::map<std::string, Mat> kept;
    Mat keep(const std::string& name, long long rows, long long cols) const {
        Mat m;
        m.rows = m.rows_held = rows;
        m.cols = cols;
        m.dtype = DType::F32;
        const int lane = dev->lane();
        dev->set_lane(0, false);
        m.p = dev->alloc(m.bytes());
        dev->set_lane(lane, false);
        kept[name] = m;
        return m;
    }
};

// What a mixer gets of its cache entry for the step.
struct CacheView {
    enum Kind { None, KV, State } kind = None;
    KVView kv;
    StateView st;
    // the second, fixed-state entry of a mixer that asked for one (Mixer::aux_cache_request)
    bool has_aux = false;
    StateView aux;
};

// The float32 residual stream [T, H] with an addition pending (or two: the sublayers of a parallel block).  A part's
// output is not added at once: the next norm adds it while it reads the row anyway (one kernel for add + norm), which is
// also where the sum is rounded: never, it stays float32.
class Norm;
struct ResidualStream {
    Device* dev = nullptr;
    Mat x;
    bool has_pending = false, has_pending2 = false;
    MatOrPartials pending, pending2;
    // a norm that the pending addition passes on its way into the stream (a block that norms a sublayer's output):
    // x + pending_post(pending); the next norm of the same kind does both in one kernel, flush() asks the norm itself
    Norm* pending_post = nullptr;
    Mat h;      // the stream's rows in the compute dtype, where a block keeps them (norm after the sum); empty otherwise
    void add(const MatOrPartials& delta) {
        if (has_pending || has_pending2) flush();
        pending = delta;
        has_pending = true;
    }
    // x + post(delta): delta a finished float32 matrix
    void add_normed(const MatOrPartials& delta, Norm* post) {
        add(delta);
        pending_post = post;
    }
    // A second addition behind a pending one, both finished matrices: x + pending + delta, added in that order by flush()
    // or by a norm that folds both in.  Anything else is added like add().
    void add_second(const MatOrPartials& delta) {
        if (has_pending && !has_pending2 && !pending.is_partials() && !delta.is_partials()) {
            pending2 = delta;
            has_pending2 = true;
        } else {
            add(delta);
        }
    }
    Mat& flush();
};

class Norm : public Part {
public:
    using Part::Part;
    // Fold the stream's pending addition in and return the normed rows in the compute dtype; `rows`
    // (int32, device) restricts it to those rows (the stream itself is then left as it is).
    virtual Mat forward(ResidualStream& stream, const int* rows, long long n_rows) = 0;
    // Norm after the sum: stream.x <- norm(residual_scale * stream.x + pending), the norm's own
    // residual_scale; the normed rows ARE the stream from then on, and they are also returned in the
    // compute dtype for the sublayer that reads them next.  Only norms that can do this override it.
    // false for a norm whose optional weight was not in the file: the block leaves the norm out
    virtual bool present() const { return true; }
    virtual Mat forward_into_stream(ResidualStream& stream) { throw EngineError("norm '" + spec.kind + "' cannot replace the stream by its output"); }
    // stream.x += norm(stream.pending), for the norm a sublayer's output passes before it joins the stream
    // (ResidualStream::add_normed); only norms that can stand there override it.
    virtual void add_normed_pending(ResidualStream& stream) { throw EngineError("norm '" + spec.kind + "' cannot norm a sublayer's output into the stream"); }
    // The same, and the new rows of the stream in the compute dtype, for a block whose sublayers read the stream as it is
    // (nothing comes back unless `want_rows`; in the float32 mode it is the stream itself).
    virtual Mat join_stream(ResidualStream& stream, bool want_rows) { throw EngineError("norm '" + spec.kind + "' cannot norm a sublayer's output into the stream"); }
    // A part that stands behind a sublayer and is nothing but a factor per channel (a layer scale) gives its float32
    // factors [size] here, so that the next norm can fold x + factors * pending into its own kernel.
    virtual const Mat* channel_scale() const { return nullptr; }
};

inline Mat& ResidualStream::flush() {
    if (has_pending && pending_post) {
        Norm* post = pending_post;
        pending_post = nullptr;
        post->add_normed_pending(*this);       // adds and clears the pending addition
    }
    if (has_pending) ops::residual_add(*dev, x, pending);
    if (has_pending2) ops::residual_add(*dev, x, pending2);
    has_pending = has_pending2 = false;
    pending_post = nullptr;
    return x;
}

class PositionEncoding : public Part {
public:
    using Part::Part;
    // true: encode_and_store also takes the packed projection as unreduced slices of a split matrix
    // product and adds them up itself.  false (default): it always gets a finished matrix.
    virtual bool takes_partials() const { return false; }
    virtual void prepare() {}     // build device tables; called once after construction on a device
    // true if all this encoding does is the rotate-half rotation of the first rot_dim channels of every
    // Q and K head by angles from a cos/sin table float32 [positions, rot_dim / 2, 2] (rot_dim 0: nothing
    // at all), so that a mixer whose kernel can do that itself may skip encode_and_store.
    virtual bool rotation_table(const float** table, int* rot_dim, long long* n_pos) const { return false; }
    // The same for either pairing of the channels: true if the encoding is a rotation of the first rot_dim
    // channels of every head by table angles, *pairs saying whether channel 2j goes with 2j + 1 (true) or
    // j with j + rot_dim / 2 (false).  A mixer with a kernel of its own between projection and attention
    // (biases, norms) asks this and does the rotation there.
    virtual bool table_rotation(const float** table, int* rot_dim, long long* n_pos, bool* pairs) const {
        *pairs = false;
        return rotation_table(table, rot_dim, n_pos);
    }
    // Encode positions into the Q and K heads of the packed projection and store the new K and V in the
    // cache (if kv.writes).  Returns the matrix that holds the encoded queries in its first
    // heads * head_dim columns: qkv itself (encoded in place) or, for unreduced slices, a new one.
    virtual Mat encode_and_store(const MatOrPartials& qkv, ops::Geometry g, const StepContext& ctx, const KVView& kv) = 0;
};

class Mixer : public Part {
public:
    using Part::Part;
    // true promises that a one-token-per-sequence step launches the same kernels with the same
    // arguments whenever the batch size is the same (everything that varies is read from device
    // memory), so the engine may capture it in a CUDA graph.  A mixer that reads host-side fields of
    // the step context (q_lens, past, ...) says false.
    virtual bool graph_safe() const { return false; }
    // true when tokens appended behind a sequence's real tokens in a step change nothing that is kept
    // (they may leave keys and values behind the sequence's length in its own pages, which the next
    // tokens overwrite) and nothing the real tokens get back, and when a step of many tokens of one
    // sequence launches the same kernels whenever the token count is the same.  The engine then pads
    // single prompts to whole buckets of tokens and replays them from captured graphs.
    virtual bool pad_safe() const { return false; }
    virtual CacheRequest cache_request() const { return CacheRequest(); }
    // A second cache entry, of fixed per-sequence state, beside the first (a mixer with keys and values AND a few
    // rows of state, say): the decoder gives it an entry number of its own and hands it over as CacheView::aux.
    virtual CacheRequest aux_cache_request() const { return CacheRequest(); }
    // Which earlier positions the mixer's queries see (0, 0: all; as in CacheRequest), for a mixer that attends to keys and
    // values which another layer wrote: the cache keeps every position that one of the entry's readers still needs.
    struct Reach { bool known = false; int window = 0, chunk = 0; };
    virtual Reach reach() const { return Reach(); }
    // true: in a block whose sublayers read the stream as it is, forward() gets the float32 stream instead of its rows in
    // the compute dtype
    virtual bool reads_stream() const { return false; }
    // h [T, H] in the compute dtype -> [T, H].  `may_defer`: the result may be the unreduced slices of
    // a split matrix product, for a caller that only adds it to the residual stream.
    virtual MatOrPartials forward(const Mat& h, const StepContext& ctx, const CacheView& cache, bool writes, bool may_defer) = 0;
};

class FeedForward : public Part {
public:
    using Part::Part;
    virtual bool graph_safe() const { return true; }
    virtual MatOrPartials forward(const Mat& h, const StepContext& ctx, bool may_defer) = 0;
};

class EmbeddingPart : public Part {
public:
    using Part::Part;
    virtual ResidualStream forward(const StepContext& ctx) = 0;     // ctx.ids -> the float32 stream [T, H]
    virtual const Mat* table() const { return nullptr; }            // what a tied head may use
    // An embedding that depends on earlier tokens of the sequence keeps per-sequence state: it asks for a cache
    // entry of its own here and is then run through forward_with_state.
    virtual CacheRequest cache_request() const { return CacheRequest(); }
    virtual ResidualStream forward_with_state(const StepContext& ctx, const CacheView&) { return forward(ctx); }
    // false if tokens appended behind a sequence's real ones would change what is kept (see Mixer::pad_safe)
    virtual bool pad_safe() const { return true; }
};

class HeadPart : public Part {
public:
    using Part::Part;
    virtual bool tied() const { return false; }
    virtual void tie(const EmbeddingPart&) {}
    virtual Mat forward(const Mat& y, const StepContext& ctx) = 0;  // normed rows -> float32 logits [rows, vocab]
};

// An arrangement of norms, a mixer and a feed-forward around the residual stream.
class Block {
public:
    virtual ~Block() {}
    Mixer* mixer = nullptr;
    FeedForward* ffn = nullptr;
    std::map<std::string, Norm*> norms;
    virtual void forward(ResidualStream& stream, const StepContext& ctx, const CacheView& cache, bool writes) = 0;
};
struct BlockKind {
    std::vector<std::string> norm_roles;                   // keys of LayerSpec::norms and LayerSpec::names
    std::function<std::unique_ptr<Block>()> make;
};

// ---- registries

template <typename T> using PartFactory = std::function<std::unique_ptr<T>(const PartSpec&, Runtime*)>;
void register_mixer(const std::string& kind, PartFactory<Mixer> f);
void register_feed_forward(const std::string& kind, PartFactory<FeedForward> f);
void register_norm(const std::string& kind, PartFactory<Norm> f);
void register_position(const std::string& kind, PartFactory<PositionEncoding> f);
void register_embedding(const std::string& kind, PartFactory<EmbeddingPart> f);
void register_head(const std::string& kind, PartFactory<HeadPart> f);
void register_block(const std::string& kind, BlockKind k);
void unregister_part(const std::string& family, const std::string& kind);
std::vector<std::string> registered_parts(const std::string& family);

// ConfigError "unknown <family> kind '...'; registered: ..." for a kind that is not there.
std::unique_ptr<Mixer> build_mixer(const PartSpec& s, Runtime* rt);
std::unique_ptr<FeedForward> build_feed_forward(const PartSpec& s, Runtime* rt);
std::unique_ptr<Norm> build_norm(const PartSpec& s, Runtime* rt);
std::unique_ptr<PositionEncoding> build_position(const PartSpec& s, Runtime* rt);
std::unique_ptr<EmbeddingPart> build_embedding(const PartSpec& s, Runtime* rt);
std::unique_ptr<HeadPart> build_head(const PartSpec& s, Runtime* rt);
const BlockKind& lookup_block(const std::string& kind);

// A cos/sin table of a rotate-half encoding on the device: float32 [positions, rot_dim / 2, 2],
// angles p * theta^(-2j / rot_dim) computed in float64 on the host.
struct PositionTable {
    DeviceBuffer buf;
    long long positions = 0;
    int rot_dim = 0;
    const float* data() const { return (const float*)buf.get(); }
};
std::shared_ptr<PositionTable> shared_position_table(Runtime* rt, double theta, int rot_dim, long long positions);
// The general form: entry (p, j) = magnitude * (cos, sin)(p * freqs[j]), freqs of rot_dim / 2 pairs.
std::shared_ptr<PositionTable> shared_position_table(Runtime* rt, const std::vector<double>& freqs, double magnitude, long long positions);
// Frequencies theta^(-2j / rot_dim), optionally blended with the ones stretched by `factor`: along a
// linear ramp over the pair index (the "YaRN" scaling {factor, original, fast, slow}: pairs that turn more than `fast` times
// within `original` positions keep their frequency, pairs that turn less than `slow` times are stretched;
// *magnitude gets the factor 0.1 ln(factor) + 1 that goes with it), or along a ramp over the turns themselves (the scaling of
// Llama 3.1, {factor, original, low, high}: pairs that turn more than `high` times within `original` positions keep their
// frequency, pairs that turn less than `low` times are stretched, linear in the number of turns between; *magnitude is 1, as
// it is without scaling).
std::vector<double> rotary_frequencies(double theta, int rot_dim, const Json* scaling, double* magnitude);

}  // namespace illm
