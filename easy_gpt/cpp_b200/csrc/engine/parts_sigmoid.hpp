// Further parts: sines and cosines of the position added to the embedding; attention whose weights are sigmoids of the scores,
// with a bias by distance, a norm over whole projections, a query temperature and a gate per head; linear attention whose
// state fades by a constant of the head; and the generalised delta rule with a decay and a removal rate per key channel.
// Each takes its sizes, constants and tensor-name suffixes from its parameters and knows nothing of the model around it.
#pragma once
#include "../host/distance_bucket.hpp"
#include "parts_delta.hpp"

namespace easygpt::engine {

// the rows of several matrices [., in] under one another, filled up with zero rows to a multiple of 16 (every row of the
// product's output then starts on a 16-byte boundary)
inline std::vector<float> stacked_rows(const HostTensors& file, const std::string& prefix, const std::vector<const char*>& names, int in, int* rows) {
    std::vector<float> w;
    for (const char* n : names) {
        const std::vector<float> part = host_floats(need_tensor(file, prefix + n));
        w.insert(w.end(), part.begin(), part.end());
    }
    *rows = (int)((w.size() / (size_t)in + 15) / 16 * 16);
    w.resize((size_t)*rows * in, 0.f);
    return w;
}

// ---- positions as waves ------------------------------------------------------------------------------------------------------
// stream[p, 2i] += sin(p base^(-2i / width)), stream[p, 2i + 1] += cos(the same), right behind the embedding.
// Parameters: size, base.
class WavePositions : public PositionEncoding {
public:
    WavePositions(const Params& p, const std::string& prefix) : PositionEncoding(p, prefix), size_((int)p.integer("size")), base_(p.real("base", 10000.0)) {
        if (size_ <= 0 || base_ <= 0.0) throw std::invalid_argument("wave positions: size and base must be positive");
    }
    void load(const HostTensors&, DType) override {
        const int pairs = (size_ + 1) / 2;
        std::vector<float> head(pairs), tail(pairs);
        for (int i = 0; i < pairs; ++i) {
            const double f = std::pow(base_, -2.0 * i / size_);
            head[i] = (float)f;
            tail[i] = (float)(f - (double)head[i]);
        }
        head_ = upload(head.data(), head.size(), DType::F32);
        tail_ = upload(tail.data(), tail.size(), DType::F32);
    }
    bool capturable() const override { return true; }
    void add_to_embedding(float* residual, const StepContext& ctx) const override {
        launch_check(eg_add_waves(ctx.stream, residual, ctx.positions, head_.as<float>(), tail_.as<float>(), ctx.num_tokens, size_), "add_waves");
    }

private:
    int size_;
    double base_;
    DeviceBuffer head_, tail_;
};

// ---- attention with sigmoid weights --------------------------------------------------------------------------------------------
// H heads with queries of `dim` values, G key/value heads (head h reads head h / (H / G)) with keys of `dim` and values of `vdim`
// values:  q, k, v = W h + b as ONE product together with the heads' gates (rows stacked), float32 out;  with norm_eps given, q and k
// are divided by their root mean square over the WHOLE projection (norm_eps under the root) and multiplied by a gain per row
// (.q.norm [H dim], .k.norm [G dim]);  with temp_every given, q is multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1);
// score = (q . k) * scale + rel[bucket(i - j)][h] + pb[h] over all earlier keys and its own, where with B rows in .rel, half =
// floor(B / 2): bucket(n) = n below half, else min(B - 1, half + floor(ln(n / half) / ln(bias_max / half) (B - half)));
// weight = sigmoid(score), not normalised;  out = W_o (heads' sums times sigmoid(gate_h), side by side).
// Without `distance_bias` there is no .rel, without `head_bias` no .pb, without `head_gate` no .g, without `proj_bias` no biases.
// The cache keeps one row (key | value) per token and key head, where dim = vdim planes of their own.  float32 and sizes that are
// no multiples of 8 run on the generic kernel; bfloat16 runs on the tensor cores (attention_tcgen05.cu for longer prompt portions of
// heads of 64 and 128, else attention_sigmoid.cu).
// Parameters: hidden_size, heads, kv_heads, dim, vdim, scale, norm_eps, temp_coef, temp_every, bias_max, distance_bias, head_bias,
// head_gate, proj_bias.  Tensors: .q .k .v .o (+ .q.b .k.b .v.b, .q.norm .k.norm, .rel, .pb, .g).
class SigmoidAttention : public Mixer {
public:
    SigmoidAttention(const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> position)
        : Mixer(p, prefix, std::move(position)), hidden_((int)p.integer("hidden_size")), heads_((int)p.integer("heads")), kv_heads_((int)p.integer("kv_heads")),
          dk_((int)p.integer("dim")), dv_((int)p.integer("vdim")), scale_((float)p.real("scale")), norm_eps_((float)p.real("norm_eps", -1.0)),
          temp_coef_((float)p.real("temp_coef", 0.0)), temp_every_((int)p.integer("temp_every", 0)), bias_max_(p.real("bias_max", 0.0)),
          distance_bias_(p.integer("distance_bias", 0) != 0), head_bias_(p.integer("head_bias", 0) != 0), head_gate_(p.integer("head_gate", 0) != 0),
          proj_bias_(p.integer("proj_bias", 0) != 0) {
        if (hidden_ <= 0 || heads_ <= 0 || kv_heads_ <= 0 || dk_ <= 0 || dv_ <= 0) throw std::invalid_argument("sigmoid attention: sizes must be positive");
        if (heads_ % kv_heads_) throw std::invalid_argument("sigmoid attention: heads must be a multiple of kv_heads");
        if (temp_every_ < 0) throw std::invalid_argument("sigmoid attention: temp_every must not be negative");
        if (distance_bias_ && bias_max_ <= 0.0) throw std::invalid_argument("sigmoid attention: a distance bias needs a positive bias_max");
        if (dv_ > 256 || dk_ > 2048) throw std::invalid_argument("sigmoid attention: vdim up to 256 and dim up to 2048 are what the kernels take");
        if (this->position) throw std::invalid_argument("sigmoid attention takes no rotation");
    }
    std::vector<TensorRequest> tensor_requests() const override {
        const long long nq = (long long)heads_ * dk_, nk = (long long)kv_heads_ * dk_, nv = (long long)kv_heads_ * dv_;
        std::vector<TensorRequest> r = {TensorRequest::matrix(prefix + ".q", nq, hidden_), TensorRequest::matrix(prefix + ".k", nk, hidden_),
                                        TensorRequest::matrix(prefix + ".v", nv, hidden_), TensorRequest::matrix(prefix + ".o", hidden_, (long long)heads_ * dv_)};
        if (proj_bias_) {
            r.push_back(TensorRequest::vector(prefix + ".q.b", nq));
            r.push_back(TensorRequest::vector(prefix + ".k.b", nk));
            r.push_back(TensorRequest::vector(prefix + ".v.b", nv));
        }
        if (norm_eps_ >= 0.f) {
            r.push_back(TensorRequest::vector(prefix + ".q.norm", nq).with_init("one"));
            r.push_back(TensorRequest::vector(prefix + ".k.norm", nk).with_init("one"));
        }
        if (distance_bias_) r.push_back(TensorRequest::matrix(prefix + ".rel", 32, heads_).with_free_dim(0));
        if (head_bias_) r.push_back(TensorRequest::vector(prefix + ".pb", heads_));
        if (head_gate_) r.push_back(TensorRequest::matrix(prefix + ".g", heads_, hidden_));
        return r;
    }
    void load(const HostTensors& file, DType dtype) override {
        std::vector<const char*> names = {".q", ".k", ".v"};
        if (head_gate_) names.push_back(".g");
        int rows = 0;
        const std::vector<float> w = stacked_rows(file, prefix, names, hidden_, &rows);
        std::vector<float> b;
        if (proj_bias_) {
            for (const char* n : {".q.b", ".k.b", ".v.b"}) {
                const std::vector<float> part = host_floats(need_tensor(file, prefix + n));
                b.insert(b.end(), part.begin(), part.end());
            }
            b.resize((size_t)rows, 0.f);
        }
        in_ = Linear(w.data(), rows, hidden_, proj_bias_ ? b.data() : nullptr, dtype);
        out_ = Linear(need_tensor(file, prefix + ".o"), nullptr, dtype);
        if (norm_eps_ >= 0.f) {
            q_gain_ = upload_f32(file, prefix + ".q.norm");
            k_gain_ = upload_f32(file, prefix + ".k.norm");
        }
        // the bias by distance and head, up to the first distance from which on it no longer changes
        std::vector<float> rel, pb((size_t)heads_, 0.f);
        reach_ = 1;
        int buckets = 0;
        if (distance_bias_) {
            const StoredTensor& t = need_tensor(file, prefix + ".rel");
            rel = host_floats(t);
            buckets = (int)t.shape[0];
            while (host::distance_bucket(reach_ - 1, buckets, bias_max_) < buckets - 1) ++reach_;
        }
        if (head_bias_) pb = host_floats(need_tensor(file, prefix + ".pb"));
        const float log2e = 1.4426950408889634f;
        std::vector<float> table((size_t)heads_ * reach_);
        for (int n = 0; n < reach_; ++n)
            for (int h = 0; h < heads_; ++h)
                table[(size_t)h * reach_ + n] = (distance_bias_ ? rel[(size_t)host::distance_bucket(n, buckets, bias_max_) * heads_ + h] : 0.f) + pb[h];
        mma_ = dtype == DType::BF16 && eg_sigmoid_attention_mma_takes(dk_, dv_, reach_);
        if (mma_)
            for (float& v : table) v *= -log2e;               // the tensor-core kernels work on negated scores in base 2
        table_ = upload(table.data(), table.size(), DType::F32);
    }
    size_t weight_bytes() const override { return in_.weight_bytes() + out_.weight_bytes(); }
    size_t arena_bytes(long long T) const override {
        // partial sums of single tokens whose keys are dealt to several CTAs: bounded by the CTAs of a few waves
        const size_t partials = plans::PREFILL_PARTS_SCRATCH_BYTES + (size_t)(4 * plans::sm_count() + 64) * 128 * (size_t)(dv_ + 2) * 4;
        return (size_t)T * ((size_t)in_.out_features * 4 + (size_t)heads_ * (dk_ + dv_) * 4 + (size_t)hidden_ * 4) + partials + (1u << 16);
    }
    bool capturable() const override { return true; }
    bool planes() const { return dk_ == dv_; }
    CacheNeed cache_need() const override { return planes() ? CacheNeed::paged(kv_heads_, dk_, -1) : CacheNeed::paged_joint(kv_heads_, dk_, dv_, -1); }

    Delta forward(const StepContext& ctx, PartInput in, const CacheView& cache, const FollowingNorm*) override {
        const int T = ctx.num_tokens;
        const DType dtype = ctx.dtype;
        if (cache.group < 0) throw DeviceError("sigmoid attention was handed no paged cache");
        const GroupTables& tables = ctx.groups.at(cache.group);
        const Rows h = in.pending ? in.pending->materialize() : in.rows;
        const float* bias = nullptr;                                          // what the product left for its consumer
        const Rows proj = in_.f32_bias_pending(ctx, h, &bias);
        Rows q{ctx.take_rows(T, heads_ * dk_, dtype), dtype, T, heads_ * dk_, heads_ * dk_};
        void* values = planes() ? cache.v : (char*)cache.k + (size_t)dk_ * dtype_size(dtype);
        const int row_stride = planes() ? dk_ : dk_ + dv_;
        launch_check(eg_sigmoid_attention_prepare(ctx.stream, (int)dtype, (const float*)proj.p, proj.ld, bias, norm_eps_ >= 0.f ? q_gain_.as<float>() : nullptr,
                                                  norm_eps_ >= 0.f ? k_gain_.as<float>() : nullptr, norm_eps_, temp_coef_, temp_every_, ctx.positions, tables.slot_map,
                                                  cache.writes ? cache.k : nullptr, values, row_stride, cache.head_stride, cache.page_size, cache.page_stride,
                                                  (long long)cache.num_pages * cache.page_size, q.p, T, heads_, kv_heads_, dk_, dv_, ctx.status),
                     "sigmoid_attention_prepare");
        Rows attn{ctx.take_rows(T, heads_ * dv_, dtype), dtype, T, heads_ * dv_, heads_ * dv_};
        const float* gate = head_gate_ ? (const float*)proj.p + (size_t)(heads_ + kv_heads_) * dk_ + (size_t)kv_heads_ * dv_ : nullptr;
        if (mma_ && cache.head_stride % 8 == 0 && cache.page_stride % 8 == 0) {
            // prompt portions in tiles of query tokens: on tcgen05 where they are long enough to fill its 128-row tiles (heads of 64 and 128,
            // keys and values of one size), else on the warp-level tensor cores; single tokens split over their keys
            if (ctx.query_tiles && planes() && reach_ <= eg_attention_prefill_tcgen05_sigmoid_reach() && ctx.max_query_len >= plans::TCGEN05_ATTENTION_MIN_QUERY &&
                plans::attention_prefill_tcgen05_takes(dtype, dk_, cache.page_size)) {
                int parts, part_tiles;
                plans::attention_prefill_parts(ctx.num_tiles, heads_, dk_, ctx.max_context_len, &parts, &part_tiles);
                const size_t slots = (size_t)ctx.num_tiles * heads_;
                while (parts > 1 && slots * parts * 128 * (dk_ + 2) * 4 > plans::PREFILL_PARTS_SCRATCH_BYTES) --parts;
                float *partial_o = nullptr, *partial_ml = nullptr;
                if (parts > 1) {
                    partial_o = ctx.take<float>(slots * parts * 128 * dk_);
                    partial_ml = ctx.take<float>(slots * parts * 128 * 2);
                }
                launch_check(eg_attention_prefill_tcgen05_sigmoid(ctx.stream, q.p, q.ld, T, cache.k, cache.v, tables.block_table, tables.table_width, ctx.positions,
                                                                  ctx.query_tiles, ctx.num_tiles, attn.p, attn.ld, heads_, kv_heads_, dk_, cache.page_size,
                                                                  cache.page_stride, cache.head_stride, cache.num_pages, scale_, table_.as<float>(), reach_, gate,
                                                                  proj.ld, ctx.status, parts, part_tiles, partial_o, partial_ml,
                                                                  ctx.scratch->prefill_queue.as<int>()), "attention_prefill_tcgen05_sigmoid");
            } else if (ctx.query_tiles) {
                launch_check(eg_sigmoid_attention_tiles(ctx.stream, q.p, cache.k, values, row_stride, cache.head_stride, tables.block_table, tables.table_width,
                                                        ctx.positions, ctx.query_tiles, ctx.num_tiles, table_.as<float>(), reach_, gate, proj.ld, attn.p, attn.ld,
                                                        heads_, kv_heads_, dk_, dv_, cache.page_size, cache.page_stride, cache.num_pages, scale_, ctx.status),
                             "sigmoid_attention_tiles");
            }
            const int singles = ctx.query_tiles ? ctx.num_small : T;
            if (singles > 0) {
                const int blocks = (heads_ / kv_heads_ + 15) / 16 * kv_heads_;
                int splits = plans::attention_paged_splits(singles, heads_, kv_heads_, ctx.max_context_len, dk_);
                float* partial = nullptr;
                int* counters = nullptr;
                if (splits > 1 && (size_t)singles * blocks > KernelScratch::ATTENTION_COUNTERS) splits = 1;
                if (splits > 1) {
                    partial = ctx.take<float>((size_t)singles * heads_ * splits * dv_);
                    counters = ctx.scratch->attention_counters.as<int>();
                }
                launch_check(eg_sigmoid_attention_split(ctx.stream, q.p, cache.k, values, row_stride, cache.head_stride, tables.block_table, tables.table_width,
                                                        ctx.token_seq, ctx.positions, ctx.query_tiles ? ctx.small_tokens : nullptr, singles, table_.as<float>(), reach_,
                                                        gate, proj.ld, attn.p, attn.ld, partial, counters, splits, heads_, kv_heads_, dk_, dv_, cache.page_size,
                                                        cache.page_stride, cache.num_pages, scale_, ctx.status), "sigmoid_attention_split");
            }
        } else {
            if (mma_) throw DeviceError("sigmoid attention: a cache whose rows do not start on 16-byte boundaries");
            launch_check(eg_sigmoid_attention(ctx.stream, (int)dtype, q.p, cache.k, values, row_stride, cache.head_stride, tables.block_table, tables.table_width,
                                              ctx.token_seq, ctx.positions, table_.as<float>(), reach_, gate, proj.ld, attn.p, attn.ld, T, heads_, kv_heads_, dk_, dv_,
                                              cache.page_size, cache.page_stride, cache.num_pages, scale_, ctx.status), "sigmoid_attention");
        }
        const Rows o = out_(ctx, attn, /*out_f32=*/true);
        Delta d;
        d.p = o.p;
        d.dtype = o.dtype;
        return d;
    }

private:
    int hidden_, heads_, kv_heads_, dk_, dv_;
    float scale_, norm_eps_, temp_coef_;
    int temp_every_;
    double bias_max_;
    bool distance_bias_, head_bias_, head_gate_, proj_bias_, mma_ = false;
    int reach_ = 1;
    Linear in_, out_;
    DeviceBuffer q_gain_, k_gain_, table_;
};

// ---- linear attention with a state that fades by a constant -------------------------------------------------------------------
// q, k, v = silu(W h), H heads of `dim` (queries, keys) and `vdim` (values) values, and g = W_g h as ONE product, float32 out;
// S <- decay_h S + k v^T;  o = S^T q  (S [dim, vdim] per head, float32, in the request's slot as [H, vdim, dim]);
// out = W_o (o / rms(o) * .norm * sigmoid(g)), the root mean square over all heads' values together (eps under the root).
// Parameters: hidden_size, heads, dim, vdim, eps, decay.0 .. decay.(H-1).  Tensors: .q .k [H dim, hidden], .v .g [H vdim, hidden],
// .norm [H vdim], .o [hidden, H vdim].
class LightningMixer : public Mixer {
public:
    LightningMixer(const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> position)
        : Mixer(p, prefix, std::move(position)), hidden_((int)p.integer("hidden_size")), heads_((int)p.integer("heads")), dk_((int)p.integer("dim")),
          dv_((int)p.integer("vdim")), eps_((float)p.real("eps")) {
        if (hidden_ <= 0 || heads_ <= 0 || dk_ <= 0 || dv_ <= 0) throw std::invalid_argument("lightning attention: sizes must be positive");
        if (dk_ > 256) throw std::invalid_argument("lightning attention: dim up to 256 is what the kernel takes");
        for (int h = 0; h < heads_; ++h) decays_.push_back(p.real("decay." + std::to_string(h)));
    }
    std::vector<TensorRequest> tensor_requests() const override {
        const long long k = (long long)heads_ * dk_, v = (long long)heads_ * dv_;
        return {TensorRequest::matrix(prefix + ".q", k, hidden_), TensorRequest::matrix(prefix + ".k", k, hidden_), TensorRequest::matrix(prefix + ".v", v, hidden_),
                TensorRequest::matrix(prefix + ".g", v, hidden_), TensorRequest::vector(prefix + ".norm", v).with_init("one"), TensorRequest::matrix(prefix + ".o", hidden_, v)};
    }
    void load(const HostTensors& file, DType dtype) override {
        int rows = 0;
        const std::vector<float> w = stacked_rows(file, prefix, {".q", ".k", ".v", ".g"}, hidden_, &rows);
        in_ = Linear(w.data(), rows, hidden_, nullptr, dtype);
        out_ = Linear(need_tensor(file, prefix + ".o"), nullptr, dtype);
        norm_w_ = upload_f32(file, prefix + ".norm");
        std::vector<float> powers;                                            // of every head's decay, from 0 to 64
        for (double d : decays_) {
            double x = 1.0;
            for (int i = 0; i <= 64; ++i, x *= d) powers.push_back((float)x);
        }
        powers_ = upload(powers.data(), powers.size(), DType::F32);
    }
    size_t weight_bytes() const override { return in_.weight_bytes() + out_.weight_bytes(); }
    size_t arena_bytes(long long T) const override {
        const size_t chunks = (size_t)(T / 64 + T / 32 + 1) * heads_ * dv_ * dk_ * 4;
        return (size_t)T * ((size_t)in_.out_features * 4 + (size_t)heads_ * dv_ * 8 + (size_t)hidden_ * 4) + chunks + (1u << 16);
    }
    bool capturable() const override { return true; }
    long long slot_floats() const { return (long long)heads_ * dv_ * dk_; }
    CacheNeed cache_need() const override { return CacheNeed::state({slot_floats()}); }

    Delta forward(const StepContext& ctx, PartInput in, const CacheView& cache, const FollowingNorm*) override {
        const int T = ctx.num_tokens;
        const DType dtype = ctx.dtype;
        if (!cache.state || cache.state_bytes_per_slot != (size_t)slot_floats() * 4) throw DeviceError("lightning attention was handed no state of its shape");
        if (!cache.writes) throw DeviceError("lightning attention cannot read another entry's state without advancing it");
        const Rows h = in.pending ? in.pending->materialize() : in.rows;
        const Rows proj = in_(ctx, h, /*out_f32=*/true);                      // [T, q | k | v | g] float32
        Rows y{ctx.take_rows(T, heads_ * dv_, dtype), dtype, T, heads_ * dv_, heads_ * dv_};
        float* o_raw = ctx.take<float>((size_t)T * heads_ * dv_);
        const int k = heads_ * dk_, v = heads_ * dv_;
        const long long in_chunks = eg_lightning_chunk_floats(T, ctx.num_seqs, ctx.max_query_len, heads_, dk_, dv_);
        float* chunks = in_chunks > 0 ? ctx.take<float>((size_t)in_chunks) : nullptr;
        launch_check(eg_lightning(ctx.stream, (const float*)proj.p, proj.ld, 0, k, 2 * k, 2 * k + v, powers_.as<float>(), norm_w_.as<float>(), (float*)cache.state,
                                  slot_floats(), 0, ctx.seq_starts, ctx.seq_slots, o_raw, chunks, y.p, (int)dtype, y.ld,
                                  plans::delta_column_slices(ctx.num_seqs, heads_, dv_), T, ctx.num_seqs, heads_, dk_, dv_, eps_), "lightning");
        const Rows o = out_(ctx, y, /*out_f32=*/true);
        Delta d;
        d.p = o.p;
        d.dtype = o.dtype;
        return d;
    }

private:
    int hidden_, heads_, dk_, dv_;
    float eps_;
    std::vector<double> decays_;
    Linear in_, out_;
    DeviceBuffer norm_w_, powers_;
};

// ---- the generalised delta rule ---------------------------------------------------------------------------------------------------
// With h the input and H heads of `dim` values:  (r | k | v | g | a' | w') = W h as ONE product, float32 out;
// w = exp(-decay_scale sigmoid(W_2 tanh(w') + w0)),  a = sigmoid(a' + a.b)  per head and key channel;  u = k / sqrt(|k|^2 + unit_eps)
// per head;  S <- diag(w) S - (a u)(u^T S) + k v^T, both terms reading the old S;  o = S^T r  (S [dim, dim] per head, float32, in the
// request's slot as [H, column, row]);  out = W_o (o / rms(o) * .norm * sigmoid(g)), rms per head with eps, the gain over all heads.
// The inner size of the decays' map is what the file's tensors have (parameter rank: what random-weights mode writes).
// Parameters: hidden_size, heads, dim, eps, unit_eps, decay_scale, rank.  Tensors: .r .k .v .g .a [H dim, hidden], .a.b .w0 .norm
// [H dim], .w1 [rank, hidden], .w2 [H dim, rank], .o [hidden, H dim].
class GeneralDeltaMixer : public Mixer {
public:
    GeneralDeltaMixer(const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> position)
        : Mixer(p, prefix, std::move(position)), hidden_((int)p.integer("hidden_size")), heads_((int)p.integer("heads")), dim_((int)p.integer("dim")),
          eps_((float)p.real("eps")), unit_eps_((float)p.real("unit_eps", 1e-6)), decay_scale_((float)p.real("decay_scale")), request_rank_((int)p.integer("rank", 16)) {
        if (hidden_ <= 0 || heads_ <= 0 || dim_ <= 0 || request_rank_ <= 0) throw std::invalid_argument("general delta: sizes must be positive");
        if (dim_ > 256) throw std::invalid_argument("general delta: dim up to 256 is what the kernel takes");
    }
    std::vector<TensorRequest> tensor_requests() const override {
        const long long n = (long long)heads_ * dim_;
        return {TensorRequest::matrix(prefix + ".r", n, hidden_), TensorRequest::matrix(prefix + ".k", n, hidden_), TensorRequest::matrix(prefix + ".v", n, hidden_),
                TensorRequest::matrix(prefix + ".g", n, hidden_), TensorRequest::matrix(prefix + ".a", n, hidden_), TensorRequest::vector(prefix + ".a.b", n),
                TensorRequest::matrix(prefix + ".w1", request_rank_, hidden_).with_free_dim(0), TensorRequest::matrix(prefix + ".w2", n, request_rank_).with_free_dim(1),
                TensorRequest::vector(prefix + ".w0", n), TensorRequest::vector(prefix + ".norm", n).with_init("one"), TensorRequest::matrix(prefix + ".o", hidden_, n)};
    }
    static int padded(int r) { return (r + 15) / 16 * 16; }
    void load(const HostTensors& file, DType dtype) override {
        const StoredTensor &w1 = need_tensor(file, prefix + ".w1"), &w2 = need_tensor(file, prefix + ".w2");
        rank_ = (int)w1.shape[0];
        if (w2.shape[1] != rank_) throw WeightError("the two halves of a low-rank map under '" + prefix + "' differ in their inner size");
        int rows = 0;
        const std::vector<float> w = stacked_rows(file, prefix, {".r", ".k", ".v", ".g", ".a", ".w1"}, hidden_, &rows);
        in_ = Linear(w.data(), rows, hidden_, nullptr, dtype);
        // the second half reads rows padded to a multiple of sixteen values: its weights are padded alike
        const std::vector<float> src = host_floats(w2);
        const size_t n = (size_t)heads_ * dim_, rp = (size_t)padded(rank_);
        std::vector<float> dst(n * rp, 0.f);
        for (size_t i = 0; i < n; ++i) std::memcpy(&dst[i * rp], &src[i * rank_], (size_t)rank_ * 4);
        w2_ = Linear(dst.data(), (int)n, (int)rp, nullptr, dtype);
        w0_ = upload_f32(file, prefix + ".w0");
        a0_ = upload_f32(file, prefix + ".a.b");
        norm_w_ = upload_f32(file, prefix + ".norm");
        out_ = Linear(need_tensor(file, prefix + ".o"), nullptr, dtype);
    }
    size_t weight_bytes() const override { return in_.weight_bytes() + w2_.weight_bytes() + out_.weight_bytes(); }
    size_t arena_bytes(long long T) const override {
        return (size_t)T * ((size_t)in_.out_features * 4 + (size_t)padded(rank_) * 4 + (size_t)heads_ * (dim_ * (4 + 4 + 4) + eg_general_delta_record(dim_) * 4) + (size_t)hidden_ * 4) + (1u << 16);
    }
    bool capturable() const override { return true; }
    long long slot_floats() const { return (long long)heads_ * dim_ * dim_; }
    CacheNeed cache_need() const override { return CacheNeed::state({slot_floats()}); }

    Delta forward(const StepContext& ctx, PartInput in, const CacheView& cache, const FollowingNorm*) override {
        const int T = ctx.num_tokens, n = heads_ * dim_;
        const DType dtype = ctx.dtype;
        if (!cache.state || cache.state_bytes_per_slot != (size_t)slot_floats() * 4) throw DeviceError("a general delta mixer was handed no state of its shape");
        if (!cache.writes) throw DeviceError("a general delta mixer cannot read another entry's state without advancing it");
        const Rows h = in.pending ? in.pending->materialize() : in.rows;
        const Rows proj = in_(ctx, h, /*out_f32=*/true);                      // [T, r | k | v | g | a' | w'] float32
        // the decays' logits: a product of its own, or, in steps whose entries are a few tokens each, worked out by the recurrence's blocks
        Rows x;
        float* records = nullptr;
        if (!eg_general_delta_inline_takes(ctx.max_query_len, rank_)) {
            Rows inner{ctx.take_rows(T, w2_.in_features, dtype), dtype, T, w2_.in_features, w2_.in_features};
            launch_check(eg_tanh_columns(ctx.stream, (const float*)proj.p + 5 * (size_t)n, proj.ld, inner.p, (int)dtype, inner.ld, T, rank_, w2_.in_features), "tanh_columns");
            x = w2_(ctx, inner, /*out_f32=*/true);
            records = ctx.take<float>((size_t)T * heads_ * eg_general_delta_record(dim_));
        }
        Rows y{ctx.take_rows(T, n, dtype), dtype, T, n, n};
        float* o_raw = ctx.take<float>((size_t)T * n);
        launch_check(eg_general_delta(ctx.stream, (const float*)proj.p, proj.ld, 0, n, 2 * n, 3 * n, 4 * n, 5 * n, (const float*)x.p, x.ld, w2_.weight,
                                      w2_.in_features, rank_, w0_.as<float>(), a0_.as<float>(), norm_w_.as<float>(), records, (float*)cache.state, slot_floats(), 0,
                                      ctx.seq_starts, ctx.seq_slots, y.p, (int)dtype, y.ld, o_raw, plans::general_delta_slices(ctx.num_seqs, heads_, dim_), T,
                                      ctx.num_seqs, heads_, dim_, unit_eps_, eps_, decay_scale_, ctx.status), "general_delta");
        const Rows o = out_(ctx, y, /*out_f32=*/true);
        Delta d;
        d.p = o.p;
        d.dtype = o.dtype;
        return d;
    }

private:
    int hidden_, heads_, dim_;
    float eps_, unit_eps_, decay_scale_;
    int request_rank_, rank_ = 0;
    Linear in_, w2_, out_;
    DeviceBuffer w0_, a0_, norm_w_;
};

inline void register_sigmoid_parts() {
    PartRegistry& r = PartRegistry::instance();
    if (r.mixers.count("sigmoid_attention")) return;
    r.positions["waves"] = [](const Params& p, const std::string& prefix) { return std::make_shared<WavePositions>(p, prefix); };
    r.mixers["sigmoid_attention"] = [](const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> pos) {
        return std::make_shared<SigmoidAttention>(p, prefix, std::move(pos));
    };
    r.mixers["lightning"] = [](const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> pos) {
        return std::make_shared<LightningMixer>(p, prefix, std::move(pos));
    };
    r.mixers["general_delta"] = [](const Params& p, const std::string& prefix, std::shared_ptr<PositionEncoding> pos) {
        return std::make_shared<GeneralDeltaMixer>(p, prefix, std::move(pos));
    };
}

}  // namespace easygpt::engine
