// See parts.hpp.  Built-in kinds: rmsnorm, rope, gqa_attention, swiglu, prenorm, sandwich, postnorm, embedding, lm_head (the
// retention mixer lives in parts_recurrent.cpp, the plain and the expert feed-forwards in parts_experts.cpp); and
// the adapter that runs a part registered from outside through fastgguf_parts.h.
#include "parts.hpp"

#include <cmath>
#include <cstring>
#include <mutex>

namespace fg {

static const int EPI_BF16 = 0, EPI_F32 = 1, EPI_ADD_F32 = 2, EPI_SILU_MUL = 3, EPI_GELU_MUL = 5, EPI_RELU_MUL = 6;
static const int KERNEL_BAD_SIZE = 10002;

const char *role_name(int role) {
    static const char *n[] = {"norm", "position", "mixer", "feed_forward", "block", "embedding", "head", "stream_map", "token_input"};
    return role >= 0 && role <= 8 ? n[role] : "?";
}

// ------------------------------------------------------------------------------------ parameters
static const Json &need(const Json &params, const char *key, const char *part) {
    const Json *v = params.find(key);
    if (!v || v->is_null()) fail(FG_E_CONFIG, format("%s: parameter '%s' is missing", part, key));
    return *v;
}
long long param_int(const Json &params, const char *key, const char *part) {
    const Json &v = need(params, key, part);
    if (!v.is_int() && !(v.is_number() && v.as_double() == std::floor(v.as_double())))
        fail(FG_E_CONFIG, format("%s: parameter '%s' must be an integer, got %s", part, key, v.dump().c_str()));
    return v.is_int() ? v.as_int() : (long long)v.as_double();
}
long long param_int(const Json &params, const char *key, long long dflt, const char *part) {
    const Json *v = params.find(key);
    return (!v || v->is_null()) ? dflt : param_int(params, key, part);
}
double param_float(const Json &params, const char *key, const char *part) {
    const Json &v = need(params, key, part);
    if (!v.is_number() || v.is_bool()) fail(FG_E_CONFIG, format("%s: parameter '%s' must be a number, got %s", part, key, v.dump().c_str()));
    return v.as_double();
}
double param_float(const Json &params, const char *key, double dflt, const char *part) {
    const Json *v = params.find(key);
    return (!v || v->is_null()) ? dflt : param_float(params, key, part);
}

// ------------------------------------------------------------------------------------ views
fg_batch_view Batch::view(cudaStream_t s) const {
    fg_batch_view v = {};
    v.n_seq = n_seq; v.n_rows = n_rows; v.n_want = n_want; v.max_new = max_new; v.max_len = max_len;
    v.single_token = single_token; v.want_all = want_all;
    v.tokens = tokens; v.positions = positions; v.row_seq = row_seq; v.cu_rows = cu_rows;
    v.seq_start = seq_start; v.slots = slots; v.want_rows = want_rows;
    v.n_groups = (int)block_tables.size();
    v.block_tables = block_tables.empty() ? nullptr : block_tables.data();
    v.table_width = table_width;
    v.host_cu_rows = host_cu_rows.empty() ? nullptr : host_cu_rows.data();
    v.host_seq_start = host_seq_start.empty() ? nullptr : host_seq_start.data();
    v.host_slots = host_slots.empty() ? nullptr : host_slots.data();
    v.stream = s;
    return v;
}

fg_layer_io LayerIO::view() const {
    fg_layer_io v = {};
    v.group = group; v.k_pool = k_pool; v.v_pool = v_pool; v.n_pages = n_pages; v.page_size = page_size;
    v.n_kv_heads = n_kv_heads; v.head_dim = head_dim; v.cache_dtype = cache_dtype; v.write_cache = write_cache;
    v.state = state; v.state_bytes = state_bytes; v.n_slots = n_slots;
    v.v_head_dim = v_head_dim > 0 ? v_head_dim : head_dim;
    return v;
}

// ------------------------------------------------------------------------------------ weights
Weight make_weight(int64_t rows, int64_t cols, int dtype, const char *what) {
    Weight w;
    w.buffer = std::make_shared<DeviceBuffer>((size_t)rows * (size_t)cols * elem_size(dtype), what);
    w.t.data = w.buffer->get();
    w.t.dtype = dtype;
    w.t.rows = rows;
    w.t.cols = cols;
    w.t.ld = cols;
    return w;
}

Weight concat_rows(const std::vector<Weight> &parts, int dtype, cudaStream_t s) {
    int64_t rows = 0, cols = parts.at(0).t.cols;
    for (auto &p : parts) {
        if (p.t.cols != cols || p.t.ld != p.t.cols) fail(FG_E_INTERNAL, "concat_rows: parts must be contiguous and equally wide");
        rows += p.t.rows;
    }
    Weight out = make_weight(rows, cols, dtype, "a fused weight matrix");
    int64_t at = 0;
    for (auto &p : parts) {
        dev_convert(p.t.data, p.t.dtype, (char *)out.t.data + at * cols * elem_size(dtype), dtype, p.t.numel(), s);
        at += p.t.rows;
    }
    return out;
}

Weight gather_rows(const Weight &w, const std::vector<int64_t> &rows, cudaStream_t s) {
    if (w.t.ld != w.t.cols) fail(FG_E_INTERNAL, "gather_rows: the matrix must be contiguous");
    Weight out = make_weight((int64_t)rows.size(), w.t.cols, w.t.dtype, "a permuted weight matrix");
    dev_gather_rows(w.t.data, out.t.data, rows, w.t.cols, w.t.dtype, s);
    return out;
}

const Weight &tensor_of(const std::map<std::string, Weight> &tensors, const char *name) {
    auto it = tensors.find(name);
    if (it == tensors.end()) fail(FG_E_INTERNAL, format("a part was not given its tensor '%s'", name));
    return it->second;
}

// ------------------------------------------------------------------------------------ deferred norm
Tensor DeferredNorm::materialize(Runtime &rt) const {
    Tensor out = rt.arena->matrix(x.rows, x.cols, FG_BF16);
    FG_LAUNCH("core", fg_rmsnorm, x.ptr<float>(), weight, nullptr, out.data, FG_BF16, (int)x.rows, (int)x.cols, eps, rt.stream);
    return out;
}

// ------------------------------------------------------------------------------------ Linear
Linear::Linear(Weight w) : w_(std::move(w)) {
    const Tensor &t = w_.t;
    fast_ = t.dtype == FG_BF16 && t.cols % 8 == 0 && t.ld % 8 == 0 && ((uintptr_t)t.data % 16) == 0;
}

Linear Linear::rows(int64_t begin, int64_t end) const {
    Weight w = w_;
    w.t = w_.t.row_range(begin, end);
    return Linear(w);
}

Tensor Linear::forward(Runtime &rt, const Tensor &a_in, const DeferredNorm *deferred, Tensor out, int out_dtype, bool accumulate,
                       Norm *emit_norm, DeferredNorm *emitted) const {
    if (emitted) *emitted = DeferredNorm();
    const Tensor &W = w_.t;
    Tensor a = deferred ? deferred->xw : a_in;
    const int64_t M = a.rows, K = a.cols, N = W.rows;
    if (K != W.cols) fail(FG_E_INTERNAL, format("contraction: the input is [%lld, %lld] but the weight is [%lld, %lld]", (long long)M, (long long)K, (long long)N, (long long)W.cols));
    if (accumulate && (!out.defined() || out.dtype != FG_F32))
        fail(FG_E_INTERNAL, "contraction: the residual sum is 32-bit; accumulate needs a float32 output");
    if (!out.defined()) out = rt.arena->matrix(M, N, out_dtype);
    if (out.rows != M || out.cols != N) fail(FG_E_INTERNAL, "contraction: the output has the wrong shape");
    if (M == 0) return out;
    if (fast_ && !rt.plain_kernels && a.dtype == FG_BF16 && (out.dtype == FG_BF16 || out.dtype == FG_F32)) {
        int epi = accumulate ? EPI_ADD_F32 : out.dtype == FG_BF16 ? EPI_BF16 : EPI_F32;
        const float *ss_in = nullptr;
        int ss_tiles = 0, ss_size = 1;
        float ss_eps = 0.f;
        if (deferred) { ss_in = deferred->ss; ss_tiles = deferred->tiles; ss_size = deferred->size; ss_eps = deferred->eps; }
        Tensor xw_out;
        float *ss_out = nullptr;
        const float *norm_w = nullptr;
        bool emit = emit_norm && emitted && accumulate && emit_norm->deferrable() && emit_norm->size() == N;
        if (emit) {
            norm_w = emit_norm->weight();
            xw_out = rt.arena->matrix(M, N, FG_BF16);
            int max_tiles = FG_KERNEL("tc", fg_gemm_tc_max_ss_tiles)((int)N);
            ss_out = (float *)rt.arena->alloc((size_t)max_tiles * (size_t)M * sizeof(float));
        }
        int tiles_out = 0;
        count_launch();
        ProfileScope scope("fg_gemm_tc", profile_on() ? format("%lld x %lld, %lld rows%s", (long long)N, (long long)K, (long long)M, accumulate ? ", residual add" : "").c_str() : nullptr);
        // scratch memory for a split along K (a prompt of a few hundred rows through a projection of few output tiles)
        const long long ws_bytes = FG_KERNEL("tc", fg_gemm_tc_workspace_bytes)((int)M, (int)N, (int)K, epi);
        void *ws = ws_bytes > 0 ? rt.arena->alloc((size_t)ws_bytes) : nullptr;
        int code = FG_KERNEL("tc", fg_gemm_tc_ws)(a.data, (int)a.ld, W.data, (int)W.ld, out.data, (int)out.ld, epi, (int)M, (int)N,
                                                  (int)K, 0, ss_in, ss_tiles, ss_size, ss_eps, norm_w, xw_out.data, ss_out,
                                                  &tiles_out, ws, ws_bytes, rt.stream);
        if (code != KERNEL_BAD_SIZE) {
            check_kernel(code, "fg_gemm_tc");
            if (emit) {
                emitted->xw = xw_out; emitted->ss = ss_out; emitted->tiles = tiles_out; emitted->size = (int)N;
                emitted->eps = emit_norm->eps(); emitted->x = out; emitted->weight = norm_w;
            }
            return out;
        }
    }
    if (deferred) a = deferred->materialize(rt);
    FG_LAUNCH("core", fg_gemm_generic, a.data, a.dtype, (int)a.ld, W.data, W.dtype, (int)W.ld, out.data, out.dtype, (int)out.ld,
              accumulate ? 1 : 0, (int)M, (int)N, (int)K, rt.stream);
    return out;
}

Tensor Linear::forward_relu2(Runtime &rt, const Tensor &a) const {
    const Tensor &W = w_.t;
    const int64_t M = a.rows, K = a.cols, N = W.rows;
    if (K != W.cols) fail(FG_E_INTERNAL, "contraction: the input does not fit the weight");
    if (fast_ && !rt.plain_kernels && a.dtype == FG_BF16 && rt.dtype == FG_BF16) {
        Tensor out = rt.arena->matrix(M, N, FG_BF16);
        if (M == 0) return out;
        const int EPI_RELU2_BF16 = 4;
        int tiles_out = 0;
        count_launch();
        ProfileScope scope("fg_gemm_tc", profile_on() ? format("%lld x %lld, %lld rows, relu2", (long long)N, (long long)K, (long long)M).c_str() : nullptr);
        const long long ws_bytes = FG_KERNEL("tc", fg_gemm_tc_workspace_bytes)((int)M, (int)N, (int)K, EPI_RELU2_BF16);
        void *ws = ws_bytes > 0 ? rt.arena->alloc((size_t)ws_bytes) : nullptr;
        int code = FG_KERNEL("tc", fg_gemm_tc_ws)(a.data, (int)a.ld, W.data, (int)W.ld, out.data, (int)out.ld, EPI_RELU2_BF16, (int)M, (int)N,
                                                  (int)K, 0, nullptr, 0, 1, 0.f, nullptr, nullptr, nullptr, &tiles_out, ws, ws_bytes,
                                                  rt.stream);
        if (code != KERNEL_BAD_SIZE) {
            check_kernel(code, "fg_gemm_tc (relu2)");
            return out;
        }
    }
    Tensor t = forward(rt, a, nullptr, Tensor(), rt.dtype, false, nullptr, nullptr);
    if (t.rows > 0) FG_LAUNCH("core", fg_activation, t.data, t.dtype, (long long)t.rows * t.ld, 0, rt.stream);
    return t;
}

bool Linear::forward_gelu_gather(Runtime &rt, const Tensor &a, const Tensor &table, const int *tokens, int64_t col, Tensor *out) const {
    const Tensor &W = w_.t;
    if (!fast_ || rt.plain_kernels || a.dtype != FG_BF16 || table.dtype != FG_BF16) return false;
    const int64_t M = a.rows, K = a.cols, N = W.rows;
    Tensor t = rt.arena->matrix(M, N, FG_BF16);
    if (M == 0) { *out = t; return true; }
    count_launch();
    ProfileScope scope("fg_gemm_tc", profile_on() ? format("%lld x %lld, %lld rows, gelu x table", (long long)N, (long long)K, (long long)M).c_str() : nullptr);
    const long long ws_bytes = FG_KERNEL("tc", fg_gemm_tc_workspace_bytes)((int)M, (int)N, (int)K, EPI_BF16);
    void *ws = ws_bytes > 0 ? rt.arena->alloc((size_t)ws_bytes) : nullptr;
    int code = FG_KERNEL("tc", fg_gemm_tc_gelu_gather)(a.data, (int)a.ld, W.data, (int)W.ld, t.data, (int)t.ld, (int)M, (int)N, (int)K, table.data,
                                                       (int)table.ld, (int)col, tokens, ws, ws_bytes, rt.stream);
    if (code == KERNEL_BAD_SIZE) return false;
    check_kernel(code, "fg_gemm_tc (gelu x table)");
    *out = t;
    return true;
}

bool Linear::forward_gated(Runtime &rt, const Tensor &a_in, const DeferredNorm *deferred, int act, Tensor *out) const {
    static const int epi_of[3] = {EPI_SILU_MUL, EPI_GELU_MUL, EPI_RELU_MUL};
    static const char *name_of[3] = {"silu", "gelu", "relu"};
    const Tensor &W = w_.t;
    Tensor a = deferred ? deferred->xw : a_in;
    if (!fast_ || rt.plain_kernels || a.dtype != FG_BF16 || W.rows % 128) return false;
    const int64_t M = a.rows, F = W.rows / 2;
    Tensor t = rt.arena->matrix(M, F, FG_BF16);
    if (M == 0) { *out = t; return true; }
    const float *ss_in = nullptr;
    int ss_tiles = 0, ss_size = 1, tiles_out = 0;
    float ss_eps = 0.f;
    if (deferred) { ss_in = deferred->ss; ss_tiles = deferred->tiles; ss_size = deferred->size; ss_eps = deferred->eps; }
    count_launch();
    ProfileScope scope("fg_gemm_tc", profile_on() ? format("%lld x %lld, %lld rows, %s", (long long)W.rows, (long long)a.cols, (long long)M, name_of[act]).c_str() : nullptr);
    int code = FG_KERNEL("tc", fg_gemm_tc)(a.data, (int)a.ld, W.data, (int)W.ld, t.data, (int)t.ld, epi_of[act], (int)M,
                                           (int)W.rows, (int)a.cols, 0, ss_in, ss_tiles, ss_size, ss_eps, nullptr, nullptr,
                                           nullptr, &tiles_out, rt.stream);
    if (code == KERNEL_BAD_SIZE) return false;
    check_kernel(code, "fg_gemm_tc (gated)");
    *out = t;
    return true;
}

// ------------------------------------------------------------------------------------ attention ops
// How many CTAs share one sequence's pages in a decode step: about one and a half CTAs per SM in all, and
// never more than fit on the GPU at once - three per SM at head size 64, one at 128 (each warp holds a K and
// a V page in shared memory).  What does not fit runs as a second wave whose page loads start late; measured
// at batch 8 with 8 KV heads and head size 64, 4 splits (256 CTAs) beat both 2 and 8, and at head size 128
// two splits beat four.  Up to 8 splits (a power of two) are merged inside a thread-block cluster; only
// contexts beyond 16K positions take more splits and the scratch-memory path.
int decode_splits(int n_sm, int n_seq, int n_heads, int n_kv_heads, int table_width, int head_dim) {
    int ctas = n_seq * n_kv_heads * ((n_heads / n_kv_heads + 15) / 16);
    int want = head_dim <= 64 ? (3 * n_sm / 2 + ctas - 1) / ctas : n_sm / ctas;
    want = std::max(1, std::min(want, table_width));
    if (want > 8 && table_width > 256) return want;
    int s = 1;
    while (s < want && s < 8) s *= 2;
    return s;
}

// The tensor-core attention kernels take bfloat16, head size 64 / 128 for keys and values alike and pages of 64; other
// sizes go to the any-size kernel.  Kept first keys: every kernel walks their pages in front of the window's.
static bool fast_attention_ok(const Runtime &rt, const Tensor &q, const LayerIO &io, const AttentionShape &a) {
    return !rt.plain_kernels && q.dtype == FG_BF16 && io.cache_dtype == FG_BF16 && (a.head_dim == 64 || a.head_dim == 128) &&
           a.v_head_dim == a.head_dim && io.page_size == 64 && q.ld % 2 == 0 && ((uintptr_t)q.data % 4) == 0;
}

static Tensor attention(Runtime &rt, const Tensor &q, const Batch &b, const LayerIO &io, const AttentionShape &a) {
    const int H = a.n_heads, KV = a.n_kv_heads, hd = a.head_dim;
    const int *table = b.block_tables.at((size_t)io.group);
    Tensor out = rt.arena->matrix(q.rows, (int64_t)H * a.v_head_dim, q.dtype);
    if (fast_attention_ok(rt, q, io, a)) {
        if (b.single_token) {
            int n_splits = decode_splits(rt.n_sm, b.n_seq, H, KV, b.table_width, hd);
            float *part_o = nullptr, *part_ml = nullptr;
            if (n_splits != 1 && n_splits != 2 && n_splits != 4 && n_splits != 8) {      // very long contexts
                part_o = (float *)rt.arena->alloc((size_t)b.n_seq * H * n_splits * hd * sizeof(float));
                part_ml = (float *)rt.arena->alloc((size_t)b.n_seq * H * n_splits * 2 * sizeof(float));
            }
            FG_LAUNCH("attn", fg_attention_decode_kept, q.data, (int)q.ld, out.data, (int)out.ld, b.positions, table, b.table_width,
                      io.k_pool, io.v_pool, b.n_seq, H, KV, hd, io.page_size, a.scale, a.window, a.keep_first, n_splits, part_o, part_ml,
                      rt.stream);
            return out;
        }
        // Many new tokens: 128-row tiles on the tcgen05 tensor cores.  A few rows (a sequence fed in short
        // pieces) waste less of the mma.sync kernel's 64-row tile.
        bool tc = b.max_new * (H / KV) >= 64 && q.ld % 8 == 0 && ((uintptr_t)q.data % 16) == 0;
        if (tc)
            FG_LAUNCH("attn", fg_attention_prefill_tc_kept, q.data, (int)q.ld, out.data, (int)out.ld, b.cu_rows, b.seq_start, table,
                      b.table_width, io.k_pool, io.v_pool, io.n_pages, b.n_seq, b.max_new, H, KV, hd, io.page_size, a.scale, a.window,
                      a.keep_first, rt.stream);
        else
            FG_LAUNCH("attn", fg_attention_prefill_kept, q.data, (int)q.ld, out.data, (int)out.ld, b.cu_rows, b.seq_start, table,
                      b.table_width, io.k_pool, io.v_pool, b.n_seq, b.max_new, H, KV, hd, io.page_size, a.scale, a.window, a.keep_first,
                      rt.stream);
        return out;
    }
    if (q.dtype != io.cache_dtype) fail(FG_E_INTERNAL, "attention: q and the cache must share a dtype");
    if (hd > 256 || a.v_head_dim > 256)
        fail(FG_E_KERNEL, format("attention: head size %d / %d exceeds 256, the largest the any-size kernel takes", hd, a.v_head_dim));
    FG_LAUNCH("core", fg_attention_generic_kept, q.data, (int)q.ld, out.data, (int)out.ld, q.dtype, b.positions, b.row_seq, table,
              b.table_width, io.k_pool, io.v_pool, (int)q.rows, H, KV, hd, a.v_head_dim, io.page_size, a.scale, a.window, a.keep_first,
              rt.stream);
    return out;
}

Tensor rope_attention(Runtime &rt, const Tensor &qkv, const Batch &b, const LayerIO &io, const float *cos_t, const float *sin_t,
                      const AttentionShape &a) {
    const int H = a.n_heads, KV = a.n_kv_heads, hd = a.head_dim;
    if (io.group < 0 || !io.k_pool) fail(FG_E_INTERNAL, "attention: the schedule entry has no cache");
    if (io.head_dim != hd || (io.v_head_dim > 0 ? io.v_head_dim : io.head_dim) != a.v_head_dim || io.n_kv_heads != KV)
        fail(FG_E_INTERNAL, "attention: the entry's cache has other sizes than its mixer");
    const int *table = b.block_tables.at((size_t)io.group);
    // A decode step in bfloat16 with head size 64 / 128 on the entry's own cache runs as ONE kernel.  It reads
    // positions, the page table and its own pages before waiting for the kernel in front of it; see common.cuh
    // for why that is allowed here and only here.
    if (io.write_cache && b.single_token && fast_attention_ok(rt, qkv, io, a) && qkv.ld % 8 == 0 && ((uintptr_t)qkv.data % 16) == 0) {
        int n_splits = decode_splits(rt.n_sm, b.n_seq, H, KV, b.table_width, hd);
        if (n_splits == 1 || n_splits == 2 || n_splits == 4 || n_splits == 8) {
            Tensor out = rt.arena->matrix(qkv.rows, (int64_t)H * hd, FG_BF16);
            FG_LAUNCH("attn", fg_attention_decode_fused_kept, qkv.data, (int)qkv.ld, out.data, (int)out.ld, b.positions, table,
                      b.table_width, io.k_pool, io.v_pool, cos_t, sin_t, b.n_seq, H, KV, hd, io.page_size, a.scale, a.window,
                      a.keep_first, n_splits, rt.stream);
            return out;
        }
    }
    if (!a.rotate) {
        // nothing to rotate: keys and values go to the cache as they are
        if (io.write_cache)
            FG_LAUNCH("core", fg_kv_append, qkv.data, qkv.dtype, (int)qkv.ld, H * hd, b.positions, b.row_seq, table, b.table_width, io.k_pool,
                      io.v_pool, (int)qkv.rows, KV, hd, a.v_head_dim, io.page_size, rt.stream);
    } else {
        if (a.v_head_dim != hd) fail(FG_E_KERNEL, "attention: rotated keys with values of another head size have no kernel");
        FG_LAUNCH("core", fg_rope_append, qkv.data, qkv.dtype, (int)qkv.ld, b.positions, b.row_seq, table, b.table_width,
                  io.write_cache ? io.k_pool : nullptr, io.write_cache ? io.v_pool : nullptr, cos_t, sin_t, (int)qkv.rows, H, KV, hd,
                  io.page_size, io.write_cache ? 1 : 0, rt.stream);
    }
    return attention(rt, qkv, b, io, a);
}

// ------------------------------------------------------------------------------------ RMSNorm
// y = x * (1 / sqrt(mean(x^2) + eps)) * w; the weight multiplies directly (no +1), in the order x * inv * w
// (rmsnorm_w, fastgguf.c:3100-3105).  Statistics are 32-bit here (the reference sums in double).
// offset: checkpoints that store the weight around zero apply (offset + w); gain: the output times a constant (a final norm in
// front of a head whose logits are scaled).  gain * (offset + w) is formed once, in float32, when the weights are loaded, so
// every kernel (and a norm started inside a contraction) reads a plain weight.
class RMSNorm : public Norm {
public:
    RMSNorm(const Json &p)
        : size_((int)param_int(p, "size", "rmsnorm")), eps_((float)param_float(p, "eps", "rmsnorm")),
          offset_((float)param_float(p, "offset", 0.0, "rmsnorm")), gain_((float)param_float(p, "gain", 1.0, "rmsnorm")) {
        if (size_ <= 0 || !(eps_ > 0.f)) fail(FG_E_CONFIG, "rmsnorm: size and eps must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override { return {{"weight", {size_}, false, offset_ != 0.f ? 0 : 1, offset_ != 0.f ? 0.1f : 0.01f}}; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        const Weight &w = tensor_of(tensors, "weight");
        // widening bf16 -> f32 is exact; the kernels read the weight as f32
        if (w.t.dtype == FG_F32 && offset_ == 0.f && gain_ == 1.f) w_ = w;
        else w_ = concat_rows({w}, FG_F32, rt.stream);
        if (offset_ != 0.f) dev_shift_f32(w_.t.ptr<float>(), w_.t.numel(), offset_, rt.stream);
        if (gain_ != 1.f) dev_scale_f32(w_.t.ptr<float>(), w_.t.numel(), gain_, rt.stream);
    }
    Tensor forward(Runtime &rt, const Tensor &x, const int *rows, int n_rows) override {
        int R = rows ? n_rows : (int)x.rows;
        Tensor out = rt.arena->matrix(R, x.cols, rt.dtype);
        if (R > 0)
            FG_LAUNCH("core", fg_rmsnorm, x.ptr<float>(), w_.t.ptr<float>(), rows, out.data, rt.dtype, R, (int)x.cols, eps_, rt.stream);
        return out;
    }
    bool deferrable() const override { return true; }
    const float *weight() const override { return w_.t.ptr<float>(); }
    float eps() const override { return eps_; }
    int size() const override { return size_; }

private:
    int size_;
    float eps_, offset_, gain_;
    Weight w_;
};

// ------------------------------------------------------------------------------------ rotary encoding
// apply_rope (fastgguf.c:3123-3145): for pair j of a head, angle = pos / theta^(2j / n_rot), divided by
// freq_factors[j] when the model file carries such a vector (:3131), computed in double and rounded to float
// (:3130-3133); the pair is rotated by (a, b) <- (a cos - b sin, a sin + b cos) (:3140-3141).  Pair members
// are (j, j + n_rot/2) ("halves", the row order of model folders; the neox branch of :3138-3139) or adjacent
// (2j, 2j + 1) (the reference's own Llama layout).  The kernels rotate pairs (j, j + head_dim/2) of a head, so
// any other pairing, and a rotary dimension smaller than the head, is brought to that form by permuting the
// rows of the q and k projections once at load (scores do not change under a common permutation of q and k)
// and by identity entries (cos 1, sin 0) for the dimensions that are not rotated.
//
// The llama3 divisors are what GGUF files store as rope_freqs.weight (fastgguf.c:4278); the reference has no
// code that computes them.  With base frequency f_j = theta^(-2j/n_rot) and wavelength l_j = 2 pi / f_j:
//     l_j < orig / high_freq_factor   -> divisor 1                   (high frequencies: untouched)
//     l_j > orig / low_freq_factor    -> divisor factor              (low frequencies: slowed)
//     else  s = (orig / l_j - low) / (high - low);  divisor = 1 / ((1 - s) / factor + s)
std::vector<double> rotary_divisors(int rotary_dim, double theta, const Json &scaling) {
    int half = rotary_dim / 2;
    std::vector<double> div((size_t)half, 1.0);
    if (!scaling.is_object()) return div;
    const Json &kind = scaling.get("rope_type");
    if (kind.is_null() || (kind.is_string() && kind.as_string() == "default")) return div;
    if (kind.is_string() && kind.as_string() == "linear") {
        // every frequency divided by one factor
        double factor = param_float(scaling, "factor", "rope scaling");
        if (!(factor > 0)) fail(FG_E_CONFIG, "rope scaling linear: factor must be positive");
        div.assign((size_t)half, factor);
        return div;
    }
    if (kind.is_string() && kind.as_string() == "yarn") {
        // Frequencies between two wavelengths are blended from "as trained" to "slowed by factor".  With
        // dim(t) = n_rot ln(orig / (2 pi t)) / (2 ln theta) - the (fractional) rotary dimension whose wave turns t times over
        // the original length - lo = max(floor(dim(beta_fast)), 0), hi = min(ceil(dim(beta_slow)), n_rot - 1) and
        // ramp_j = clamp((j - lo) / max(hi - lo, 0.001), 0, 1), pair j's frequency is f_j / factor * ramp_j + f_j (1 - ramp_j).
        double factor = param_float(scaling, "factor", "rope scaling"), orig = param_float(scaling, "original_max_position_embeddings", "rope scaling");
        double fast = param_float(scaling, "beta_fast", "rope scaling"), slow = param_float(scaling, "beta_slow", "rope scaling");
        if (!(factor > 0) || !(orig > 0) || !(fast > 0) || !(slow > 0) || !(theta > 1)) fail(FG_E_CONFIG, "rope scaling yarn: factor, original length and betas must be positive");
        const double two_pi = 2.0 * 3.14159265358979323846;
        auto dim_of = [&](double turns) { return rotary_dim * std::log(orig / (two_pi * turns)) / (2.0 * std::log(theta)); };
        double lo = std::max(std::floor(dim_of(fast)), 0.0), hi = std::min(std::ceil(dim_of(slow)), (double)rotary_dim - 1.0);
        for (int j = 0; j < half; j++) {
            double ramp = std::min(std::max((j - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
            div[(size_t)j] = 1.0 / (ramp / factor + (1.0 - ramp));
        }
        return div;
    }
    if (!kind.is_string() || kind.as_string() != "llama3")
        fail(FG_E_CONFIG, "rotary scaling " + kind.dump() + " is not known (known: default, linear, llama3, yarn)");
    double factor = param_float(scaling, "factor", "rope scaling"), low = param_float(scaling, "low_freq_factor", "rope scaling");
    double high = param_float(scaling, "high_freq_factor", "rope scaling");
    double orig = param_float(scaling, "original_max_position_embeddings", "rope scaling");
    const double two_pi = 2.0 * 3.14159265358979323846;
    for (int j = 0; j < half; j++) {
        double freq = std::pow(theta, -2.0 * j / rotary_dim);
        double wavelen = two_pi / freq;
        if (wavelen < orig / high) div[(size_t)j] = 1.0;
        else if (wavelen > orig / low) div[(size_t)j] = factor;
        else {
            double smooth = (orig / wavelen - low) / (high - low);
            div[(size_t)j] = 1.0 / ((1.0 - smooth) / factor + smooth);
        }
    }
    return div;
}

// yarn also stretches the rotated vectors: cos and sin are both multiplied by 0.1 ln(factor) + 1
double rotary_amplitude(const Json &scaling) {
    if (!scaling.is_object()) return 1.0;
    const Json &kind = scaling.get("rope_type");
    if (!kind.is_string() || kind.as_string() != "yarn") return 1.0;
    return 0.1 * std::log(param_float(scaling, "factor", "rope scaling")) + 1.0;
}

class RotaryEncoding : public PositionEncoding {
public:
    RotaryEncoding(const Json &p) {
        hd_ = (int)param_int(p, "head_dim", "rope");
        theta_ = param_float(p, "theta", "rope");
        n_rot_ = (int)param_int(p, "rotary_dim", hd_, "rope");
        scaling_ = p.get("scaling");
        std::string layout = p.get("layout").is_string() ? p.get("layout").as_string() : "halves";
        if (hd_ <= 0 || hd_ % 2) fail(FG_E_CONFIG, format("rope: head_dim must be even and positive, got %d", hd_));
        if (n_rot_ <= 0 || n_rot_ % 2 || n_rot_ > hd_)
            fail(FG_E_CONFIG, format("rope: rotary_dim must be even, positive and at most head_dim, got %d", n_rot_));
        if (layout != "halves" && layout != "adjacent")
            fail(FG_E_CONFIG, "rope: layout '" + layout + "' is not known (known: halves, adjacent)");
        if (!(theta_ > 0)) fail(FG_E_CONFIG, "rope: theta must be positive");
        rotary_divisors(n_rot_, theta_, scaling_);           // refuses unknown scaling kinds at build time
        adjacent_ = layout == "adjacent";
        if (adjacent_ || n_rot_ != hd_) {
            // canonical row i < hd/2 pairs with i + hd/2; first the rotated pairs, then the untouched dimensions
            perm_.assign((size_t)hd_, 0);
            int half = hd_ / 2, rh = n_rot_ / 2, rest = (hd_ - n_rot_) / 2;
            for (int j = 0; j < rh; j++) {
                perm_[(size_t)j] = adjacent_ ? 2 * j : j;
                perm_[(size_t)(half + j)] = adjacent_ ? 2 * j + 1 : j + rh;
            }
            for (int t = 0; t < rest; t++) {
                perm_[(size_t)(rh + t)] = n_rot_ + t;
                perm_[(size_t)(half + rh + t)] = n_rot_ + rest + t;
            }
        }
    }
    void prepare(Runtime &rt, int max_positions) override {
        if (cos_.buffer && max_positions_ >= max_positions) return;
        int half = hd_ / 2, rh = n_rot_ / 2;
        std::vector<double> div = rotary_divisors(n_rot_, theta_, scaling_);
        std::vector<double> inv((size_t)rh);
        for (int j = 0; j < rh; j++) inv[(size_t)j] = std::pow(theta_, -2.0 * j / n_rot_) / div[(size_t)j];
        const double amp = rotary_amplitude(scaling_);
        std::vector<float> c((size_t)max_positions * half), s((size_t)max_positions * half);
        for (int pos = 0; pos < max_positions; pos++) {
            for (int j = 0; j < half; j++) {
                double ang = j < rh ? (double)pos * inv[(size_t)j] : 0.0;
                c[(size_t)pos * half + j] = (float)((j < rh ? amp : 1.0) * std::cos(ang));
                s[(size_t)pos * half + j] = (float)((j < rh ? amp : 1.0) * std::sin(ang));
            }
        }
        cos_ = make_weight(max_positions, half, FG_F32, "rotary tables");
        sin_ = make_weight(max_positions, half, FG_F32, "rotary tables");
        FG_CUDA(cudaMemcpyAsync(cos_.t.data, c.data(), c.size() * 4, cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaMemcpyAsync(sin_.t.data, s.data(), s.size() * 4, cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaStreamSynchronize(rt.stream));
        max_positions_ = max_positions;
    }
    const float *cos_table() const override { return cos_.t.ptr<float>(); }
    const float *sin_table() const override { return sin_.t.ptr<float>(); }
    int head_dim() const override { return hd_; }
    const std::vector<int> &permutation() const override { return perm_; }

private:
    int hd_ = 0, n_rot_ = 0, max_positions_ = 0;
    double theta_ = 0;
    bool adjacent_ = false;
    Json scaling_;
    std::vector<int> perm_;
    Weight cos_, sin_;
};

// no position encoding: identity tables (cos 1, sin 0), so that the same kernels append keys and values
class NoPosition : public PositionEncoding {
public:
    explicit NoPosition(int hd) : hd_(hd) {}
    void prepare(Runtime &rt, int max_positions) override {
        if (cos_.buffer && max_positions_ >= max_positions) return;
        int half = hd_ / 2;
        std::vector<float> c((size_t)max_positions * half, 1.0f);
        cos_ = make_weight(max_positions, half, FG_F32, "identity rotation tables");
        sin_ = make_weight(max_positions, half, FG_F32, "identity rotation tables");
        FG_CUDA(cudaMemcpyAsync(cos_.t.data, c.data(), c.size() * 4, cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaMemsetAsync(sin_.t.data, 0, c.size() * 4, rt.stream));
        FG_CUDA(cudaStreamSynchronize(rt.stream));
        max_positions_ = max_positions;
    }
    const float *cos_table() const override { return cos_.t.ptr<float>(); }
    const float *sin_table() const override { return sin_.t.ptr<float>(); }
    int head_dim() const override { return hd_; }
    const std::vector<int> &permutation() const override { return perm_; }

private:
    int hd_, max_positions_ = 0;
    std::vector<int> perm_;
    Weight cos_, sin_;
};

// ------------------------------------------------------------------------------------ attention mixer
// GQAAttention(hidden_size, n_heads, n_kv_heads, head_dim, position, scale, window).  Reference, per token
// (fastgguf.c): q, k, v projections in one fused pass (:4692-4696), rotary encoding of q and k (:4702, :4718),
// K stored after rotation and V raw at the token's position (:4720, :4738-4739), scale = 1/sqrt(head_dim)
// (:4744), each query head h attends with KV head h / (H / KV) (:4781) to positions [start, pos] (:4754-4758),
// softmax and value sum (attn_rows :3273-3326), output projection added onto the un-normalized input
// (:4860-4862).  A run that borrows the cache of an earlier entry computes only q and attends to the owner's
// keys and values (the reference's shared-KV layers, :4745-4751).  window w: a row sees the last w keys (:4754-4758);
// keep_first n: and, besides, the first n keys of its sequence, at their own places (what "attention sinks" models
// keep when their window slides on); v_head_dim: values of another size than the keys.
class GQAAttention : public Mixer {
public:
    GQAAttention(const Json &p, BuildContext &ctx) {
        const char *me = "gqa_attention";
        E_ = (int)param_int(p, "hidden_size", me);
        H_ = (int)param_int(p, "n_heads", me);
        KV_ = (int)param_int(p, "n_kv_heads", me);
        hd_ = (int)param_int(p, "head_dim", me);
        if (E_ <= 0 || H_ <= 0 || KV_ <= 0 || hd_ <= 0) fail(FG_E_CONFIG, "gqa_attention: sizes must be positive");
        if (H_ % KV_) fail(FG_E_CONFIG, format("gqa_attention: %d heads are not a multiple of %d KV heads", H_, KV_));
        if (hd_ % 2) fail(FG_E_CONFIG, format("gqa_attention: head_dim must be even, got %d", hd_));
        scale_ = (float)param_float(p, "scale", 1.0 / std::sqrt((double)hd_), me);
        window_ = (int)param_int(p, "window", 0, me);
        keep_first_ = (int)param_int(p, "keep_first", 0, me);
        hdv_ = (int)param_int(p, "v_head_dim", hd_, me);
        if (window_ < 0 || keep_first_ < 0) fail(FG_E_CONFIG, "gqa_attention: window and keep_first cannot be negative");
        if (hdv_ <= 0) fail(FG_E_CONFIG, "gqa_attention: v_head_dim must be positive");
        const Json &qo = p.get("queries_only");
        queries_only_ = qo.is_bool() && qo.as_bool();
        const Json &pos = p.get("position");
        rotate_ = !pos.is_null();
        if (pos.is_null()) {
            own_position_ = std::make_unique<NoPosition>(hd_);
            position_ = own_position_.get();
        } else {
            if (hdv_ != hd_) fail(FG_E_CONFIG, "gqa_attention: a position encoding needs v_head_dim == head_dim");
            position_ = dynamic_cast<PositionEncoding *>(ctx.nested(FG_ROLE_POSITION, pos));
            if (!position_) fail(FG_E_CONFIG, "gqa_attention: 'position' is not a position encoding");
            if (position_->head_dim() != hd_)
                fail(FG_E_CONFIG, format("gqa_attention: the position encoding is built for head_dim %d, the mixer has %d",
                                         position_->head_dim(), hd_));
        }
    }
    std::vector<TensorDecl> tensor_decls() const override {
        int64_t Q = (int64_t)H_ * hd_, D = (int64_t)KV_ * hd_;
        if (queries_only_) return {{"q_proj.weight", {Q, E_}}, {"o_proj.weight", {E_, (int64_t)H_ * hdv_}}};
        return {{"q_proj.weight", {Q, E_}}, {"k_proj.weight", {D, E_}}, {"v_proj.weight", {(int64_t)KV_ * hdv_, E_}},
                {"o_proj.weight", {E_, (int64_t)H_ * hdv_}}};
    }
    bool cache_request(CacheRequest *out) const override {
        out->n_kv_heads = KV_; out->head_dim = hd_; out->window = window_;
        out->v_head_dim = hdv_; out->keep_first = window_ > 0 ? keep_first_ : 0;
        return true;
    }
    bool supports_deferred_norm() const override { return true; }
    bool can_overwrite() const override { return true; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        if (queries_only_) {
            // a layer that only ever runs on another entry's keys and values: its own rows of q, in the order the
            // owner's keys are stored in
            Weight q = tensor_of(tensors, "q_proj.weight");
            const std::vector<int> &perm = position_->permutation();
            if (!perm.empty()) {
                std::vector<int64_t> rows;
                for (int h = 0; h < H_; h++)
                    for (int i = 0; i < hd_; i++) rows.push_back((int64_t)h * hd_ + perm[(size_t)i]);
                q = gather_rows(q, rows, rt.stream);
            }
            q_only_ = Linear(q);
            return;
        }
        Weight q = tensor_of(tensors, "q_proj.weight"), k = tensor_of(tensors, "k_proj.weight");
        const Weight &v = tensor_of(tensors, "v_proj.weight");
        const std::vector<int> &perm = position_->permutation();
        if (!perm.empty()) {
            auto head_rows = [&](int heads) {
                std::vector<int64_t> rows;
                for (int h = 0; h < heads; h++)
                    for (int i = 0; i < hd_; i++) rows.push_back((int64_t)h * hd_ + perm[(size_t)i]);
                return rows;
            };
            q = gather_rows(q, head_rows(H_), rt.stream);
            k = gather_rows(k, head_rows(KV_), rt.stream);
        }
        int dt = (q.t.dtype == k.t.dtype && k.t.dtype == v.t.dtype) ? q.t.dtype : FG_F32;
        qkv_ = Linear(concat_rows({q, k, v}, dt, rt.stream));
        q_only_ = qkv_.rows(0, (int64_t)H_ * hd_);
    }
    void prepare(Runtime &rt, int max_positions) override { position_->prepare(rt, max_positions); }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &batch, const LayerIO &io,
                         Tensor &residual, Norm *emit_norm) override {
        if (io.write_cache && queries_only_) fail(FG_E_CONFIG, "gqa_attention: a queries-only mixer must read another entry's cache");
        const Linear &proj = io.write_cache ? qkv_ : q_only_;
        Tensor qkv = proj.forward(rt, xn, deferred, Tensor(), rt.dtype, false, nullptr, nullptr);
        AttentionShape shape;
        shape.n_heads = H_; shape.n_kv_heads = KV_; shape.head_dim = hd_; shape.v_head_dim = hdv_; shape.scale = scale_;
        shape.window = window_; shape.keep_first = window_ > 0 ? keep_first_ : 0; shape.rotate = rotate_;
        Tensor attn = rope_attention(rt, qkv, batch, io, position_->cos_table(), position_->sin_table(), shape);
        DeferredNorm started;
        o_.forward(rt, attn, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    int E_, H_, KV_, hd_, hdv_, window_, keep_first_;
    bool rotate_ = true, queries_only_ = false;
    float scale_;
    PositionEncoding *position_ = nullptr;
    std::unique_ptr<PositionEncoding> own_position_;
    Linear qkv_, q_only_, o_;
};

// ------------------------------------------------------------------------------------ SwiGLU
// down( silu(gate x) * (up x) ): gate and up in one fused pass (fastgguf.c:4870-4872), silu(z) = z / (1 + exp(-z))
// (:3118) times up (:4876), down projection added onto the layer's input (:4877-4880).
// activation "gelu_tanh": down(gelu_tanh(gate x) * (up x)) instead; "relu": down(max(gate x, 0) * (up x)).
class SwiGLU : public FeedForward {
public:
    SwiGLU(const Json &p) : E_((int)param_int(p, "hidden_size", "swiglu")), F_((int)param_int(p, "d_ff", "swiglu")) {
        if (E_ <= 0 || F_ <= 0) fail(FG_E_CONFIG, "swiglu: sizes must be positive");
        const Json &a = p.get("activation");
        const std::string act = a.is_string() ? a.as_string() : "silu";
        if (act != "silu" && act != "gelu_tanh" && act != "relu") fail(FG_E_CONFIG, "swiglu: activation '" + act + "' is not known (known: silu, gelu_tanh, relu)");
        act_ = act == "gelu_tanh" ? GATED_GELU : act == "relu" ? GATED_RELU : GATED_SILU;
    }
    std::vector<TensorDecl> tensor_decls() const override {
        return {{"gate_proj.weight", {F_, E_}}, {"up_proj.weight", {F_, E_}}, {"down_proj.weight", {E_, F_}}};
    }
    bool supports_deferred_norm() const override { return true; }
    bool can_overwrite() const override { return true; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        const Weight &g = tensor_of(tensors, "gate_proj.weight"), &u = tensor_of(tensors, "up_proj.weight");
        int dt = g.t.dtype == u.t.dtype ? g.t.dtype : FG_F32;
        Weight both = concat_rows({g, u}, dt, rt.stream);
        if (dt == FG_BF16 && F_ % 64 == 0 && E_ % 8 == 0 && !rt.plain_kernels) {
            // gate, up and their product in one tensor-core kernel: rows interleaved in blocks of 64
            std::vector<int64_t> rows;
            for (int64_t blk = 0; blk < F_ / 64; blk++) {
                for (int64_t i = 0; i < 64; i++) rows.push_back(blk * 64 + i);
                for (int64_t i = 0; i < 64; i++) rows.push_back(F_ + blk * 64 + i);
            }
            fused_ = Linear(gather_rows(both, rows, rt.stream));
        } else {
            gate_up_ = Linear(both);
        }
        down_ = Linear(tensor_of(tensors, "down_proj.weight"));
    }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &, Tensor &residual,
                         Norm *emit_norm) override {
        Tensor t;
        bool done = fused_.defined() && fused_.forward_gated(rt, xn, deferred, act_, &t);
        if (!done) {
            if (fused_.defined()) fail(FG_E_KERNEL, "the fused gate/up kernel refused a shape it was planned for");
            Tensor gu = gate_up_.forward(rt, xn, deferred, Tensor(), rt.dtype, false, nullptr, nullptr);
            t = rt.arena->matrix(gu.rows, F_, gu.dtype);
            if (gu.rows > 0 && act_ == GATED_RELU) FG_LAUNCH("core", fg_relu_mul, gu.data, t.data, gu.dtype, (int)gu.rows, F_, rt.stream);
            else if (gu.rows > 0 && act_ == GATED_GELU) FG_LAUNCH("core", fg_gelu_mul, gu.data, t.data, gu.dtype, (int)gu.rows, F_, rt.stream);
            else if (gu.rows > 0) FG_LAUNCH("core", fg_silu_mul, gu.data, t.data, gu.dtype, (int)gu.rows, F_, rt.stream);
        }
        DeferredNorm started;
        down_.forward(rt, t, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    int E_, F_;
    int act_ = GATED_SILU;
    Linear fused_, gate_up_, down_;
};

std::unique_ptr<FeedForward> make_swiglu(const Json &params) { return std::make_unique<SwiGLU>(params); }

// ------------------------------------------------------------------------------------ pre-norm block
// x += mixer(norm1(x)); x += feed_forward(norm2(x)): the norm stands before attention (fastgguf.c:4686-4687) and
// before the feed-forward (:4865-4866); both residual sums add the projection onto the un-normalized input
// (:4862, :4880).  The residual stream x is float32 and is updated in place by the parts' output projections.
// In bfloat16 a norm may be STARTED by the contraction that writes the residual stream and FINISHED by the one
// that reads the normalised rows; parts that do not take part get plain normalised tensors.
class PreNormBlock : public Block {
public:
    bool takes_finished_norm() const override { return true; }
    void check_layer() const override {
        Block::check_layer();
        if (mixer_post_norm || feed_forward_post_norm) fail(FG_E_CONFIG, "block 'prenorm' has no norms behind its sublayers (see 'sandwich')");
    }
    DeferredNorm forward(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &pending,
                         Norm *next_norm) override {
        bool bf16 = rt.dtype == FG_BF16;
        bool mixer_defers = bf16 && mixer->supports_deferred_norm();
        bool ffn_defers = bf16 && feed_forward && feed_forward->supports_deferred_norm();
        DeferredNorm started;
        const bool finished = pending.defined() && pending.tiles == 0;          // (the norm itself, in the activation dtype)
        auto mixer_in = [&]() -> Tensor { return finished ? pending.xw : mixer_norm->forward(rt, x, nullptr, 0); };
        if (!feed_forward) {
            // a layer of a mixer alone: its output projection may start the next layer's norm
            if (mixer_defers && pending.defined() && !finished) return mixer->forward(rt, Tensor(), &pending, batch, io, x, next_norm);
            if (mixer_defers) return mixer->forward(rt, mixer_in(), nullptr, batch, io, x, next_norm);
            mixer->forward(rt, mixer_in(), nullptr, batch, io, x, nullptr);
            return DeferredNorm();
        }
        if (mixer_defers) {
            Norm *emit = (ffn_defers && feed_forward_norm->deferrable()) ? feed_forward_norm : nullptr;
            if (pending.defined() && !finished) started = mixer->forward(rt, Tensor(), &pending, batch, io, x, emit);
            else started = mixer->forward(rt, mixer_in(), nullptr, batch, io, x, emit);
        } else {
            mixer->forward(rt, mixer_in(), nullptr, batch, io, x, nullptr);
        }
        if (ffn_defers) {
            if (started.defined()) return feed_forward->forward(rt, Tensor(), &started, batch, x, next_norm);
            return feed_forward->forward(rt, feed_forward_norm->forward(rt, x, nullptr, 0), nullptr, batch, x, next_norm);
        }
        feed_forward->forward(rt, feed_forward_norm->forward(rt, x, nullptr, 0), nullptr, batch, x, nullptr);
        return DeferredNorm();
    }
};

void Block::check_layer() const {
    if (!mixer || !mixer_norm) fail(FG_E_CONFIG, "a layer needs a mixer and its norm");
    if ((feed_forward == nullptr) != (feed_forward_norm == nullptr)) fail(FG_E_CONFIG, "a layer has a feed-forward and its norm, or neither");
    if (!feed_forward && feed_forward_post_norm) fail(FG_E_CONFIG, "a layer without a feed-forward cannot have a norm behind it");
}

// ------------------------------------------------------------------------------------ sandwich block
// x += post1(mixer(norm1(x))); x += post2(feed_forward(norm2(x))): each sublayer's output is normalised before it
// joins the residual stream.  The sublayer writes its output into a zeroed float32 buffer of the stream's shape (its
// last projection adds into it as it would into the stream), and ONE kernel then normalises that buffer, adds it to the
// stream and, where the next reader of the stream is a norm of this block or the next, produces that norm's output as
// well - so the stream is read and written once per sublayer.  The residual sum and all statistics are 32-bit.
class SandwichBlock : public Block {
public:
    void check_layer() const override {
        Block::check_layer();
        if (!mixer_post_norm || (feed_forward && !feed_forward_post_norm))
            fail(FG_E_CONFIG, "block 'sandwich' needs mixer_post_norm (and feed_forward_post_norm where there is a feed-forward)");
        for (Norm *n : {mixer_norm, mixer_post_norm, feed_forward_norm, feed_forward_post_norm})
            if (n && !n->deferrable()) fail(FG_E_CONFIG, "block 'sandwich' takes norms of the form x / rms(x) * w");
    }
    bool finished_norms() const override { return true; }
    bool takes_finished_norm() const override { return true; }
    // pending.xw (when defined, with tiles == 0) holds the FINISHED norm of x for this block's mixer, made by the block before
    DeferredNorm forward(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &pending,
                         Norm *next_norm) override {
        const int M = (int)x.rows, E = (int)x.cols;
        Tensor xn = !pending.defined() ? mixer_norm->forward(rt, x, nullptr, 0) : pending.tiles == 0 ? pending.xw : pending.materialize(rt);
        Tensor t = rt.arena->matrix(M, E, FG_F32);
        // a part that can write its output instead of adding it needs no zeroed buffer
        auto open = [&](bool can_overwrite) {
            rt.overwrite = can_overwrite;
            if (!can_overwrite && M > 0) FG_CUDA(cudaMemsetAsync(t.data, 0, (size_t)M * E * sizeof(float), rt.stream));
        };
        // the norm that reads x after a sublayer: produced by the kernel that adds the sublayer's output
        auto join = [&](Norm *post, Norm *reader) -> Tensor {
            Tensor out;
            if (reader) out = rt.arena->matrix(M, E, rt.dtype);
            if (M > 0)
                FG_LAUNCH("core", fg_norm_add_norm, t.ptr<float>(), post->weight(), x.ptr<float>(), reader ? reader->weight() : nullptr,
                          out.data, rt.dtype, M, E, post->eps(), reader ? reader->eps() : 0.f, rt.stream);
            return out;
        };
        auto finished = [&](const Tensor &xn_next, Norm *reader) {
            DeferredNorm d;
            if (reader && xn_next.defined()) { d.xw = xn_next; d.tiles = 0; d.size = E; d.eps = reader->eps(); d.x = x; d.weight = reader->weight(); }
            return d;
        };
        Norm *hand_over = (next_norm && next_norm->deferrable() && next_norm->weight() && E * sizeof(float) <= 48 * 1024) ? next_norm : nullptr;
        bool fuse_inner = E * sizeof(float) <= 48 * 1024;
        open(mixer->can_overwrite());
        mixer->forward(rt, xn, nullptr, batch, io, t, nullptr);
        rt.overwrite = false;
        if (!feed_forward) return finished(join(mixer_post_norm, hand_over), hand_over);
        Tensor hn = join(mixer_post_norm, fuse_inner ? feed_forward_norm : nullptr);
        if (!hn.defined()) hn = feed_forward_norm->forward(rt, x, nullptr, 0);
        open(feed_forward->can_overwrite());
        feed_forward->forward(rt, hn, nullptr, batch, t, nullptr);
        rt.overwrite = false;
        return finished(join(feed_forward_post_norm, hand_over), hand_over);
    }
};

// ------------------------------------------------------------------------------------ post-norm block
// x += post1(mixer(x)); x += post2(feed_forward(x)): no norm in front, the sublayers read the stream itself - in bfloat16 its
// rounding, as every contraction's input is, in float32 the stream.  The norm stands on a sublayer's output only.  ONE kernel
// normalises that output, adds it to the float32 stream and writes the rounded stream for the next reader (or, where the next
// reader of the stream is a norm, that norm's output).
class PostNormBlock : public Block {
public:
    void check_layer() const override {
        if (!mixer || !mixer_post_norm) fail(FG_E_CONFIG, "block 'postnorm' needs a mixer and mixer_post_norm");
        if (mixer_norm || feed_forward_norm) fail(FG_E_CONFIG, "block 'postnorm' has no norms in front of its sublayers");
        if ((feed_forward == nullptr) != (feed_forward_post_norm == nullptr)) fail(FG_E_CONFIG, "a layer has a feed-forward and its norm, or neither");
        for (Norm *n : {mixer_post_norm, feed_forward_post_norm})
            if (n && !n->deferrable()) fail(FG_E_CONFIG, "block 'postnorm' takes norms of the form x / rms(x) * w");
    }
    bool finished_norms() const override { return true; }
    bool reads_stream() const override { return true; }
    DeferredNorm forward(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &pending,
                         Norm *next_norm) override {
        const int M = (int)x.rows, E = (int)x.cols;
        const bool rounds = rt.dtype != FG_F32;
        Tensor xin = x;
        if (rounds && pending.defined() && pending.tiles == 0 && !pending.weight) xin = pending.xw;
        else if (rounds) {
            xin = rt.arena->matrix(M, E, rt.dtype);
            if (M > 0) FG_LAUNCH("core", fg_cast_rows, x.ptr<float>(), (int)x.ld, xin.data, xin.dtype, (int)xin.ld, M, E, rt.stream);
        }
        Tensor t = rt.arena->matrix(M, E, FG_F32);
        auto run = [&](bool can_overwrite, auto &&sublayer) {
            rt.overwrite = can_overwrite;
            if (!can_overwrite && M > 0) FG_CUDA(cudaMemsetAsync(t.data, 0, (size_t)M * E * sizeof(float), rt.stream));
            sublayer();
            rt.overwrite = false;
        };
        auto join = [&](Norm *post, Norm *reader) -> Tensor {
            Tensor out;
            if (reader || rounds) out = rt.arena->matrix(M, E, rt.dtype);
            if (M > 0)
                FG_LAUNCH("core", fg_norm_add_norm, t.ptr<float>(), post->weight(), x.ptr<float>(), reader ? reader->weight() : nullptr,
                          out.data, rt.dtype, M, E, post->eps(), reader ? reader->eps() : 0.f, rt.stream);
            return out;
        };
        Norm *reader = (next_norm && next_norm->deferrable() && next_norm->weight() && E * sizeof(float) <= 48 * 1024) ? next_norm : nullptr;
        auto hand_over = [&](const Tensor &out) {
            DeferredNorm d;
            if (next_norm && !reader) return d;              // (the reader makes its norm itself)
            if (out.defined()) { d.xw = out; d.tiles = 0; d.size = E; d.eps = reader ? reader->eps() : 0.f; d.x = x; d.weight = reader ? reader->weight() : nullptr; }
            return d;
        };
        run(mixer->can_overwrite(), [&] { mixer->forward(rt, xin, nullptr, batch, io, t, nullptr); });
        if (!feed_forward) return hand_over(join(mixer_post_norm, reader));
        Tensor hin = join(mixer_post_norm, nullptr);
        if (!rounds) hin = x;
        run(feed_forward->can_overwrite(), [&] { feed_forward->forward(rt, hin, nullptr, batch, t, nullptr); });
        return hand_over(join(feed_forward_post_norm, reader));
    }
};

// ------------------------------------------------------------------------------------ parallel block
// x += mixer(norm1(x)) + feed_forward(norm1(x)): ONE norm, both sublayers read its output, and both add their results to the
// float32 stream (the mixer first).  In bfloat16 the started norm that the block before handed over serves both sublayers,
// and the last sublayer's output projection starts the next block's norm.
// With a feed_forward_norm: x += mixer(norm1(x)) + feed_forward(norm2(x)), two norms of the SAME x with a weight each.  Both
// are formed (one kernel, one statistic a row) before either sublayer adds to the stream.
class ParallelBlock : public Block {
public:
    bool takes_finished_norm() const override { return !feed_forward_norm; }
    void check_layer() const override {
        if (!mixer || !mixer_norm) fail(FG_E_CONFIG, "a layer needs a mixer and its norm");
        if (mixer_post_norm || feed_forward_post_norm) fail(FG_E_CONFIG, "block 'parallel' has its norms in front of the sublayers");
        if (feed_forward_norm && !feed_forward) fail(FG_E_CONFIG, "a layer without a feed-forward cannot have a norm for one");
    }
    DeferredNorm forward(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &pending,
                         Norm *next_norm) override {
        if (feed_forward_norm) return forward_two_norms(rt, x, batch, io, pending, next_norm);
        const bool bf16 = rt.dtype == FG_BF16;
        const bool mixer_defers = bf16 && mixer->supports_deferred_norm();
        const bool ffn_defers = bf16 && feed_forward && feed_forward->supports_deferred_norm();
        const bool started = pending.defined() && pending.tiles > 0;
        Tensor xn;                                   // the finished norm, made once if anybody needs it
        auto finished = [&]() -> const Tensor & {
            if (!xn.defined()) xn = !pending.defined() ? mixer_norm->forward(rt, x, nullptr, 0) : pending.tiles == 0 ? pending.xw : pending.materialize(rt);
            return xn;
        };
        // both sublayers must have read the stream's norm before either adds to the stream: a finished norm is a copy, and a
        // started one (xw and the row sums) is a copy as well, so the order of the two additions is free
        DeferredNorm out;
        Norm *mixer_emits = feed_forward ? nullptr : next_norm;
        if (mixer_defers && started) out = mixer->forward(rt, Tensor(), &pending, batch, io, x, mixer_emits);
        else out = mixer->forward(rt, finished(), nullptr, batch, io, x, mixer_defers ? mixer_emits : nullptr);
        if (!feed_forward) return mixer_defers ? out : DeferredNorm();
        if (ffn_defers && started) return feed_forward->forward(rt, Tensor(), &pending, batch, x, next_norm);
        out = feed_forward->forward(rt, finished(), nullptr, batch, x, ffn_defers ? next_norm : nullptr);
        return ffn_defers ? out : DeferredNorm();
    }

private:
    DeferredNorm forward_two_norms(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &pending,
                                   Norm *next_norm) {
        const int M = (int)x.rows, E = (int)x.cols;
        Tensor xa, xb;
        // a norm the block before finished for this block's mixer is taken; the feed-forward's is made here
        if (pending.defined() && pending.tiles == 0) {
            xa = pending.xw;
            xb = feed_forward_norm->forward(rt, x, nullptr, 0);
        } else if (mixer_norm->deferrable() && feed_forward_norm->deferrable() && mixer_norm->weight() && feed_forward_norm->weight() &&
                   mixer_norm->size() == E && feed_forward_norm->size() == E) {
            xa = rt.arena->matrix(M, E, rt.dtype);
            xb = rt.arena->matrix(M, E, rt.dtype);
            if (M > 0)
                FG_LAUNCH("core", fg_rmsnorm_pair, x.ptr<float>(), mixer_norm->weight(), feed_forward_norm->weight(), xa.data, xb.data, rt.dtype, M, E,
                          mixer_norm->eps(), feed_forward_norm->eps(), rt.stream);
        } else {
            xa = mixer_norm->forward(rt, x, nullptr, 0);
            xb = feed_forward_norm->forward(rt, x, nullptr, 0);
        }
        const bool ffn_defers = rt.dtype == FG_BF16 && feed_forward->supports_deferred_norm();
        mixer->forward(rt, xa, nullptr, batch, io, x, nullptr);
        DeferredNorm out = feed_forward->forward(rt, xb, nullptr, batch, x, ffn_defers ? next_norm : nullptr);
        return ffn_defers ? out : DeferredNorm();
    }
};

// ------------------------------------------------------------------------------------ per-layer token input
// A second embedding table gives every layer a few numbers a token: e = table[token, column .. column + dim).  The layer gates
// them by the stream, projects them to the width and adds the normalised result:
//     g = gelu_tanh(W_gate x) * e,   y = W_proj g,   x <- x + y / sqrt(mean(y^2) + eps) * w
// x is the stream itself (no norm in front).  The residual sum and the norm's statistics are 32-bit; in bfloat16 the stream is
// rounded for the gate contraction as every contraction's input is (by the contraction that writes the stream, where it can), and its
// float32 result meets gelu and e in float32 - in the contraction's epilogue, where that runs on the tensor cores.
class GatedTokenEmbedding : public TokenInput {
public:
    GatedTokenEmbedding(const Json &p) {
        const char *me = "gated_token_embedding";
        E_ = param_int(p, "hidden_size", me);
        V_ = param_int(p, "vocab_size", me);
        D_ = param_int(p, "dim", me);
        col_ = param_int(p, "column", 0, me);
        TD_ = param_int(p, "table_dim", col_ + D_, me);
        eps_ = (float)param_float(p, "eps", me);
        if (E_ <= 0 || V_ <= 0 || D_ <= 0 || col_ < 0 || col_ + D_ > TD_) fail(FG_E_CONFIG, "gated_token_embedding: sizes must be positive and the columns inside the table");
        if (!(eps_ > 0.f)) fail(FG_E_CONFIG, "gated_token_embedding: eps must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override {
        return {{"table", {V_, TD_}, false, 0, 1.0f}, {"gate", {D_, E_}}, {"proj", {E_, D_}}, {"norm", {E_}, false, 1, 0.01f}};
    }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        table_ = tensor_of(tensors, "table");
        gate_ = Linear(tensor_of(tensors, "gate"));
        proj_ = Linear(tensor_of(tensors, "proj"));
        const Weight &w = tensor_of(tensors, "norm");
        norm_w_ = w.t.dtype == FG_F32 ? w : concat_rows({w}, FG_F32, rt.stream);
        stream_.load(E_, rt);
    }
    Norm *stream_norm() override { return &stream_; }
    DeferredNorm forward(Runtime &rt, const Batch &b, Tensor &x, const DeferredNorm &stream, const float *add_row, Norm *reader) override {
        const int M = (int)x.rows;
        DeferredNorm next;
        if (M == 0) return next;
        Tensor xin = x;
        if (rt.dtype == FG_BF16 && stream.defined() && stream.weight == stream_.weight()) {
            xin = stream.xw;                     // the contraction that wrote the stream rounded it as well
        } else if (rt.dtype != FG_F32) {
            xin = rt.arena->matrix(M, E_, rt.dtype);
            FG_LAUNCH("core", fg_cast_rows, x.ptr<float>(), (int)x.ld, xin.data, xin.dtype, (int)xin.ld, M, (int)E_, rt.stream);
        }
        Tensor g;
        if (!gate_.forward_gelu_gather(rt, xin, table_.t, b.tokens, col_, &g)) {
            Tensor z = gate_.forward(rt, xin, nullptr, Tensor(), FG_F32, false, nullptr, nullptr);
            g = rt.arena->matrix(M, D_, rt.dtype);
            FG_LAUNCH("core", fg_gelu_mul_gather, z.ptr<float>(), (int)z.ld, table_.t.data, table_.t.dtype, (int)table_.t.ld, (int)col_, b.tokens, g.data,
                      g.dtype, (int)g.ld, M, (int)D_, rt.stream);
        }
        Tensor y = proj_.forward(rt, g, nullptr, Tensor(), FG_F32, false, nullptr, nullptr);
        if (reader && !(reader->deferrable() && reader->weight() && reader->size() == E_ && E_ * (int64_t)sizeof(float) <= 48 * 1024)) reader = nullptr;
        if (reader) {
            next.xw = rt.arena->matrix(M, E_, rt.dtype);
            next.tiles = 0; next.size = (int)E_; next.eps = reader->eps(); next.x = x; next.weight = reader->weight();
        }
        FG_LAUNCH("core", fg_norm_add_norm_row, y.ptr<float>(), norm_w_.t.ptr<float>(), add_row, x.ptr<float>(), next.weight, next.xw.data, rt.dtype, M, (int)E_,
                  eps_, next.eps, rt.stream);
        return next;
    }

private:
    // x * 1: what a contraction writes as this norm's started form is the stream rounded to bfloat16
    class UnitNorm : public Norm {
    public:
        void load(int64_t E, Runtime &rt) {
            ones_ = make_weight(1, E, FG_F32, "a unit norm weight");
            FG_CUDA(cudaMemsetAsync(ones_.t.data, 0, (size_t)E * sizeof(float), rt.stream));
            dev_shift_f32(ones_.t.ptr<float>(), E, 1.0f, rt.stream);
        }
        Tensor forward(Runtime &, const Tensor &, const int *, int) override { fail(FG_E_INTERNAL, "the stream's rounding is not a norm of its own"); }
        bool deferrable() const override { return true; }
        const float *weight() const override { return ones_.t.ptr<float>(); }
        float eps() const override { return 0.f; }
        int size() const override { return (int)ones_.t.cols; }

    private:
        Weight ones_;
    };
    UnitNorm stream_;
    int64_t E_ = 0, V_ = 0, D_ = 0, col_ = 0, TD_ = 0;
    float eps_ = 0.f;
    Weight table_, norm_w_;
    Linear gate_, proj_;
};

// ------------------------------------------------------------------------------------ stream maps
// out = W [x; x0]: the stream and the embedding's output side by side through one matrix [E, 2 E] (x's columns first).
// The sum is 32-bit; in bfloat16 the two inputs are rounded for the contraction as every contraction's input is.
class ConcatLinear : public StreamMap {
public:
    ConcatLinear(const Json &p) : E_(param_int(p, "hidden_size", "concat_linear")) {
        if (E_ <= 0) fail(FG_E_CONFIG, "concat_linear: hidden_size must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override { return {{"weight", {E_, 2 * E_}}}; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &) override { w_ = Linear(tensor_of(tensors, "weight")); }
    void forward(Runtime &rt, const Tensor &x, const Tensor &x0, Tensor &out) override {
        const int64_t M = x.rows;
        Tensor both = rt.arena->matrix(M, 2 * E_, rt.dtype);
        FG_LAUNCH("core", fg_concat2, x.ptr<float>(), (int)x.ld, x0.ptr<float>(), (int)x0.ld, both.data, both.dtype, (int)both.ld, (int)M, (int)E_, rt.stream);
        w_.forward(rt, both, nullptr, out, FG_F32, false, nullptr, nullptr);
    }

private:
    int64_t E_;
    Linear w_;
};

// x <- x + step[t] in front of pass t of a looped span: one vector a pass, from a table [rows, E].  Nothing runs by itself: the
// kernel that writes the stream in front of the pass adds the vector, or a kernel of the model's step does.
class AddRow : public StreamMap {
public:
    AddRow(const Json &p) : E_(param_int(p, "hidden_size", "add_row")), rows_(param_int(p, "rows", "add_row")) {
        if (E_ <= 0 || rows_ <= 0) fail(FG_E_CONFIG, "add_row: hidden_size and rows must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override { return {{"table", {rows_, E_}}}; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        const Weight &w = tensor_of(tensors, "table");
        table_ = w.t.dtype == FG_F32 ? w : concat_rows({w}, FG_F32, rt.stream);
    }
    void check_pass(int pass) const override {
        if (pass < 0 || pass >= rows_) fail(FG_E_CONFIG, format("add_row: there is no vector for pass %d of %lld", pass, (long long)rows_));
    }
    const float *added_row(int pass) const override { return table_.t.ptr<float>() + (int64_t)pass * E_; }
    void forward(Runtime &, const Tensor &, const Tensor &, Tensor &) override { fail(FG_E_INTERNAL, "add_row is added where the stream is written"); }

private:
    int64_t E_, rows_;
    Weight table_;
};

// ------------------------------------------------------------------------------------ embedding and head
// read_embedding copies row `token` of token_embd into the residual stream, times embd_scale, which is 1 for
// Llama (fastgguf.c:4576-4581, :4652, :4219); the head is output.weight or, when that tensor is absent, the
// embedding table again (:4269-4270); logits are float (:4900).  Here tied-ness comes from the spec (both parts
// name the same checkpoint tensor), and a tied head shares the embedding's storage.
class TokenEmbedding : public Embedding {
public:
    TokenEmbedding(const Json &p)
        : V_(param_int(p, "vocab_size", "embedding")), E_(param_int(p, "hidden_size", "embedding")),
          scale_((float)param_float(p, "scale", 1.0, "embedding")) {
        if (V_ <= 0 || E_ <= 0) fail(FG_E_CONFIG, "embedding: sizes must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override { return {{"weight", {V_, E_}}}; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &) override { w_ = tensor_of(tensors, "weight"); }
    bool takes_row() const override { return true; }
    DeferredNorm forward(Runtime &rt, const Batch &batch, Tensor &x, Norm *emit_norm, const float *add_row) override {
        DeferredNorm started;
        int M = batch.n_rows;
        if (M == 0) return started;
        if (emit_norm && emit_norm->deferrable() && emit_norm->size() == E_ && rt.dtype == FG_BF16 && scale_ == 1.0f) {
            Tensor xw = rt.arena->matrix(M, E_, FG_BF16);
            float *ss = (float *)rt.arena->alloc((size_t)M * sizeof(float));
            FG_LAUNCH("core", fg_embed_gather_norm_row, w_.t.data, w_.t.dtype, batch.tokens, add_row, x.ptr<float>(), emit_norm->weight(), xw.data,
                      ss, M, (int)E_, rt.stream);
            started.xw = xw; started.ss = ss; started.tiles = 1; started.size = (int)E_; started.eps = emit_norm->eps();
            started.x = x; started.weight = emit_norm->weight();
            return started;
        }
        FG_LAUNCH("core", fg_embed_gather_row, w_.t.data, w_.t.dtype, batch.tokens, add_row, x.ptr<float>(), M, (int)E_, scale_, rt.stream);
        return started;
    }

private:
    int64_t V_, E_;
    float scale_;
    Weight w_;
};

// softcap c: logits <- c * tanh(logits / c), on the float32 logits (the reference's final_softcap, fastgguf.c:4064-4100).
class LMHead : public Head {
public:
    LMHead(const Json &p)
        : V_(param_int(p, "vocab_size", "lm_head")), E_(param_int(p, "hidden_size", "lm_head")),
          softcap_((float)param_float(p, "softcap", 0.0, "lm_head")) {
        if (V_ <= 0 || E_ <= 0) fail(FG_E_CONFIG, "lm_head: sizes must be positive");
        if (softcap_ < 0.f) fail(FG_E_CONFIG, "lm_head: softcap must be positive (or absent)");
    }
    std::vector<TensorDecl> tensor_decls() const override { return {{"weight", {V_, E_}}}; }
    void load(const std::map<std::string, Weight> &tensors, Runtime &) override { linear_ = Linear(tensor_of(tensors, "weight")); }
    bool supports_deferred_norm() const override { return true; }
    Tensor forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred) override {
        Tensor logits = linear_.forward(rt, xn, deferred, Tensor(), FG_F32, false, nullptr, nullptr);
        if (softcap_ > 0.f && logits.rows > 0)
            FG_LAUNCH("core", fg_softcap, logits.ptr<float>(), (int)logits.rows, (int)logits.cols, (int)logits.ld, softcap_, rt.stream);
        return logits;
    }

private:
    int64_t V_, E_;
    float softcap_;
    Linear linear_;
};

// ------------------------------------------------------------------------------------ parts from outside
static void *arena_alloc_cb(void *ctx, size_t bytes) {
    try {
        return ((Arena *)ctx)->alloc(bytes);
    } catch (...) {
        return nullptr;
    }
}

struct ExternalCore {
    fg_part_vtable vt;
    std::string kind;
    int role;
    void *self = nullptr;
    ExternalCore(const fg_part_vtable &v, std::string k, int r, const Json &params, int dtype) : vt(v), kind(std::move(k)), role(r) {
        if (!vt.create) fail(FG_E_CONFIG, "part '" + kind + "' has no create function");
        char err[512] = {0};
        self = vt.create(params.dump().c_str(), dtype, vt.user, err, sizeof err);
        if (!self) fail(FG_E_CONFIG, std::string(role_name(role)) + " '" + kind + "': " + (err[0] ? err : "refused its parameters"));
    }
    ~ExternalCore() {
        if (self && vt.destroy) vt.destroy(self);
    }
    std::vector<TensorDecl> decls() const {
        std::vector<TensorDecl> out;
        int n = vt.n_tensors ? vt.n_tensors(self) : 0;
        for (int i = 0; i < n; i++) {
            fg_tensor_decl d = {};
            if (!vt.tensor_decl || vt.tensor_decl(self, i, &d) != 0) fail(FG_E_CONFIG, "part '" + kind + "' could not describe its tensors");
            TensorDecl t;
            d.name[sizeof d.name - 1] = 0;
            t.name = d.name;
            for (int k = 0; k < d.ndim && k < 4; k++) t.shape.push_back(d.shape[k]);
            t.is_int = d.is_int != 0;
            t.init = d.init;
            t.std = d.std;
            out.push_back(t);
        }
        return out;
    }
    void load(const std::map<std::string, Weight> &tensors) {
        auto ds = decls();
        for (size_t i = 0; i < ds.size(); i++) {
            const Weight &w = tensor_of(tensors, ds[i].name.c_str());
            held.push_back(w);                                  // the part may keep the pointer
            fg_dev_tensor v = w.t.view();
            v.ndim = (int)ds[i].shape.size();
            for (size_t k = 0; k < ds[i].shape.size(); k++) v.shape[k] = ds[i].shape[k];
            if (vt.load && vt.load(self, (int)i, &v) != 0) fail(FG_E_WEIGHTS, "part '" + kind + "' refused tensor '" + ds[i].name + "'");
        }
    }
    void call(fg_part_call &c, Runtime &rt) {
        c.role = role;
        c.alloc = arena_alloc_cb;
        c.alloc_ctx = rt.arena;
        c.stream = rt.stream;
        if (!vt.forward) fail(FG_E_CONFIG, "part '" + kind + "' has no forward function");
        count_launch();
        int code = vt.forward(self, &c);
        if (code != 0) fail(code > 0 && code <= FG_E_INTERNAL ? code : FG_E_KERNEL, format("%s '%s' failed with status %d", role_name(role), kind.c_str(), code));
    }
    std::vector<Weight> held;
};

class ExternalNorm : public Norm {
public:
    ExternalNorm(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_NORM, p, dtype) {}
    std::vector<TensorDecl> tensor_decls() const override { return core.decls(); }
    void load(const std::map<std::string, Weight> &t, Runtime &) override { core.load(t); }
    Tensor forward(Runtime &rt, const Tensor &x, const int *rows, int n_rows) override {
        int R = rows ? n_rows : (int)x.rows;
        Tensor out = rt.arena->matrix(R, x.cols, rt.dtype);
        fg_part_call c = {};
        c.x = x.view(); c.out = out.view(); c.rows = rows; c.n_rows = R;
        core.call(c, rt);
        return out;
    }
    ExternalCore core;
};

class ExternalPosition : public PositionEncoding {
public:
    ExternalPosition(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_POSITION, p, dtype) {
        hd_ = (int)param_int(p, "head_dim", k.c_str());
        if (hd_ <= 0 || hd_ % 2) fail(FG_E_CONFIG, "position '" + k + "': head_dim must be even and positive");
        if (!core.vt.position_tables) fail(FG_E_CONFIG, "position '" + k + "' has no position_tables function");
        std::vector<float> c(hd_ / 2), s(hd_ / 2);
        tables(1, c, s);                                        // the permutation is known at build time
    }
    void tables(int max_positions, std::vector<float> &c, std::vector<float> &s) {
        int half = hd_ / 2;
        c.assign((size_t)max_positions * half, 1.f);
        s.assign((size_t)max_positions * half, 0.f);
        std::vector<int> perm((size_t)hd_);
        for (int i = 0; i < hd_; i++) perm[(size_t)i] = i;
        if (core.vt.position_tables(core.self, max_positions, hd_, c.data(), s.data(), perm.data()) != 0)
            fail(FG_E_CONFIG, "position '" + core.kind + "' could not build its tables");
        std::vector<char> seen((size_t)hd_, 0);
        bool identity = true;
        for (int i = 0; i < hd_; i++) {
            int p = perm[(size_t)i];
            if (p < 0 || p >= hd_ || seen[(size_t)p]) fail(FG_E_CONFIG, "position '" + core.kind + "': its row permutation is no permutation");
            seen[(size_t)p] = 1;
            identity = identity && p == i;
        }
        perm_ = identity ? std::vector<int>() : perm;
    }
    void prepare(Runtime &rt, int max_positions) override {
        if (cos_.buffer && max_positions_ >= max_positions) return;
        std::vector<float> c, s;
        tables(max_positions, c, s);
        cos_ = make_weight(max_positions, hd_ / 2, FG_F32, "position tables");
        sin_ = make_weight(max_positions, hd_ / 2, FG_F32, "position tables");
        FG_CUDA(cudaMemcpyAsync(cos_.t.data, c.data(), c.size() * 4, cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaMemcpyAsync(sin_.t.data, s.data(), s.size() * 4, cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaStreamSynchronize(rt.stream));
        max_positions_ = max_positions;
    }
    const float *cos_table() const override { return cos_.t.ptr<float>(); }
    const float *sin_table() const override { return sin_.t.ptr<float>(); }
    int head_dim() const override { return hd_; }
    const std::vector<int> &permutation() const override { return perm_; }
    ExternalCore core;

private:
    int hd_ = 0, max_positions_ = 0;
    std::vector<int> perm_;
    Weight cos_, sin_;
};

class ExternalMixer : public Mixer {
public:
    ExternalMixer(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_MIXER, p, dtype) {}
    std::vector<TensorDecl> tensor_decls() const override { return core.decls(); }
    void load(const std::map<std::string, Weight> &t, Runtime &) override { core.load(t); }
    bool cache_request(CacheRequest *out) const override {
        if (!core.vt.cache_request) return false;
        int kv = 0, hd = 0, w = 0;
        if (!core.vt.cache_request(core.self, &kv, &hd, &w)) return false;
        out->n_kv_heads = kv; out->head_dim = hd; out->window = w;
        return true;
    }
    int64_t state_bytes() const override { return core.vt.state_bytes ? core.vt.state_bytes(core.self) : 0; }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *, const Batch &batch, const LayerIO &io, Tensor &residual,
                         Norm *) override {
        fg_batch_view bv = batch.view(rt.stream);
        fg_layer_io iv = io.view();
        fg_part_call c = {};
        c.batch = &bv; c.io = &iv; c.xn = xn.view(); c.residual = residual.view();
        core.call(c, rt);
        return DeferredNorm();
    }
    ExternalCore core;
};

class ExternalFeedForward : public FeedForward {
public:
    ExternalFeedForward(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_FEED_FORWARD, p, dtype) {}
    std::vector<TensorDecl> tensor_decls() const override { return core.decls(); }
    void load(const std::map<std::string, Weight> &t, Runtime &) override { core.load(t); }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *, const Batch &batch, Tensor &residual, Norm *) override {
        fg_batch_view bv = batch.view(rt.stream);
        fg_part_call c = {};
        c.batch = &bv; c.xn = xn.view(); c.residual = residual.view();
        core.call(c, rt);
        return DeferredNorm();
    }
    ExternalCore core;
};

class ExternalEmbedding : public Embedding {
public:
    ExternalEmbedding(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_EMBEDDING, p, dtype) {}
    std::vector<TensorDecl> tensor_decls() const override { return core.decls(); }
    void load(const std::map<std::string, Weight> &t, Runtime &) override { core.load(t); }
    DeferredNorm forward(Runtime &rt, const Batch &batch, Tensor &x, Norm *, const float *) override {
        fg_batch_view bv = batch.view(rt.stream);
        fg_part_call c = {};
        c.batch = &bv; c.x = x.view();
        core.call(c, rt);
        return DeferredNorm();
    }
    ExternalCore core;
};

class ExternalHead : public Head {
public:
    ExternalHead(const fg_part_vtable &v, const std::string &k, const Json &p, int dtype) : core(v, k, FG_ROLE_HEAD, p, dtype) {
        V_ = param_int(p, "vocab_size", k.c_str());
    }
    std::vector<TensorDecl> tensor_decls() const override { return core.decls(); }
    void load(const std::map<std::string, Weight> &t, Runtime &) override { core.load(t); }
    Tensor forward(Runtime &rt, const Tensor &xn, const DeferredNorm *) override {
        Tensor out = rt.arena->matrix(xn.rows, V_, FG_F32);
        fg_part_call c = {};
        c.xn = xn.view(); c.out = out.view();
        core.call(c, rt);
        return out;
    }
    ExternalCore core;

private:
    int64_t V_;
};

// A block arrangement from outside runs the engine's parts through fg_block_ops.
struct BlockCallContext {
    Runtime *rt;
    Block *block;
    const Batch *batch;
    const LayerIO *io;
    Tensor *x;
    std::string error;
};

static int block_op_guard(const fg_part_call *call, const std::function<void(BlockCallContext &)> &f) {
    BlockCallContext *ctx = (BlockCallContext *)call->engine_ctx;
    try {
        f(*ctx);
        return 0;
    } catch (const Error &e) {
        ctx->error = e.what();
        return e.code;
    } catch (const std::exception &e) {
        ctx->error = e.what();
        return FG_E_INTERNAL;
    }
}
static Tensor tensor_from_view(const fg_dev_tensor &v) {
    Tensor t;
    t.data = v.data; t.dtype = v.dtype; t.rows = v.shape[0]; t.cols = v.shape[1]; t.ld = v.ld;
    return t;
}
static int block_op_norm(const fg_part_call *call, int which, fg_dev_tensor *xn_out) {
    return block_op_guard(call, [&](BlockCallContext &c) {
        Norm *n = which == 0 ? c.block->mixer_norm : c.block->feed_forward_norm;
        *xn_out = n->forward(*c.rt, *c.x, nullptr, 0).view();
    });
}
static int block_op_mixer(const fg_part_call *call, const fg_dev_tensor *xn) {
    return block_op_guard(call, [&](BlockCallContext &c) {
        c.block->mixer->forward(*c.rt, tensor_from_view(*xn), nullptr, *c.batch, *c.io, *c.x, nullptr);
    });
}
static int block_op_ffn(const fg_part_call *call, const fg_dev_tensor *xn) {
    return block_op_guard(call, [&](BlockCallContext &c) {
        c.block->feed_forward->forward(*c.rt, tensor_from_view(*xn), nullptr, *c.batch, *c.x, nullptr);
    });
}
static const fg_block_ops kBlockOps = {block_op_norm, block_op_mixer, block_op_ffn};

class ExternalBlock : public Block {
public:
    ExternalBlock(const fg_part_vtable &v, const std::string &k, int dtype) : core(v, k, FG_ROLE_BLOCK, Json::object(), dtype) {}
    DeferredNorm forward(Runtime &rt, Tensor &x, const Batch &batch, const LayerIO &io, const DeferredNorm &, Norm *) override {
        BlockCallContext ctx{&rt, this, &batch, &io, &x, ""};
        fg_batch_view bv = batch.view(rt.stream);
        fg_layer_io iv = io.view();
        fg_part_call c = {};
        c.batch = &bv; c.io = &iv; c.residual = x.view(); c.x = x.view();
        c.block_ops = &kBlockOps; c.engine_ctx = &ctx;
        try {
            core.call(c, rt);
        } catch (const Error &e) {
            if (!ctx.error.empty()) fail(e.code, ctx.error);
            throw;
        }
        return DeferredNorm();
    }
    ExternalCore core;
};

// ------------------------------------------------------------------------------------ registries
static std::mutex g_parts_mutex;
static std::map<std::string, PartFactory> &factories(int role) {
    static std::map<std::string, PartFactory> r[9];
    static bool init = false;
    if (!init) {
        init = true;
        r[FG_ROLE_NORM]["rmsnorm"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<RMSNorm>(p); };
        r[FG_ROLE_POSITION]["rope"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<RotaryEncoding>(p); };
        r[FG_ROLE_MIXER]["gqa_attention"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<GQAAttention>(p, c); };
        r[FG_ROLE_FEED_FORWARD]["swiglu"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<SwiGLU>(p); };
        r[FG_ROLE_EMBEDDING]["embedding"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<TokenEmbedding>(p); };
        r[FG_ROLE_HEAD]["lm_head"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<LMHead>(p); };
        r[FG_ROLE_TOKEN_INPUT]["gated_token_embedding"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<GatedTokenEmbedding>(p); };
        r[FG_ROLE_STREAM_MAP]["concat_linear"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<ConcatLinear>(p); };
        r[FG_ROLE_STREAM_MAP]["add_row"] = [](Runtime &, const Json &p, BuildContext &) { return std::make_unique<AddRow>(p); };
        add_recurrent_kinds(r[FG_ROLE_MIXER]);
        add_attention_kinds(r[FG_ROLE_MIXER]);
        add_expert_kinds(r[FG_ROLE_FEED_FORWARD]);
        add_pair_kinds(r[FG_ROLE_MIXER]);
    }
    if (role < 0 || role > 8) fail(FG_E_USAGE, format("role %d does not exist", role));
    return r[role];
}
static std::map<std::string, BlockFactory> &block_factories() {
    static std::map<std::string, BlockFactory> r = {{"prenorm", [](Runtime &) { return std::make_unique<PreNormBlock>(); }},
                                                     {"sandwich", [](Runtime &) { return std::make_unique<SandwichBlock>(); }},
                                                     {"postnorm", [](Runtime &) { return std::make_unique<PostNormBlock>(); }},
                                                     {"parallel", [](Runtime &) { return std::make_unique<ParallelBlock>(); }}};
    return r;
}

void register_part_factory(int role, const std::string &kind, PartFactory f) {
    std::lock_guard<std::mutex> lock(g_parts_mutex);
    factories(role)[kind] = std::move(f);
}
void register_block_factory(const std::string &kind, BlockFactory f) {
    std::lock_guard<std::mutex> lock(g_parts_mutex);
    block_factories()[kind] = std::move(f);
}

template <typename M>
static std::string known_kinds(const M &m) {
    std::string s;
    for (auto &kv : m) s += (s.empty() ? "" : ", ") + kv.first;
    return s.empty() ? "none" : s;
}

std::unique_ptr<Part> build_part(int role, const std::string &kind, Runtime &rt, const Json &params, BuildContext &ctx) {
    PartFactory f;
    {
        std::lock_guard<std::mutex> lock(g_parts_mutex);
        auto &m = factories(role);
        auto it = m.find(kind);
        if (it == m.end())
            fail(FG_E_CONFIG, format("no %s of kind '%s' is registered (registered: %s)", role_name(role), kind.c_str(), known_kinds(m).c_str()));
        f = it->second;
    }
    return f(rt, params.is_object() ? params : Json::object(), ctx);
}

std::unique_ptr<Block> build_block(const std::string &kind, Runtime &rt) {
    BlockFactory f;
    {
        std::lock_guard<std::mutex> lock(g_parts_mutex);
        auto &m = block_factories();
        auto it = m.find(kind);
        if (it == m.end())
            fail(FG_E_CONFIG, format("no block of kind '%s' is registered (registered: %s)", kind.c_str(), known_kinds(m).c_str()));
        f = it->second;
    }
    return f(rt);
}

void register_external_part(int role, const std::string &kind, const fg_part_vtable &vt) {
    static const char *builtin[] = {"rmsnorm", "rope", "gqa_attention", "retention", "swiglu", "mlp", "moe", "prenorm", "sandwich",
                                    "embedding", "lm_head"};
    for (auto b : builtin)
        if (kind == b) fail(FG_E_USAGE, "kind '" + kind + "' is built in and cannot be replaced");
    if (kind.empty()) fail(FG_E_USAGE, "a part kind needs a name");
    fg_part_vtable v = vt;
    switch (role) {
    case FG_ROLE_NORM:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalNorm>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_POSITION:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalPosition>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_MIXER:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalMixer>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_FEED_FORWARD:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalFeedForward>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_EMBEDDING:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalEmbedding>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_HEAD:
        register_part_factory(role, kind, [v, kind](Runtime &rt, const Json &p, BuildContext &) { return std::make_unique<ExternalHead>(v, kind, p, rt.dtype); });
        break;
    case FG_ROLE_BLOCK:
        register_block_factory(kind, [v, kind](Runtime &rt) { return std::make_unique<ExternalBlock>(v, kind, rt.dtype); });
        break;
    default:
        fail(FG_E_USAGE, format("role %d does not exist", role));
    }
}

}  // namespace fg
