// Bandwidth-bound kernels of the model step: embedding gather, residual add fused
// with RMSNorm, SwiGLU, rotary tables, and rotary rotation fused with the write of
// keys and values into cache pages.
//
// Parity (formulas): kernels/execution.cu:2-5 (embedding), kernels/ops.cu:3-19 and
// kernels/execution.cu:12-24 (norm, residual+norm), kernels/execution.cu:7-10
// (SwiGLU), kernels/ops.cu:21-33 and kernels/execution.cu:28-40 (rotation, scatter)
// of nehanmohammed19/cuda-inference-serving-runtime.  The residual stream and every
// reduction stay in float here whatever the storage type.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_elementwise_set_pdl(int on) { g_pdl = on != 0; }

// ---------------------------------------------------------------- embedding
template <typename TT>
__global__ void embedding_kernel(const TT* __restrict__ table, const int* __restrict__ ids,
                                 float* __restrict__ out, int hidden, int vocab, float scale) {
    CISR_TRACE_SCOPE(TRACE_EMBEDDING);
    // Under programmatic dependent launch the kernels after this one may start (and fetch their weights) while it runs.
    // It waits for the kernel before it although it reads nothing of it: a later kernel's wait on this one then also
    // covers everything before (the block table update at the head of a step).
    pdl_trigger();
    pdl_wait();
    CISR_TRACE_WAITED();
    const int row = blockIdx.x;
    int id = ids[row];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);  // host validates; clamp keeps a bad id from reading outside
    const TT* src = table + (size_t)id * hidden;
    float* dst = out + (size_t)row * hidden;
    for (int d = threadIdx.x; d < hidden; d += blockDim.x) dst[d] = to_float(src[d]) * scale;   // scale 1 leaves the value as stored
}

CISR_EXPORT int cisr_embedding(const void* table, int table_dtype, const int* ids, float* out, int tokens,
                               int hidden, int vocab, float scale, void* stream) {
    if (tokens <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (table_dtype == CISR_BF16)
        return launch_kernel(embedding_kernel<__nv_bfloat16>, dim3(tokens), dim3(128), 0, s, g_pdl, (const __nv_bfloat16*)table, ids, out, hidden, vocab, scale);
    return launch_kernel(embedding_kernel<float>, dim3(tokens), dim3(128), 0, s, g_pdl, (const float*)table, ids, out, hidden, vocab, scale);
}

__device__ __forceinline__ float4 load_four(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load_four(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}

// The same with a second table, looked up by a hash of the token and the one before it in its sequence:
//   out[t] = table[id] * scale + pairs[(before * mul_prev + id * mul_cur) mod buckets],
// or, for a sequence's first token, the row behind the buckets.  The token before comes from the step itself, or, for
// the first token that a request brings to the step, from `last` [slots]: the last token the request brought before.
// That token's CTA, the only one that reads the slot's entry, then puts the request's newest token there.
template <typename TT>
__global__ void embedding_pairs_kernel(const TT* __restrict__ table, const TT* __restrict__ pairs, const int* __restrict__ ids,
                                       const int* __restrict__ positions, const int* __restrict__ token_req,
                                       const int* __restrict__ req_slot, const int* __restrict__ q_start, const int* __restrict__ q_len,
                                       int* __restrict__ last, float* __restrict__ out, int hidden, int vocab, float scale, int buckets,
                                       int mul_prev, int mul_cur) {
    CISR_TRACE_SCOPE(TRACE_EMBEDDING);
    __shared__ int bucket;
    pdl_trigger();
    pdl_wait();
    CISR_TRACE_WAITED();
    const int t = blockIdx.x;
    const auto token = [&](int i) { const int v = ids[i]; return v < 0 ? 0 : (v >= vocab ? vocab - 1 : v); };
    const int id = token(t);
    if (threadIdx.x == 0) {
        const int req = token_req[t], first = q_start[req];
        int before;
        if (t == first) {
            int* kept = last + req_slot[req];
            before = *kept;
            *kept = token(first + q_len[req] - 1);
        } else {
            before = token(t - 1);
        }
        // the multipliers come reduced modulo the buckets, so the sum stays below 2^62
        bucket = positions[t] == 0 ? buckets
                                   : (int)(((long long)before * mul_prev + (long long)id * mul_cur) % buckets);
    }
    __syncthreads();
    const TT* src = table + (size_t)id * hidden;
    const TT* add = pairs + (size_t)bucket * hidden;
    float* dst = out + (size_t)t * hidden;
    if (!(hidden & 3) && !((reinterpret_cast<uintptr_t>(table) | reinterpret_cast<uintptr_t>(pairs) | reinterpret_cast<uintptr_t>(out)) & 15)) {
        for (int d = 4 * threadIdx.x; d < hidden; d += 4 * blockDim.x) {
            const float4 a = load_four(src + d), b = load_four(add + d);
            *reinterpret_cast<float4*>(dst + d) = make_float4(a.x * scale + b.x, a.y * scale + b.y, a.z * scale + b.z, a.w * scale + b.w);
        }
        return;
    }
    for (int d = threadIdx.x; d < hidden; d += blockDim.x) dst[d] = to_float(src[d]) * scale + to_float(add[d]);
}

CISR_EXPORT int cisr_embedding_pairs(const void* table, const void* pairs, int table_dtype, const int* ids, const int* positions,
                                     const int* token_req, const int* req_slot, const int* q_start, const int* q_len, int* last,
                                     float* out, int tokens, int hidden, int vocab, float scale, int buckets, int mul_prev, int mul_cur,
                                     void* stream) {
    if (tokens <= 0) return 0;
    if (buckets <= 0 || mul_prev < 0 || mul_prev >= buckets || mul_cur < 0 || mul_cur >= buckets) return -2;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 block(hidden >= 2048 ? 256 : 128);
    if (table_dtype == CISR_BF16)
        return launch_kernel(embedding_pairs_kernel<__nv_bfloat16>, dim3(tokens), block, 0, s, g_pdl, (const __nv_bfloat16*)table,
                             (const __nv_bfloat16*)pairs, ids, positions, token_req, req_slot, q_start, q_len, last, out, hidden, vocab, scale,
                             buckets, mul_prev, mul_cur);
    return launch_kernel(embedding_pairs_kernel<float>, dim3(tokens), block, 0, s, g_pdl, (const float*)table, (const float*)pairs, ids,
                         positions, token_req, req_slot, q_start, q_len, last, out, hidden, vocab, scale, buckets, mul_prev, mul_cur);
}

// ---------------------------------------------------------------- residual add + RMSNorm
// For output row r: src = rows ? rows[r] : r;  v = x[src] + delta[src] * dscale;  (x[src] = v if write_back)
// out[r] = v * rsqrt(mean(v^2) + eps) * w.  dscale (float, one per channel; null: 1) is a layer scale: the output of a
// sub-block is multiplied by it on its way into the stream.
template <typename WT, typename OT>
__global__ void add_rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ delta,
                                   const WT* __restrict__ weight, OT* __restrict__ out,
                                   const int* __restrict__ rows, int hidden, float eps, int write_back,
                                   const float* __restrict__ dscale) {
    CISR_TRACE_SCOPE(TRACE_ADD_RMSNORM);
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[r] : r) * hidden;
    float* xr = x + src;
    const float* dr = delta ? delta + src : nullptr;
    extern __shared__ float row_cache[];  // hidden floats
    float sq = 0.f;
    for (int d = threadIdx.x; d < hidden; d += blockDim.x) {
        float v = xr[d];
        if (dr) v += dscale ? dr[d] * dscale[d] : dr[d];
        if (write_back && dr) xr[d] = v;
        row_cache[d] = v;
        sq += v * v;
    }
    const float total = block_sum(sq, scratch);
    const float scale = rsqrtf(total / (float)hidden + eps);
    OT* o = out + (size_t)r * hidden;
    for (int d = threadIdx.x; d < hidden; d += blockDim.x)
        o[d] = from_float<OT>(row_cache[d] * scale * to_float(weight[d]));
}

// Four weights and four outputs at a time (the row and the weights start on 16-byte boundaries, hidden % 4 == 0).
__device__ __forceinline__ float4 load_weights4(const float* w, int d4) { return reinterpret_cast<const float4*>(w)[d4]; }
__device__ __forceinline__ float4 load_weights4(const __nv_bfloat16* w, int d4) {
    const uint2 raw = reinterpret_cast<const uint2*>(w)[d4];
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
}
__device__ __forceinline__ void store4(float* o, int d4, float4 v) { reinterpret_cast<float4*>(o)[d4] = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* o, int d4, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&lo); raw.y = *reinterpret_cast<const uint32_t*>(&hi);
    reinterpret_cast<uint2*>(o)[d4] = raw;
}

// The same with 16-byte accesses, for widths that are multiples of 4.
template <typename WT, typename OT>
__global__ void add_rmsnorm_vec_kernel(float* __restrict__ x, const float* __restrict__ delta,
                                       const WT* __restrict__ weight, OT* __restrict__ out,
                                       const int* __restrict__ rows, int hidden, float eps, int write_back,
                                       const float* __restrict__ dscale) {
    CISR_TRACE_SCOPE(TRACE_ADD_RMSNORM);
    __shared__ float scratch[32];
    extern __shared__ __align__(16) float row_cache[];
    pdl_trigger();
    pdl_wait();          // x and delta come from the kernels before
    CISR_TRACE_WAITED();
    const int r = blockIdx.x, h4 = hidden >> 2;
    const size_t src = (size_t)(rows ? rows[r] : r) * hidden;
    float4* xr = reinterpret_cast<float4*>(x + src);
    const float4* dr = delta ? reinterpret_cast<const float4*>(delta + src) : nullptr;
    float4* cache4 = reinterpret_cast<float4*>(row_cache);
    float sq = 0.f;
    for (int d = threadIdx.x; d < h4; d += blockDim.x) {
        float4 v = xr[d];
        if (dr) {
            float4 dv = dr[d];
            if (dscale) { const float4 ds = reinterpret_cast<const float4*>(dscale)[d]; dv.x *= ds.x; dv.y *= ds.y; dv.z *= ds.z; dv.w *= ds.w; }
            v.x += dv.x; v.y += dv.y; v.z += dv.z; v.w += dv.w;
            if (write_back) xr[d] = v;
        }
        cache4[d] = v;
        sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float total = block_sum(sq, scratch);
    const float scale = rsqrtf(total / (float)hidden + eps);
    OT* o = out + (size_t)r * hidden;
    const bool wide = !(((uintptr_t)weight | (uintptr_t)o) & 15) && (hidden * sizeof(OT)) % 16 == 0;   // the same for the whole block
    for (int d = threadIdx.x; d < h4; d += blockDim.x) {
        const float4 v = cache4[d];
        if (wide) {
            const float4 w = load_weights4(weight, d);
            store4(o, d, make_float4(v.x * scale * w.x, v.y * scale * w.y, v.z * scale * w.z, v.w * scale * w.w));
            continue;
        }
        const float w0 = to_float(weight[4 * d]), w1 = to_float(weight[4 * d + 1]);
        const float w2 = to_float(weight[4 * d + 2]), w3 = to_float(weight[4 * d + 3]);
        o[4 * d] = from_float<OT>(v.x * scale * w0);
        o[4 * d + 1] = from_float<OT>(v.y * scale * w1);
        o[4 * d + 2] = from_float<OT>(v.z * scale * w2);
        o[4 * d + 3] = from_float<OT>(v.w * scale * w3);
    }
}

// A warp per row, the row in registers (V float4 per lane: widths up to 128 V), four rows per CTA: no shared memory
// and no barrier, every load of a lane in flight before the first is used, 8- or 16-byte stores.  Steps of many tokens
// spend a tenth of their time in this kernel, and a CTA per 576-wide row with scalar stores took 7 us for what the
// memory system moves in 2.
constexpr int NORM_WARPS = 4;
template <typename WT, typename OT, int V>
__global__ void __launch_bounds__(32 * NORM_WARPS)
add_rmsnorm_warp_kernel(float* __restrict__ x, const float* __restrict__ delta, const WT* __restrict__ weight,
                        OT* __restrict__ out, const int* __restrict__ rows, int n_rows, int hidden, float eps, int write_back,
                        const float* __restrict__ dscale) {
    CISR_TRACE_SCOPE(TRACE_ADD_RMSNORM);
    pdl_trigger();
    pdl_wait();          // x and delta come from the kernels before
    CISR_TRACE_WAITED();
    const int lane = threadIdx.x & 31, r = blockIdx.x * NORM_WARPS + (threadIdx.x >> 5), h4 = hidden >> 2;
    if (r >= n_rows) return;
    const size_t src = (size_t)(rows ? rows[r] : r) * hidden;
    float4* xr = reinterpret_cast<float4*>(x + src);
    const float4* dr = delta ? reinterpret_cast<const float4*>(delta + src) : nullptr;
    float4 v[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int d = lane + 32 * i;
        v[i] = d < h4 ? xr[d] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float sq = 0.f;
    if (dr) {
        float4 dv[V];
#pragma unroll
        for (int i = 0; i < V; ++i) {
            const int d = lane + 32 * i;
            dv[i] = d < h4 ? dr[d] : make_float4(0.f, 0.f, 0.f, 0.f);
            if (dscale && d < h4) {
                const float4 ds = reinterpret_cast<const float4*>(dscale)[d];
                dv[i].x *= ds.x; dv[i].y *= ds.y; dv[i].z *= ds.z; dv[i].w *= ds.w;
            }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) {
            v[i].x += dv[i].x; v[i].y += dv[i].y; v[i].z += dv[i].z; v[i].w += dv[i].w;
            if (write_back && lane + 32 * i < h4) xr[lane + 32 * i] = v[i];
        }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) sq += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    const float scale = rsqrtf(warp_sum(sq) / (float)hidden + eps);
    OT* o = out + (size_t)r * hidden;
#pragma unroll
    for (int i = 0; i < V; ++i) {
        const int d = lane + 32 * i;
        if (d >= h4) continue;
        const float4 w = load_weights4(weight, d);
        store4(o, d, make_float4(v[i].x * scale * w.x, v[i].y * scale * w.y, v[i].z * scale * w.z, v[i].w * scale * w.w));
    }
}

template <typename WT, typename OT, int V>
static int add_rmsnorm_warp_launch(float* x, const float* delta, const void* w, void* out, const int* rows, int n_rows,
                                   int hidden, float eps, int write_back, const float* dscale, cudaStream_t s) {
    return launch_kernel(add_rmsnorm_warp_kernel<WT, OT, V>, dim3((n_rows + NORM_WARPS - 1) / NORM_WARPS), dim3(32 * NORM_WARPS), 0, s,
                         g_pdl, x, delta, (const WT*)w, (OT*)out, rows, n_rows, hidden, eps, write_back, dscale);
}

template <typename WT, typename OT>
static int add_rmsnorm_launch(float* x, const float* delta, const void* w, void* out, const int* rows, int n_rows,
                              int hidden, float eps, int write_back, const float* dscale, cudaStream_t s) {
    const size_t smem = (size_t)hidden * sizeof(float);
    if (smem > 200 * 1024) return -2;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(add_rmsnorm_kernel<WT, OT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    const bool vec = (hidden & 3) == 0 && !(((uintptr_t)x | (uintptr_t)delta | (uintptr_t)dscale) & 15);
    // rows of up to 2048 floats whose weights and outputs are aligned too: a warp per row
    if (vec && hidden <= 2048 && !(((uintptr_t)w | (uintptr_t)out) & 15) && (hidden * sizeof(OT)) % 16 == 0) {
        const int per_lane = (hidden / 4 + 31) / 32;
        if (per_lane <= 2) return add_rmsnorm_warp_launch<WT, OT, 2>(x, delta, w, out, rows, n_rows, hidden, eps, write_back, dscale, s);
        if (per_lane <= 5) return add_rmsnorm_warp_launch<WT, OT, 5>(x, delta, w, out, rows, n_rows, hidden, eps, write_back, dscale, s);
        if (per_lane <= 8) return add_rmsnorm_warp_launch<WT, OT, 8>(x, delta, w, out, rows, n_rows, hidden, eps, write_back, dscale, s);
        return add_rmsnorm_warp_launch<WT, OT, 16>(x, delta, w, out, rows, n_rows, hidden, eps, write_back, dscale, s);
    }
    if (smem > 48 * 1024 && vec) {
        cudaError_t e = cudaFuncSetAttribute(add_rmsnorm_vec_kernel<WT, OT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    if (vec) {
        const int threads = hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128);
        return launch_kernel(add_rmsnorm_vec_kernel<WT, OT>, dim3(n_rows), dim3(threads), smem, s, g_pdl, x, delta, (const WT*)w,
                             (OT*)out, rows, hidden, eps, write_back, dscale);
    } else {
        const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
        add_rmsnorm_kernel<WT, OT><<<n_rows, threads, smem, s>>>(x, delta, (const WT*)w, (OT*)out, rows, hidden, eps, write_back, dscale);
    }
    return launch_status();
}

CISR_EXPORT int cisr_add_rmsnorm(float* x, const float* delta, const void* weight, int w_dtype, void* out,
                                 int out_dtype, const int* rows, int n_rows, int hidden, float eps, int write_back,
                                 const float* dscale, void* stream) {
    if (n_rows <= 0) return 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (w_dtype == CISR_BF16 && out_dtype == CISR_BF16)
        return add_rmsnorm_launch<__nv_bfloat16, __nv_bfloat16>(x, delta, weight, out, rows, n_rows, hidden, eps, write_back, dscale, s);
    if (w_dtype == CISR_F32 && out_dtype == CISR_BF16)
        return add_rmsnorm_launch<float, __nv_bfloat16>(x, delta, weight, out, rows, n_rows, hidden, eps, write_back, dscale, s);
    if (w_dtype == CISR_BF16 && out_dtype == CISR_F32)
        return add_rmsnorm_launch<__nv_bfloat16, float>(x, delta, weight, out, rows, n_rows, hidden, eps, write_back, dscale, s);
    return add_rmsnorm_launch<float, float>(x, delta, weight, out, rows, n_rows, hidden, eps, write_back, dscale, s);
}

// ---------------------------------------------------------------- SwiGLU
// gate_up [T, 2I] float: gate in columns [0, I), up in [I, 2I).  out = act(gate) * up, act silu (gate_act 0) or the tanh form of gelu (1), or the
// clamped form (2; common.cuh: gated_product).
template <typename OT>
__global__ void swiglu_kernel(const float* __restrict__ gate_up, OT* __restrict__ out, int inter, int gate_act, float gate_limit, size_t total) {
    CISR_TRACE_SCOPE(TRACE_SWIGLU);
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / inter;
    const int c = (int)(i - t * inter);
    const float g = gate_up[t * 2 * inter + c];
    const float u = gate_up[t * 2 * inter + inter + c];
    out[i] = from_float<OT>(gated_product(g, u, gate_act, gate_limit));
}

CISR_EXPORT int cisr_swiglu(const float* gate_up, void* out, int out_dtype, int tokens, int inter, int gate_act, float gate_limit,
                            void* stream) {
    const size_t total = (size_t)tokens * inter;
    if (!total) return 0;
    const unsigned blocks = (unsigned)((total + 255) / 256);
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == CISR_BF16) swiglu_kernel<<<blocks, 256, 0, s>>>(gate_up, (__nv_bfloat16*)out, inter, gate_act, gate_limit, total);
    else swiglu_kernel<<<blocks, 256, 0, s>>>(gate_up, (float*)out, inter, gate_act, gate_limit, total);
    return launch_status();
}

// ---------------------------------------------------------------- activation of a dense feed-forward
// out[t, c] = act(x[t, c]) for c < cols, 0 for cols <= c < out_cols (columns that pad the next product's K).
// kind 0: max(z, 0)^2;  1: gelu, tanh form, 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)));  2: silu.
template <typename OT>
__global__ void activation_kernel(const float* __restrict__ x, OT* __restrict__ out, int cols, int out_cols, int kind, size_t total) {
    pdl_trigger();
    pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const size_t t = i / out_cols;
    const int c = (int)(i - t * out_cols);
    float v = 0.f;
    if (c < cols) {
        const float z = x[t * cols + c];
        if (kind == 0) { const float r = fmaxf(z, 0.f); v = r * r; }
        else if (kind == 1) v = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
        else v = z / (1.f + expf(-z));
    }
    out[i] = from_float<OT>(v);
}

CISR_EXPORT int cisr_activation(const float* x, void* out, int out_dtype, int tokens, int cols, int out_cols, int kind, void* stream) {
    const size_t total = (size_t)tokens * out_cols;
    if (!total) return 0;
    if (kind < 0 || kind > 2 || out_cols < cols) return -2;
    const dim3 grid((unsigned)((total + 255) / 256));
    if (out_dtype == CISR_BF16)
        return launch_kernel(activation_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, g_pdl, x, (__nv_bfloat16*)out, cols, out_cols, kind, total);
    return launch_kernel(activation_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, g_pdl, x, (float*)out, cols, out_cols, kind, total);
}

// ---------------------------------------------------------------- rotary tables
// cos/sin [T, half] in float from double angles pos * inv_freq[i], both times `magnitude` (1 unless the encoding
// scales its tables); run once per step
// and shared by every layer that rotates with the same theta and width.
__global__ void rotary_table_kernel(const int* __restrict__ positions, const double* __restrict__ inv_freq,
                                    float* __restrict__ cos_out, float* __restrict__ sin_out, int half, int total, double magnitude) {
    CISR_TRACE_SCOPE(TRACE_ROTARY_TABLE);
    // No early start for the kernels after this one: the fused q/k/v kernels read these tables before their own wait
    // on their predecessor, so whatever runs between this kernel and them must not start before the tables are written.
    pdl_wait();          // nothing of the kernel before is read, but the chain of waits must not break (see embedding_kernel)
    CISR_TRACE_WAITED();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int t = i / half, f = i - t * half;
    double s, c;
    sincos((double)positions[t] * inv_freq[f], &s, &c);
    cos_out[i] = (float)(c * magnitude);
    sin_out[i] = (float)(s * magnitude);
}

CISR_EXPORT int cisr_rotary_tables(const int* positions, const double* inv_freq, float* cos_out, float* sin_out,
                                   int tokens, int half, double magnitude, void* stream) {
    const int total = tokens * half;
    if (total <= 0) return 0;
    return launch_kernel(rotary_table_kernel, dim3((total + 127) / 128), dim3(128), 0, (cudaStream_t)stream, g_pdl, positions, inv_freq,
                         cos_out, sin_out, half, total, magnitude);
}

// ---------------------------------------------------------------- rotation + cache write
// proj [T, row_stride] float holds q at column 0, k at k_col, v at v_col (k_col < 0: no keys/values
// in this projection, nothing is written to the cache).  The first 2*rot_half coordinates of each head
// are rotated (pairs (i, i+rot_half), or (2i, 2i+1) when interleaved); the rest pass through.
// q goes to q_out [T, Hq, D]; k (rotated) and v go to page block_table[req_slot[req]][pos / P], offset pos % P,
// in caches laid out [pages, Hkv, P, D].
template <typename QT, typename CT>
__global__ void rope_store_kernel(const float* __restrict__ proj, int row_stride, int k_col, int v_col,
                                  const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_half,
                                  int interleaved, QT* __restrict__ q_out, CT* __restrict__ k_cache,
                                  CT* __restrict__ v_cache, const int* __restrict__ token_req,
                                  const int* __restrict__ positions, const int* __restrict__ req_slot,
                                  const int* __restrict__ block_table, int table_width, int page_size, int hq,
                                  int hkv, int dim) {
    CISR_TRACE_SCOPE(TRACE_ROPE_STORE);
    const int t = blockIdx.x;
    const float* row = proj + (size_t)t * row_stride;
    const float* cs = cos_t ? cos_t + (size_t)t * rot_half : nullptr;
    const float* sn = sin_t ? sin_t + (size_t)t * rot_half : nullptr;
    const int rot = 2 * rot_half;
    // queries
    for (int i = threadIdx.x; i < hq * dim; i += blockDim.x) {
        const int h = i / dim, d = i - h * dim;
        const float* src = row + h * dim;
        float v = src[d];
        if (d < rot) {
            int f, other; bool first;
            if (interleaved) { f = d >> 1; first = !(d & 1); other = first ? d + 1 : d - 1; }
            else { first = d < rot_half; f = first ? d : d - rot_half; other = first ? d + rot_half : d - rot_half; }
            const float c = cs[f], s = sn[f], o = src[other];
            v = first ? v * c - o * s : v * c + o * s;
        }
        q_out[((size_t)t * hq + h) * dim + d] = from_float<QT>(v);
    }
    if (k_col < 0) return;
    const int pos = positions[t];
    const int page = block_table[(size_t)req_slot[token_req[t]] * table_width + pos / page_size];
    const int off = pos % page_size;
    if (page < 0) return;  // the host reserves a page before every write; never follow a missing entry
    for (int i = threadIdx.x; i < hkv * dim; i += blockDim.x) {
        const int h = i / dim, d = i - h * dim;
        const float* src = row + k_col + h * dim;
        float v = src[d];
        if (d < rot) {
            int f, other; bool first;
            if (interleaved) { f = d >> 1; first = !(d & 1); other = first ? d + 1 : d - 1; }
            else { first = d < rot_half; f = first ? d : d - rot_half; other = first ? d + rot_half : d - rot_half; }
            const float c = cs[f], s = sn[f], o = src[other];
            v = first ? v * c - o * s : v * c + o * s;
        }
        const size_t dst = (((size_t)page * hkv + h) * page_size + off) * dim + d;
        k_cache[dst] = from_float<CT>(v);
        v_cache[dst] = from_float<CT>(row[v_col + h * dim + d]);
    }
}

CISR_EXPORT int cisr_rope_store(const float* proj, int row_stride, int k_col, int v_col, const float* cos_t,
                                const float* sin_t, int rot_half, int interleaved, void* q_out, int q_dtype,
                                void* k_cache, void* v_cache, int cache_dtype, const int* token_req,
                                const int* positions, const int* req_slot, const int* block_table, int table_width,
                                int page_size, int hq, int hkv, int dim, int tokens, void* stream) {
    if (tokens <= 0) return 0;
    if (2 * rot_half > dim || rot_half < 0) return -2;
    cudaStream_t s = (cudaStream_t)stream;
#define CISR_ROPE(QT, CT)                                                                                          \
    rope_store_kernel<QT, CT><<<tokens, 128, 0, s>>>(proj, row_stride, k_col, v_col, cos_t, sin_t, rot_half,        \
                                                      interleaved, (QT*)q_out, (CT*)k_cache, (CT*)v_cache, token_req, \
                                                      positions, req_slot, block_table, table_width, page_size, hq, hkv, dim)
    if (q_dtype == CISR_BF16 && cache_dtype == CISR_BF16) CISR_ROPE(__nv_bfloat16, __nv_bfloat16);
    else if (q_dtype == CISR_F32 && cache_dtype == CISR_F32) CISR_ROPE(float, float);
    else if (q_dtype == CISR_BF16 && cache_dtype == CISR_F32) CISR_ROPE(__nv_bfloat16, float);
    else CISR_ROPE(float, __nv_bfloat16);
#undef CISR_ROPE
    return launch_status();
}

// ---------------------------------------------------------------- stream add and plain scaling
// x[t, d] += delta[t, d] * dscale[d] + vec[d]: a pending sub-block output (with its layer scale) and a per-pass vector
// enter the residual stream in one pass over it.  Any of delta, dscale and vec may be null.
__global__ void stream_add_kernel(float* __restrict__ x, const float* __restrict__ delta, const float* __restrict__ dscale,
                                  const float* __restrict__ vec, int hidden, size_t total) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    const int d = (int)(i % hidden);
    float v = x[i];
    if (delta) v += dscale ? delta[i] * dscale[d] : delta[i];
    if (vec) v += vec[d];
    x[i] = v;
}

CISR_EXPORT int cisr_stream_add(float* x, const float* delta, const float* dscale, const float* vec, int tokens, int hidden,
                                void* stream) {
    const size_t total = (size_t)tokens * hidden;
    if (!total) return 0;
    stream_add_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, delta, dscale, vec, hidden, total);
    return launch_status();
}

__global__ void scale_kernel(float* __restrict__ x, float scale, size_t total) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) x[i] *= scale;
}

CISR_EXPORT int cisr_scale(float* x, long long total, float scale, void* stream) {
    if (total <= 0) return 0;
    scale_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(x, scale, (size_t)total);
    return launch_status();
}

// ---------------------------------------------------------------- page copy (copy-on-write of a shared page)
// Copies whole pages inside one pool: pool viewed as [n_planes, pages, page_elems]; pairs (src, dst) in `pairs`.
__global__ void page_copy_kernel(uint4* __restrict__ pool, const int* __restrict__ pairs, size_t plane_vec,
                                 size_t page_vec) {
    CISR_TRACE_SCOPE(TRACE_PAGE_COPY);
    const int pair = blockIdx.x, plane = blockIdx.y;
    const uint4* src = pool + plane * plane_vec + (size_t)pairs[2 * pair] * page_vec;
    uint4* dst = pool + plane * plane_vec + (size_t)pairs[2 * pair + 1] * page_vec;
    for (size_t i = threadIdx.x; i < page_vec; i += blockDim.x) dst[i] = src[i];
}

CISR_EXPORT int cisr_page_copy(void* pool, const int* pairs, int n_pairs, int n_planes, long long plane_bytes,
                               long long page_bytes, void* stream) {
    if (n_pairs <= 0) return 0;
    if (page_bytes % 16 || plane_bytes % 16) return -2;
    page_copy_kernel<<<dim3(n_pairs, n_planes), 128, 0, (cudaStream_t)stream>>>((uint4*)pool, pairs, plane_bytes / 16,
                                                                                 page_bytes / 16);
    return launch_status();
}

// ---------------------------------------------------------------- block table updates
// table[idx[i]] = val[i]; the host sends one value per entry, so the order does not matter.
// Launched plainly, and it never lets its successors start early: kernels further down the step read the table before
// their own wait on their predecessor, which is safe only because nothing after this kernel starts before it is done.
__global__ void table_update_kernel(int* __restrict__ table, const int* __restrict__ idx, const int* __restrict__ val, int n) {
    CISR_TRACE_SCOPE(TRACE_TABLE_UPDATE);
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n && idx[i] >= 0) table[idx[i]] = val[i];
}

CISR_EXPORT int cisr_table_update(int* table, const int* idx, const int* val, int n, void* stream) {
    if (n <= 0) return 0;
    table_update_kernel<<<(n + 127) / 128, 128, 0, (cudaStream_t)stream>>>(table, idx, val, n);
    return launch_status();
}
