// Row kernels around the recurrences: short causal convolutions with their kept inputs, the step sizes of the
// state-space mixer, the exponential gates of the matrix memory, and what turns their read-outs into the operand of an
// output projection.  Float arithmetic throughout; one rounding where the output type is narrower.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_recurrent_rows_set_pdl(int on) { g_pdl = on != 0; }

namespace {
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------ short convolution over time
// out[t][c] = act(bias[c] + sum_j taps[n - 1 - j][c] * in(t - j, c)),  in(t, c) = proj[t][col + c] + in_bias[c] inside the
// portion, the request's kept inputs before it (zeros before the sequence: they are kept inputs that were never written).
// The kept inputs (keep [taps - 1][channels] inside the request's state row, oldest first, WITH in_bias) become the portion's last.
//
// A CTA takes a tile of at most `tile` neighbouring tokens of one request and 128 channels; a channel is one thread's.  The
// tile is at least taps - 1 tokens, so only a portion's first tile reads kept inputs, and that CTA, after reading them,
// writes the new ones.
//
// STEPS: one more CTA per tile makes the step sizes of the state-space mixer from `heads` further columns of proj:
//     dt = softplus(proj[t][dt_col + h] + dt_bias[h]);   la[t][h] = -exp(a_log[h]) dt;   g[t][h] = dt
// SPLIT: out is also written as three bfloat16 numbers whose sum it is up to 2^-24 of it (the next product's operand on
// the tensor cores, kept as accurate as a float one): split [blocks][split_rows][3][block], block = channels / blocks.
struct ConvArgs {
    const float* proj; int stride, col; const float* in_bias;
    const float* taps_w; const float* bias; int taps, channels, act;
    float* state; long long state_stride, keep_offset;
    const int* req_slot; const int* q_start; const int* q_len; const int* tile_req; const int* tile_t0; int tile;
    float* out;
    int dt_col, heads; const float* dt_bias; const float* a_log; float* la; float* g;
    __nv_bfloat16* split; int split_block; long long split_rows;
};
constexpr int CONV_THREADS = 128;

// TAPS > 0: that many taps, the last inputs in registers; 0: any number, inputs read again (from cache) per tap
template <int TAPS>
__global__ void __launch_bounds__(CONV_THREADS)
short_conv_kernel(const ConvArgs a) {
    pdl_trigger();
    const int r = a.tile_req[blockIdx.x], t0 = a.tile_t0[blockIdx.x];
    const int n = a.q_len[r], first = a.q_start[r], count = min(a.tile, n - t0);
    const int conv_ctas = (a.channels + CONV_THREADS - 1) / CONV_THREADS;
    if ((int)blockIdx.y >= conv_ctas) {                       // step sizes
        pdl_wait();
        for (int i = threadIdx.x; i < count * a.heads; i += CONV_THREADS) {
            const int t = i / a.heads, h = i - t * a.heads;
            const size_t tok = (size_t)(first + t0 + t);
            const float dt = softplus_f(a.proj[tok * a.stride + a.dt_col + h] + a.dt_bias[h]);
            a.la[tok * a.heads + h] = -expf(a.a_log[h]) * dt;
            a.g[tok * a.heads + h] = dt;
        }
        return;
    }
    const int c = blockIdx.y * CONV_THREADS + threadIdx.x;
    const bool live = c < a.channels;
    const int taps = TAPS ? TAPS : a.taps;
    float w[TAPS ? TAPS : 1], bias = 0.f, in_bias = 0.f;
    if (live) {
        bias = a.bias ? a.bias[c] : 0.f;
        in_bias = a.in_bias ? a.in_bias[c] : 0.f;
        if (TAPS) {
#pragma unroll
            for (int j = 0; j < (TAPS ? TAPS : 1); ++j) w[j] = a.taps_w[(size_t)j * a.channels + c];
        }
    }
    pdl_wait();
    if (!live) return;
    float* keep = a.state + (size_t)a.req_slot[r] * a.state_stride + a.keep_offset + c;      // row i at keep[i * channels]
    const float* col = a.proj + (size_t)first * a.stride + a.col + c;                        // local token t at col[t * stride]
    const auto input = [&](int t) { return t >= 0 ? col[(size_t)t * a.stride] + in_bias : keep[(size_t)(taps - 1 + t) * a.channels]; };
    const auto write = [&](int t, float acc) {
        const float v = a.act ? silu_f(acc) : acc;
        a.out[(size_t)(first + t) * a.channels + c] = v;
        if (a.split) {
            const int block = c / a.split_block, at = c - block * a.split_block;
            __nv_bfloat16* dst = a.split + (((size_t)block * a.split_rows + first + t) * 3) * a.split_block + at;
            const __nv_bfloat16 hi = __float2bfloat16_rn(v);
            const float rest = v - __bfloat162float(hi);
            const __nv_bfloat16 mid = __float2bfloat16_rn(rest);
            dst[0] = hi;
            dst[a.split_block] = mid;
            dst[2 * a.split_block] = __float2bfloat16_rn(rest - __bfloat162float(mid));
        }
    };
    if (TAPS) {
        float x[TAPS ? TAPS : 1];
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) x[j] = input(t0 - (TAPS - 1) + j);
        for (int b = 0; b < count; b += 4) {
            float next[4];
#pragma unroll
            for (int u = 0; u < 4; ++u) next[u] = b + u < count ? input(t0 + b + u) : 0.f;
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (b + u < count) {
                    x[TAPS - 1] = next[u];
                    float acc = bias;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], x[j], acc);
#pragma unroll
                    for (int j = 0; j + 1 < TAPS; ++j) x[j] = x[j + 1];
                    write(t0 + b + u, acc);
                }
            }
        }
    } else {
        for (int t = t0; t < t0 + count; ++t) {
            float acc = bias;
            for (int j = 0; j < taps; ++j) acc = fmaf(a.taps_w[(size_t)j * a.channels + c], input(t - (taps - 1) + j), acc);
            write(t, acc);
        }
    }
    if (t0 == 0)
        for (int i = 0; i < taps - 1; ++i) {                  // rows move towards zero: each is read before it is overwritten
            const int at = n - (taps - 1) + i;
            keep[(size_t)i * a.channels] = at >= 0 ? col[(size_t)at * a.stride] + in_bias : keep[(size_t)(i + n) * a.channels];
        }
}

// ------------------------------------------------------------------ exponential gates with a running maximum
// i = cap tanh((x_i + b_i) / cap), f = logsigmoid(cap tanh((x_f + b_f) / cap)) per token and head, and with the request's
// running maximum (one float per head in its state row):
//     m_t = max(f_t + m_(t-1), i_t);   la_t = f_t + m_(t-1) - m_t;   g_t = exp(i_t - m_t)
// A CTA takes one head of one request, blockDim.x tokens at a time: m is a scan of the pairs (F, M), which stand for
// m -> max(m + F, M).  Whatever value a rounding leaves in m_t, la and g are formed from the values stored, so the state
// stays the true one times exp(-m_t).
__global__ void __launch_bounds__(256)
exp_gates_kernel(const float* __restrict__ proj, int stride, int i_col, int f_col, const float* __restrict__ i_bias,
                 const float* __restrict__ f_bias, float cap, float* __restrict__ state, long long state_stride, long long m_offset,
                 const int* __restrict__ req_slot, const int* __restrict__ q_start, const int* __restrict__ q_len, float* __restrict__ la,
                 float* __restrict__ g, float* __restrict__ m_out, int heads) {
    __shared__ float wF[8], wM[8], carry;
    pdl_trigger();
    const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int n = q_len[r], first = q_start[r];
    float* kept = state + (size_t)req_slot[r] * state_stride + m_offset + h;
    const float bi = i_bias[h], bf = f_bias[h];
    float m_before = n > 0 ? *kept : 0.f;
    pdl_wait();
    for (int t0 = 0; t0 < n; t0 += blockDim.x) {
        const int t = t0 + threadIdx.x;
        const bool in = t < n;
        float f = 0.f, i = -INFINITY;                         // beyond the portion: m -> m
        if (in) {
            const float* row = proj + (size_t)(first + t) * stride;
            i = cap * tanhf((row[i_col + h] + bi) / cap);
            f = -softplus_f(-cap * tanhf((row[f_col + h] + bf) / cap));
        }
        float F = f, M = i;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const float F0 = __shfl_up_sync(0xffffffffu, F, off), M0 = __shfl_up_sync(0xffffffffu, M, off);
            if (lane >= off) { M = fmaxf(M0 + F, M); F += F0; }
        }
        if (lane == 31) { wF[warp] = F; wM[warp] = M; }
        __syncthreads();
        float base = m_before;                                // m at the end of the warps before this one
        for (int w = 0; w < warp; ++w) base = fmaxf(base + wF[w], wM[w]);
        const float m = fmaxf(base + F, M);
        float prev = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) prev = base;
        if (in) {
            const size_t at = (size_t)(first + t) * heads + h;
            la[at] = f + prev - m;
            g[at] = expf(i - m);
            m_out[at] = m;
        }
        if (in && (threadIdx.x == blockDim.x - 1 || t == n - 1)) carry = m;      // the very number that the last token's la and g were formed with
        __syncthreads();
        m_before = carry;
    }
    if (n > 0 && threadIdx.x == 0) *kept = m_before;
}

// Per (token, head): o = y / (max(|yn|, exp(-m)) + 1e-6), o / sqrt(mean(o^2) + eps) * norm_w * sigmoid(gate); a warp each.
template <typename OT>
__global__ void __launch_bounds__(128)
exp_output_kernel(const float* __restrict__ y, const float* __restrict__ yn, const float* __restrict__ m, const float* __restrict__ gate,
                  int gate_stride, int gate_col, const float* __restrict__ norm_w, float eps, OT* __restrict__ out, int out_stride,
                  int heads, int dv, int tokens) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const size_t pair = (size_t)blockIdx.x * 4 + (threadIdx.x >> 5);
    const size_t t = pair / heads;
    const int h = (int)(pair - t * heads);
    if (t >= (size_t)tokens) return;
    const float down = 1.f / (fmaxf(fabsf(yn[pair]), expf(-m[pair])) + 1e-6f);
    const float* src = y + pair * dv;
    float sq = 0.f;
    for (int d = lane; d < dv; d += 32) { const float o = src[d] * down; sq += o * o; }
    const float inv = down / sqrtf(warp_sum(sq) / (float)dv + eps);
    const float* gr = gate + t * gate_stride + gate_col + h * dv;
    OT* dst = out + t * out_stride + h * dv;
    for (int d = lane; d < dv; d += 32) dst[d] = from_float<OT>(src[d] * inv * norm_w[h * dv + d] * sigmoid_f(gr[d]));
}

// ------------------------------------------------------------------ output of the state-space mixer
// Per token: v = (y + D_h x) silu(z), v / sqrt(mean over its part of v^2 + eps) * norm_w * scale, in `parts` equal parts of
// the row; written to columns [at, at + inner) of out.  `lead` (lead_width columns, same type as out): another operand of the same
// output projection, copied to the columns in front; columns behind the row are zeroed.
template <typename OT>
__global__ void __launch_bounds__(1024)
ssd_output_kernel(const float* __restrict__ y, const float* __restrict__ x, int x_stride, const float* __restrict__ D,
                  const float* __restrict__ z, int z_stride, int z_col, const float* __restrict__ norm_w, float eps, float scale, int parts,
                  const OT* __restrict__ lead, int lead_width, OT* __restrict__ out, int out_stride, int heads, int dv) {
    extern __shared__ float row[];            // inner floats
    __shared__ float scratch[32];
    pdl_trigger();
    const size_t t = blockIdx.x;
    const int inner = heads * dv, part = inner / parts;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
    pdl_wait();
    const float* yr = y + t * inner;
    const float* xr = x + t * x_stride;
    const float* zr = z + t * z_stride + z_col;
    float sq = 0.f;
    for (int d = threadIdx.x; d < inner; d += blockDim.x) {
        const float v = fmaf(D[d / dv], xr[d], yr[d]) * silu_f(zr[d]);
        row[d] = v;
        sq = fmaf(v, v, sq);
    }
    OT* dst = out + t * out_stride;
    for (int d = threadIdx.x; d < lead_width; d += blockDim.x) dst[d] = lead[t * lead_width + d];
    dst += lead_width;
    for (int d = inner + threadIdx.x; d < out_stride - lead_width; d += blockDim.x) dst[d] = from_float<OT>(0.f);
    if (parts == 1) {
        const float inv = scale / sqrtf(block_sum(sq, scratch) / (float)inner + eps);
        for (int d = threadIdx.x; d < inner; d += blockDim.x) dst[d] = from_float<OT>(row[d] * inv * norm_w[d]);
        return;
    }
    __syncthreads();
    for (int p = warp; p < parts; p += n_warps) {
        const float* v = row + p * part;
        float s = 0.f;
        for (int d = lane; d < part; d += 32) s = fmaf(v[d], v[d], s);
        const float inv = scale / sqrtf(warp_sum(s) / (float)part + eps);
        for (int d = lane; d < part; d += 32) dst[p * part + d] = from_float<OT>(v[d] * inv * norm_w[p * part + d]);
    }
}
}  // namespace

CISR_EXPORT int cisr_short_conv(const float* proj, int stride, int col, const float* in_bias, const float* taps_w, const float* bias, int taps,
                                int channels, int act, float* state, long long state_stride, long long keep_offset, const int* req_slot,
                                const int* q_start, const int* q_len, const int* tile_req, const int* tile_t0, int n_tiles, int tile,
                                float* out, int dt_col, int heads, const float* dt_bias, const float* a_log, float* la, float* g,
                                void* split, int split_block, long long split_rows, void* stream) {
    if (n_tiles <= 0) return 0;
    if (taps < 1 || channels <= 0 || tile < taps - 1 || tile < 1 || heads < 0) return -2;
    if (split && (split_block <= 0 || channels % split_block)) return -2;
    ConvArgs a;
    a.proj = proj; a.stride = stride; a.col = col; a.in_bias = in_bias; a.taps_w = taps_w; a.bias = bias; a.taps = taps; a.channels = channels;
    a.act = act; a.state = state; a.state_stride = state_stride; a.keep_offset = keep_offset; a.req_slot = req_slot; a.q_start = q_start;
    a.q_len = q_len; a.tile_req = tile_req; a.tile_t0 = tile_t0; a.tile = tile; a.out = out; a.dt_col = dt_col; a.heads = heads;
    a.dt_bias = dt_bias; a.a_log = a_log; a.la = la; a.g = g; a.split = (__nv_bfloat16*)split; a.split_block = split_block; a.split_rows = split_rows;
    const dim3 grid(n_tiles, (channels + CONV_THREADS - 1) / CONV_THREADS + (heads > 0 ? 1 : 0));
    cudaStream_t s = (cudaStream_t)stream;
    switch (taps) {
        case 2: return launch_kernel(short_conv_kernel<2>, grid, dim3(CONV_THREADS), 0, s, g_pdl, a);
        case 3: return launch_kernel(short_conv_kernel<3>, grid, dim3(CONV_THREADS), 0, s, g_pdl, a);
        case 4: return launch_kernel(short_conv_kernel<4>, grid, dim3(CONV_THREADS), 0, s, g_pdl, a);
        default: return launch_kernel(short_conv_kernel<0>, grid, dim3(CONV_THREADS), 0, s, g_pdl, a);
    }
}

CISR_EXPORT int cisr_exp_gates(const float* proj, int stride, int i_col, int f_col, const float* i_bias, const float* f_bias, float cap,
                               float* state, long long state_stride, long long m_offset, const int* req_slot, const int* q_start,
                               const int* q_len, float* la, float* g, float* m_out, int heads, int n_req, int longest, void* stream) {
    if (n_req <= 0) return 0;
    if (heads <= 0 || !(cap > 0.f)) return -2;
    const int threads = longest <= 32 ? 32 : longest <= 128 ? 128 : 256;       // `longest`: a bound on the portions, for speed only
    return launch_kernel(exp_gates_kernel, dim3(n_req, heads), dim3(threads), 0, (cudaStream_t)stream, g_pdl, proj, stride, i_col, f_col, i_bias,
                         f_bias, cap, state, state_stride, m_offset, req_slot, q_start, q_len, la, g, m_out, heads);
}

CISR_EXPORT int cisr_exp_output(const float* y, const float* yn, const float* m, const float* gate, int gate_stride, int gate_col,
                                const float* norm_w, float eps, void* out, int out_dtype, int out_stride, int heads, int dv, int tokens,
                                void* stream) {
    if (tokens <= 0) return 0;
    const dim3 grid((unsigned)(((size_t)tokens * heads + 3) / 4));
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == CISR_BF16)
        return launch_kernel(exp_output_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, g_pdl, y, yn, m, gate, gate_stride, gate_col, norm_w, eps,
                             (__nv_bfloat16*)out, out_stride, heads, dv, tokens);
    return launch_kernel(exp_output_kernel<float>, grid, dim3(128), 0, s, g_pdl, y, yn, m, gate, gate_stride, gate_col, norm_w, eps, (float*)out,
                         out_stride, heads, dv, tokens);
}

template <typename OT>
static int ssd_output_launch(const float* y, const float* x, int x_stride, const float* D, const float* z, int z_stride, int z_col,
                             const float* norm_w, float eps, float scale, int parts, const void* lead, int lead_width, void* out, int out_stride,
                             int heads, int dv, int tokens, cudaStream_t s) {
    const size_t smem = sizeof(float) * (size_t)heads * dv;
    if (smem > 200 * 1024) return -3;
    static size_t configured = 48 * 1024;
    if (smem > configured) {
        cudaError_t e = cudaFuncSetAttribute(ssd_output_kernel<OT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = smem;
    }
    const int threads = (tokens <= 64 && heads * dv >= 1024) ? 1024 : 256;      // few tokens (a decode step): a token's row on more threads
    return launch_kernel(ssd_output_kernel<OT>, dim3(tokens), dim3(threads), smem, s, g_pdl, y, x, x_stride, D, z, z_stride, z_col, norm_w, eps,
                         scale, parts, (const OT*)lead, lead_width, (OT*)out, out_stride, heads, dv);
}

CISR_EXPORT int cisr_ssd_output(const float* y, const float* x, int x_stride, const float* D, const float* z, int z_stride, int z_col,
                                const float* norm_w, float eps, float scale, int parts, const void* lead, int lead_width, void* out,
                                int out_dtype, int out_stride, int heads, int dv, int tokens, void* stream) {
    if (tokens <= 0) return 0;
    if (heads <= 0 || dv <= 0 || parts <= 0 || (heads * dv) % parts || lead_width < 0 || out_stride < lead_width + heads * dv) return -2;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == CISR_BF16)
        return ssd_output_launch<__nv_bfloat16>(y, x, x_stride, D, z, z_stride, z_col, norm_w, eps, scale, parts, lead, lead_width, out, out_stride,
                                                heads, dv, tokens, s);
    return ssd_output_launch<float>(y, x, x_stride, D, z, z_stride, z_col, norm_w, eps, scale, parts, lead, lead_width, out, out_stride, heads, dv,
                                    tokens, s);
}
