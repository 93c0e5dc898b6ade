// From the stacked q | k | v projection of a step to the operands of the paged attention kernels, one CTA per token:
// biases, a norm over a whole projection, rotation of part of each head, heads padded to the width the attention
// kernels are built for, keys and values written into their cache pages.
//
//   row   = proj[t] + bias                                   (bias null: none)
//   qn    = q_norm ? q / sqrt(mean(q^2) + eps) * q_norm : q  (the mean runs over ALL query heads of the token at once, or,
//           per_head, over each head by itself with one weight of key_dim numbers for all of them)
//   kn    = k_norm ? k / sqrt(mean(k^2) + eps) * k_norm : k
//   qn    *= 1 + temp_coef ln(floor((position + 1) / temp_every) + 1)           (temp_coef 0: as it is)
//   q_out[t][h] = [rotate(qn_h) | 0]                          (key_dim wide, padded with zeros to D)
//   k_cache[page][g][off] = [rotate(kn_g) | 0]
//   v_cache[page][g][off] = [v_g | 0]  with v from its own columns, or (v_col < 0) the key as projected: with its bias,
//                                      before norm and rotation; value_dim = key_dim then
//   with `v_other` the value is blended first: v <- (1 - blend) v + blend v_other[t]   (v_other: rows `other_stride` apart)
//
// The first 2 * rot_half coordinates of a head turn; pairs are (i, i + rot_half) or, interleaved, (2i, 2i + 1).
// The tables hold cos and sin per (token, pair), already multiplied by whatever factor the encoding wants.
// Float arithmetic; one rounding where q_out and the cache have a narrower type.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_attention_rows_set_pdl(int on) { g_pdl = on != 0; }

namespace {
__device__ __forceinline__ float turned(const float* head, const float* w, float inv, int d, int rot_half, int interleaved,
                                        const float* cs, const float* sn) {
    // value d of a head after the optional norm (common factor inv, per-coordinate weight w) and the rotation
    float v = head[d] * inv * (w ? w[d] : 1.f);
    if (d < 2 * rot_half) {
        int f, other; bool first;
        if (interleaved) { f = d >> 1; first = !(d & 1); other = first ? d + 1 : d - 1; }
        else { first = d < rot_half; f = first ? d : d - rot_half; other = first ? d + rot_half : d - rot_half; }
        const float o = head[other] * inv * (w ? w[other] : 1.f);
        v = first ? v * cs[f] - o * sn[f] : v * cs[f] + o * sn[f];
    }
    return v;
}

// Coordinates d .. d + 3 of a head whose weight is in the row already (times the common factor inv), pairs across the halves,
// d, rot_half and the head's place in the row multiples of four: all four lie in the same half, and so do their partners.
__device__ __forceinline__ float4 turned_four(const float* head, float inv, int d, int rot_half, const float* cs, const float* sn) {
    const float4 x = *reinterpret_cast<const float4*>(head + d);
    if (d >= 2 * rot_half) return make_float4(x.x * inv, x.y * inv, x.z * inv, x.w * inv);
    const bool first = d < rot_half;
    const int f = first ? d : d - rot_half;
    const float4 y = *reinterpret_cast<const float4*>(head + (first ? d + rot_half : f));
    const float4 c = *reinterpret_cast<const float4*>(cs + f), s = *reinterpret_cast<const float4*>(sn + f);
    const float sign = first ? -inv : inv;
    return make_float4(x.x * inv * c.x + sign * y.x * s.x, x.y * inv * c.y + sign * y.y * s.y, x.z * inv * c.z + sign * y.z * s.z,
                       x.w * inv * c.w + sign * y.w * s.w);
}
__device__ __forceinline__ void store_four(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* dst, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&lo); raw.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = raw;
}

// Coordinates d and d + 1 (d even) of a head after norm and rotation.  Neighbouring pairs turn together, so one pair of
// table entries serves both; the other pairing takes each coordinate's partner from across the head.
__device__ __forceinline__ float2 turned_pair(const float* head, const float* w, float inv, int d, int width, int rot_half,
                                              int interleaved, const float* cs, const float* sn) {
    if (d + 1 >= width || !interleaved || d >= 2 * rot_half)
        return make_float2(d < width ? turned(head, w, inv, d, rot_half, interleaved, cs, sn) : 0.f,
                           d + 1 < width ? turned(head, w, inv, d + 1, rot_half, interleaved, cs, sn) : 0.f);
    const float a = head[d] * inv * (w ? w[d] : 1.f), b = head[d + 1] * inv * (w ? w[d + 1] : 1.f);
    const float c = cs[d >> 1], s = sn[d >> 1];
    return make_float2(a * c - b * s, b * c + a * s);
}
__device__ __forceinline__ void store_pair(float* dst, float2 v) { *reinterpret_cast<float2*>(dst) = v; }
__device__ __forceinline__ void store_pair(__nv_bfloat16* dst, float2 v) { *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(v.x, v.y); }

template <typename QT, typename CT>
__global__ void __launch_bounds__(1024)
attention_rows_kernel(const float* __restrict__ proj, int row_stride, int k_col, int v_col, const float* __restrict__ bias,
                      const float* __restrict__ q_norm, const float* __restrict__ k_norm, float eps,
                      const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_half, int interleaved,
                      QT* __restrict__ q_out, CT* __restrict__ k_cache, CT* __restrict__ v_cache,
                      const int* __restrict__ token_req, const int* __restrict__ positions, const int* __restrict__ req_slot,
                      const int* __restrict__ block_table, int table_width, int page_size, int hq, int hkv, int key_dim,
                      int value_dim, int D, int n_cols, int per_head, float temp_coef, double temp_every,
                      const float* __restrict__ v_other, int other_stride, float blend) {
    extern __shared__ __align__(16) float row[];            // n_cols floats: the token's projection with its bias
    __shared__ float scratch[64];
    pdl_trigger();
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int slot = req_slot[token_req[t]];
    pdl_wait();
    const float* src = proj + (size_t)t * row_stride;
    const int nq = hq * key_dim, nk = hkv * key_dim, k_end = k_col + nk;
    const bool whole = !per_head && (q_norm || k_norm);
    // the norms' weights join the row as it comes in, unless the values are the keys as projected
    const bool weighted = whole && v_col >= 0;
    // runs of four columns that lie in one projection (and one head) each
    const bool wide = !((row_stride | k_col | k_end | n_cols | key_dim | value_dim) & 3) && v_col >= 0 && !(v_col & 3) && !bias && !per_head
                      && !(reinterpret_cast<uintptr_t>(proj) & 15)
                      && !((reinterpret_cast<uintptr_t>(q_norm) | reinterpret_cast<uintptr_t>(k_norm)) & 15);
    const float* other = v_other ? v_other + (size_t)t * other_stride : nullptr;
    float sq_q = 0.f, sq_k = 0.f;
    if (wide) {
        for (int i = threadIdx.x; i < n_cols / 4; i += blockDim.x) {
            const int col = 4 * i;
            float4 x = reinterpret_cast<const float4*>(src)[i];
            const float sq = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
            const float* w = nullptr;
            if (col < nq) { sq_q += sq; w = q_norm ? q_norm + col : nullptr; }
            else if (col >= k_col && col < k_end) { sq_k += sq; w = k_norm ? k_norm + (col - k_col) : nullptr; }
            if (w) {
                const float4 f = *reinterpret_cast<const float4*>(w);
                x.x *= f.x; x.y *= f.y; x.z *= f.z; x.w *= f.w;
            } else if (other && col >= v_col) {
                const float* o = other + (col - v_col);
                x.x = (1.f - blend) * x.x + blend * o[0]; x.y = (1.f - blend) * x.y + blend * o[1];
                x.z = (1.f - blend) * x.z + blend * o[2]; x.w = (1.f - blend) * x.w + blend * o[3];
            }
            reinterpret_cast<float4*>(row)[i] = x;
        }
    } else {
        for (int i = threadIdx.x; i < n_cols; i += blockDim.x) {
            float x = src[i] + (bias ? bias[i] : 0.f);
            if (i < nq) {
                sq_q += x * x;
                if (weighted && q_norm) x *= q_norm[i];
            } else if (i >= k_col && i < k_end) {
                sq_k += x * x;
                if (weighted && k_norm) x *= k_norm[i - k_col];
            } else if (other && i >= v_col) {
                x = (1.f - blend) * x + blend * other[i - v_col];
            }
            row[i] = x;
        }
    }
    float inv_q = 1.f, inv_k = 1.f;
    if (whole) {       // both sums in one pass over the block, in the fixed order of block_sum
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
        sq_q = warp_sum(sq_q);
        sq_k = warp_sum(sq_k);
        if (lane == 0) { scratch[warp] = sq_q; scratch[32 + warp] = sq_k; }
        __syncthreads();
        sq_q = warp_sum(lane < n_warps ? scratch[lane] : 0.f);
        sq_k = warp_sum(lane < n_warps ? scratch[32 + lane] : 0.f);
        if (q_norm) inv_q = 1.f / sqrtf(sq_q / (float)nq + eps);
        if (k_norm) inv_k = 1.f / sqrtf(sq_k / (float)nk + eps);
    } else {
        __syncthreads();
    }
    const float* cs = cos_t ? cos_t + (size_t)t * rot_half : nullptr;
    const float* sn = sin_t ? sin_t + (size_t)t * rot_half : nullptr;
    // a warp per head, a lane per pair of neighbouring coordinates (D is even: pairs never straddle heads)
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    const auto head_inv = [&](const float* head) {      // a head's own root mean square (the whole warp takes part)
        float sq = 0.f;
        for (int d = lane; d < key_dim; d += 32) sq += head[d] * head[d];
        return 1.f / sqrtf(warp_sum(sq) / (float)key_dim + eps);
    };
    const float temp = temp_coef != 0.f ? 1.f + temp_coef * logf((float)(floor((double)(pos + 1) / temp_every) + 1.0)) : 1.f;
    if (wide && !interleaved && !(rot_half & 3) && !((reinterpret_cast<uintptr_t>(cos_t) | reinterpret_cast<uintptr_t>(sin_t)) & 15)) {
        // four coordinates per thread, the heads of queries, keys and values one after the other
        const int per = D >> 2;
        const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int i = threadIdx.x; i < hq * per; i += blockDim.x) {
            const int h = i / per, d = 4 * (i - h * per);
            store_four(q_out + (size_t)t * hq * D + 4 * i, d < key_dim ? turned_four(row + h * key_dim, temp * inv_q, d, rot_half, cs, sn) : zero);
        }
        if (!k_cache) return;
        const int page = block_table[(size_t)slot * table_width + pos / page_size];
        if (page < 0) return;                 // the host reserves a page before every write; never follow a missing entry
        for (int i = threadIdx.x; i < hkv * per; i += blockDim.x) {
            const int g = i / per, d = 4 * (i - g * per);
            const size_t dst = (((size_t)page * hkv + g) * page_size + pos % page_size) * D + d;
            store_four(k_cache + dst, d < key_dim ? turned_four(row + k_col + g * key_dim, inv_k, d, rot_half, cs, sn) : zero);
            store_four(v_cache + dst, d < value_dim ? *reinterpret_cast<const float4*>(row + v_col + g * value_dim + d) : zero);
        }
        return;
    }
    for (int h = warp; h < hq; h += n_warps) {
        const float inv = temp * (q_norm && per_head ? head_inv(row + h * key_dim) : inv_q);
        const float* w = q_norm && !weighted ? q_norm + (per_head ? 0 : h * key_dim) : nullptr;
        for (int d = 2 * lane; d < D; d += 64)
            store_pair(q_out + ((size_t)t * hq + h) * D + d, turned_pair(row + h * key_dim, w, inv, d, key_dim, rot_half, interleaved, cs, sn));
    }
    if (!k_cache) return;
    const int page = block_table[(size_t)slot * table_width + pos / page_size];
    if (page < 0) return;                     // the host reserves a page before every write; never follow a missing entry
    const int off = pos % page_size;
    for (int g = warp; g < hkv; g += n_warps) {
        const float inv = k_norm && per_head ? head_inv(row + k_col + g * key_dim) : inv_k;
        const float* w = k_norm && !weighted ? k_norm + (per_head ? 0 : g * key_dim) : nullptr;
        for (int d = 2 * lane; d < D; d += 64) {
            const float* vs = v_col >= 0 ? row + v_col + g * value_dim : row + k_col + g * key_dim;
            const size_t dst = (((size_t)page * hkv + g) * page_size + off) * D + d;
            store_pair(k_cache + dst, turned_pair(row + k_col + g * key_dim, w, inv, d, key_dim, rot_half, interleaved, cs, sn));
            store_pair(v_cache + dst, make_float2(d < value_dim ? vs[d] : 0.f, d + 1 < value_dim ? vs[d + 1] : 0.f));
        }
    }
}

// out[t][c] += bias[c]
__global__ void bias_add_kernel(float* __restrict__ out, const float* __restrict__ bias, int cols, size_t total) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) out[i] += bias[i % cols];
}
}  // namespace

CISR_EXPORT int cisr_attention_rows(const float* proj, int row_stride, int k_col, int v_col, const float* bias, const float* q_norm,
                                    const float* k_norm, float eps, const float* cos_t, const float* sin_t, int rot_half,
                                    int interleaved, void* q_out, int q_dtype, void* k_cache, void* v_cache, int cache_dtype,
                                    const int* token_req, const int* positions, const int* req_slot, const int* block_table,
                                    int table_width, int page_size, int hq, int hkv, int key_dim, int value_dim, int D, int tokens,
                                    int per_head, float temp_coef, double temp_every, const float* v_other, int other_stride, float blend,
                                    void* stream) {
    if (tokens <= 0) return 0;
    if (2 * rot_half > key_dim || rot_half < 0 || key_dim > D || value_dim > D || hq <= 0 || hkv <= 0) return -2;
    if (v_col < 0 && (value_dim != key_dim || v_other)) return -2;
    if (rot_half && (!cos_t || !sin_t)) return -2;
    if (temp_coef != 0.f && !(temp_every > 0.0)) return -2;
    const int n_cols = v_col >= 0 ? v_col + hkv * value_dim : k_col + hkv * key_dim;
    if (n_cols > row_stride) return -2;
    const size_t smem = sizeof(float) * (size_t)n_cols;
    if (smem > 200 * 1024) return -3;
    cudaStream_t s = (cudaStream_t)stream;
#define CISR_ROWS(QT, CT)                                                                                                 \
    do {                                                                                                                  \
        static size_t configured = 48 * 1024;                                                                             \
        if (smem > configured) {                                                                                          \
            cudaError_t e = cudaFuncSetAttribute(attention_rows_kernel<QT, CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (e != cudaSuccess) return (int)e;                                                                          \
            configured = smem;                                                                                            \
        }                                                                                                                 \
        /* few tokens (a decode step): a token's row on four times the threads */                                        \
        const int threads = (tokens <= 64 && n_cols >= 1024) ? 1024 : 256;                                                \
        return launch_kernel(attention_rows_kernel<QT, CT>, dim3(tokens), dim3(threads), smem, s, g_pdl, proj, row_stride, k_col, v_col, bias, \
                             q_norm, k_norm, eps, cos_t, sin_t, rot_half, interleaved, (QT*)q_out, (CT*)k_cache, (CT*)v_cache,   \
                             token_req, positions, req_slot, block_table, table_width, page_size, hq, hkv, key_dim, value_dim, D, n_cols,     \
                             per_head, temp_coef, temp_every, v_other, other_stride, blend);                                                                                  \
    } while (0)
    if (q_dtype == CISR_BF16 && cache_dtype == CISR_BF16) CISR_ROWS(__nv_bfloat16, __nv_bfloat16);
    if (q_dtype == CISR_F32 && cache_dtype == CISR_F32) CISR_ROWS(float, float);
    return -2;
#undef CISR_ROWS
}

CISR_EXPORT int cisr_bias_add(float* out, const float* bias, int rows, int cols, void* stream) {
    const size_t total = (size_t)rows * cols;
    if (!total) return 0;
    bias_add_kernel<<<(unsigned)((total + 255) / 256), 256, 0, (cudaStream_t)stream>>>(out, bias, cols, total);
    return launch_status();
}
