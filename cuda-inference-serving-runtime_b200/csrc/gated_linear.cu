// A linear recurrence with a matrix state per head, a decay and a gain per head and token, and (optionally) a normaliser:
//
//   per head h (its keys and queries are group h / (heads / groups)):
//     S <- exp(la) S + g k v^T        S [N, dv]
//     n <- exp(la) n + g k            n [N]                 (NORM)
//     y  = S^T q * q_scale,   yn = n . q * q_scale          (NORM)
//
// la (never above zero) and g are float [tokens, heads], made by a kernel before this one; q, k and v are float columns of
// token rows.  The state-space mixer runs with la = -exp(A_log) dt, g = dt, k = B, q = C, v = x; the matrix memory with
// exponential gates runs with la = f + m_before - m, g = exp(i - m) and the normaliser.  A request's state is one float row
// of a state tensor: [heads][N][dv], then (NORM) [heads][N], then whatever its mixer keeps besides.
//
// Two forms of the same recurrence, which differ by rounding only:
//   walk    single tokens and short portions, token after token.  A CTA owns 16 column units of one head (a unit is four
//           neighbouring value columns, or one where dv is not a multiple of four); its 256 threads are 16 units x 16 row groups, each
//           holding its rows' share of the columns in registers, all loads of the state in flight at once.  Tokens come
//           through shared memory in blocks of eight; the read-outs of a block are summed over the row groups together.
//   chunks  portions of CHUNK tokens and more, CHUNK at a time.  With L_t the sum of la up to token t of a chunk of n
//           tokens and S0 the state before it:
//               y_t = exp(L_t) S0^T q_t + sum_{i <= t} exp(L_t - L_i) g_i (q_t . k_i) v_i
//               S   = exp(L_n) S0 + sum_i exp(L_n - L_i) g_i k_i v_i^T
//           gains   the last sum of S, for every chunk at once, into a scratch block per (chunk, head); in further CTAs of the
//                   same launch the scores q_t . k_i per (chunk, group), which every head of a group reads
//           scan    walks a request's chunks element by element: a block receives the state BEFORE its chunk
//           reads   the read-outs of every chunk at once: one running product over [q exp(L) | scores with their decays] and [S0 ; v]
//           Each is a 64 x 64 tile per CTA of 128 threads with 8 x 4 results per thread, float on the CUDA cores.
// The sums L are kept in double: their differences are what counts, and behind a run of strong decays a float sum would
// have lost the digits of the weak ones.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_gated_set_pdl(int on) { g_pdl = on != 0; }

constexpr int CHUNK = 64;
constexpr int MAX_ROWS = 512;        // largest N: 16 row groups of at most 32 rows
CISR_EXPORT int cisr_gated_chunk_tokens() { return CHUNK; }
CISR_EXPORT int cisr_gated_max_key_dim() { return MAX_ROWS; }

namespace {
struct Args {
    const float* q; const float* k; const float* v;      // at their first column; rows of `*_stride` floats
    int q_stride, k_stride, v_stride;
    const float* la; const float* g;                     // [tokens][heads]
    float* state; long long state_stride;
    const int* req_slot; const int* q_start; const int* q_len;
    const int* chunk_req; const int* chunk_t0; const int* req_chunk0;
    float* scores;                                       // [chunks][groups][CHUNK][CHUNK]
    float* blocks;                                       // [chunks][heads][N * dv (+ N)]
    float* chunk_decay;                                  // [chunks][heads]
    float* y; float* yn;                                 // [tokens][heads][dv], [tokens][heads]
    float q_scale;
    int heads, groups, N, dv, least;
};

// ------------------------------------------------------------------ token by token
constexpr int TB = 8;                // tokens staged together

template <int ROWS, int VEC, bool NORM>
__global__ void __launch_bounds__(256)
gated_walk_kernel(const Args a) {
    extern __shared__ __align__(16) float smem[];
    constexpr int NP = 16 * ROWS, UNITS = 16, COLS = UNITS * VEC;
    float* sk = smem;                        // [TB][NP]
    float* sq = sk + TB * NP;                // [TB][NP]
    float* sv = sq + TB * NP;                // [TB][COLS]
    float* sd = sv + TB * COLS;              // [TB] exp(la)
    float* sg = sd + TB;                     // [TB]
    float* red = sg + TB;                    // [8 warps][TB][COLS]
    float* redn = red + 8 * TB * COLS;       // [8 warps][TB]   (NORM)
    pdl_trigger();
    const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS, tid = threadIdx.x;
    const int unit = tid & 15, rg = tid >> 4, warp = tid >> 5, lane = tid & 31;
    const int n_tok = a.q_len[r], first = a.q_start[r];
    const int grp = h / (a.heads / a.groups);
    const int col = c0 + unit * VEC;
    const bool live = col < a.dv;            // VEC 4: dv is a multiple of four, a unit is whole or beyond the head
    float* row = a.state + (size_t)a.req_slot[r] * a.state_stride;
    float* S = row + (size_t)h * a.N * a.dv;
    float* nv = row + (size_t)a.heads * a.N * a.dv + (size_t)h * a.N;
    const bool mine = n_tok > 0 && !(a.least > 0 && n_tok >= a.least);
    float s[ROWS][VEC], nn[NORM ? ROWS : 1];
    if (mine) {                              // the state comes from no kernel of this step: it is asked for before the wait
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
            const int n = rg + 16 * j;
#pragma unroll
            for (int e = 0; e < VEC; ++e) s[j][e] = 0.f;
            if (n < a.N && live) {
                if (VEC == 4) {
                    const float4 x = *reinterpret_cast<const float4*>(S + (size_t)n * a.dv + col);
                    s[j][0] = x.x; s[j][1 % VEC] = x.y; s[j][2 % VEC] = x.z; s[j][3 % VEC] = x.w;
                } else s[j][0] = S[(size_t)n * a.dv + col];
            }
            // the normaliser is the first column tile's: the other CTAs of the head carry zeros and write none of it
            if (NORM) nn[NORM ? j : 0] = (n < a.N && blockIdx.z == 0) ? nv[n] : 0.f;
        }
    }
    pdl_wait();
    if (!mine) return;
    for (int t0 = 0; t0 < n_tok; t0 += TB) {
        const int count = min(TB, n_tok - t0);
        for (int i = tid; i < count * NP; i += 256) {
            const int t = i / NP, n = i - t * NP;
            const size_t tok = (size_t)(first + t0 + t);
            sk[i] = n < a.N ? a.k[tok * a.k_stride + grp * a.N + n] : 0.f;
            sq[i] = n < a.N ? a.q[tok * a.q_stride + grp * a.N + n] * a.q_scale : 0.f;
        }
        for (int i = tid; i < count * COLS; i += 256) {
            const int t = i / COLS, c = c0 + i - t * COLS;
            sv[i] = c < a.dv ? a.v[(size_t)(first + t0 + t) * a.v_stride + h * a.dv + c] : 0.f;
        }
        if (tid < count) {
            const size_t at = (size_t)(first + t0 + tid) * a.heads + h;
            sd[tid] = expf(a.la[at]);
            sg[tid] = a.g[at];
        }
        __syncthreads();
        for (int t = 0; t < count; ++t) {
            const float dec = sd[t], gain = sg[t];
            float vv[VEC], acc[VEC], accn = 0.f;
#pragma unroll
            for (int e = 0; e < VEC; ++e) { vv[e] = gain * sv[t * COLS + unit * VEC + e]; acc[e] = 0.f; }
#pragma unroll
            for (int j = 0; j < ROWS; ++j) {
                const float kk = sk[t * NP + rg + 16 * j], qq = sq[t * NP + rg + 16 * j];
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    s[j][e] = fmaf(kk, vv[e], dec * s[j][e]);
                    acc[e] = fmaf(qq, s[j][e], acc[e]);
                }
                if (NORM) {
                    nn[NORM ? j : 0] = fmaf(gain, kk, dec * nn[NORM ? j : 0]);
                    accn = fmaf(qq, nn[NORM ? j : 0], accn);
                }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 16);      // the warp's two row groups
            if (NORM) accn += __shfl_xor_sync(0xffffffffu, accn, 16);
            if (lane < 16) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) red[(warp * TB + t) * COLS + unit * VEC + e] = acc[e];
                if (NORM && unit == 0) redn[warp * TB + t] = accn;
            }
        }
        __syncthreads();
        for (int i = tid; i < count * COLS; i += 256) {
            const int t = i / COLS, c = i - t * COLS;
            if (c0 + c >= a.dv) continue;
            float out = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) out += red[(w * TB + t) * COLS + c];
            a.y[((size_t)(first + t0 + t) * a.heads + h) * a.dv + c0 + c] = out;
        }
        if (NORM && blockIdx.z == 0 && tid < count) {
            float out = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) out += redn[w * TB + tid];
            a.yn[(size_t)(first + t0 + tid) * a.heads + h] = out;
        }
    }
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = rg + 16 * j;
        if (n < a.N && live) {
            if (VEC == 4) *reinterpret_cast<float4*>(S + (size_t)n * a.dv + col) = make_float4(s[j][0], s[j][1 % VEC], s[j][2 % VEC], s[j][3 % VEC]);
            else S[(size_t)n * a.dv + col] = s[j][0];
        }
    }
    if (NORM && blockIdx.z == 0 && unit == 0) {
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
            const int n = rg + 16 * j;
            if (n < a.N) nv[n] = nn[NORM ? j : 0];
        }
    }
}

// ------------------------------------------------------------------ chunk by chunk
constexpr int LDT = CHUNK + 4;       // row stride of a 64 x 64 tile in shared memory: 16-byte rows, eight neighbouring rows in different banks
constexpr int THREADS = 128;

// rows [0, nr) x columns [0, nc) of src (row stride `stride`) into dst [64][LDT], zeros elsewhere
template <bool VEC>
__device__ __forceinline__ void stage(float* dst, const float* __restrict__ src, size_t stride, int nr, int nc) {
    if (VEC) {
        float4 raw[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = threadIdx.x + u * THREADS, r = i >> 4, c = (i & 15) * 4;
            raw[u] = (r < nr && c < nc) ? *reinterpret_cast<const float4*>(src + (size_t)r * stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
            const int i = threadIdx.x + u * THREADS, r = i >> 4, c = (i & 15) * 4;
            *reinterpret_cast<float4*>(dst + r * LDT + c) = raw[u];
        }
    } else {
#pragma unroll 8
        for (int i = threadIdx.x; i < CHUNK * CHUNK; i += THREADS) {
            const int r = i >> 6, c = i & 63;
            dst[r * LDT + c] = (r < nr && c < nc) ? src[(size_t)r * stride + c] : 0.f;
        }
    }
}

// Sums of la up to each token of the chunk (double), by the first warp: lane l owns tokens 2 l and 2 l + 1.  Tokens beyond
// the portion add nothing.  `gain` receives g (zero beyond the portion).
__device__ __forceinline__ void stage_decays(const Args& a, int h, int token0, int n, double* L, float* gain) {
    if (threadIdx.x < 32) {
        const int t = 2 * threadIdx.x;
        const double x = t < n ? (double)a.la[(size_t)(token0 + t) * a.heads + h] : 0.0;
        const double y = t + 1 < n ? (double)a.la[(size_t)(token0 + t + 1) * a.heads + h] : 0.0;
        double sum = x + y;
#pragma unroll
        for (int off = 1; off < 32; off <<= 1) {
            const double before = __shfl_up_sync(0xffffffffu, sum, off);
            if ((int)threadIdx.x >= off) sum += before;
        }
        L[t + 1] = sum;
        L[t] = sum - y;
    } else if (threadIdx.x >= 64) {
        const int t = threadIdx.x - 64;
        gain[t] = t < n ? a.g[(size_t)(token0 + t) * a.heads + h] : 0.f;
    }
}

// q_t . k_i of one chunk and group (n tokens from row token0 on), every pair of tokens
template <bool VEC>
__device__ __forceinline__ void chunk_scores(const Args& a, int chunk, int grp, int n, size_t token0, float* Q, float* K) {
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[8][4] = {};
    for (int n0 = 0; n0 < a.N; n0 += CHUNK) {
        const int nc = min(CHUNK, a.N - n0);
        if (n0) __syncthreads();
        stage<VEC>(Q, a.q + token0 * a.q_stride + grp * a.N + n0, a.q_stride, n, nc);
        stage<VEC>(K, a.k + token0 * a.k_stride + grp * a.N + n0, a.k_stride, n, nc);
        __syncthreads();
        const int k4s = (nc + 3) >> 2;
        for (int k4 = 0; k4 < k4s; ++k4) {
            float4 k[4];
#pragma unroll
            for (int y = 0; y < 4; ++y) k[y] = *reinterpret_cast<const float4*>(K + (tx + 16 * y) * LDT + 4 * k4);
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                const float4 q = *reinterpret_cast<const float4*>(Q + (ty + 8 * x) * LDT + 4 * k4);
#pragma unroll
                for (int y = 0; y < 4; ++y) {
                    acc[x][y] = fmaf(q.x, k[y].x, acc[x][y]); acc[x][y] = fmaf(q.y, k[y].y, acc[x][y]);
                    acc[x][y] = fmaf(q.z, k[y].z, acc[x][y]); acc[x][y] = fmaf(q.w, k[y].w, acc[x][y]);
                }
            }
        }
    }
    float* out = a.scores + ((size_t)chunk * a.groups + grp) * CHUNK * CHUNK;
#pragma unroll
    for (int x = 0; x < 8; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) out[(ty + 8 * x) * CHUNK + tx + 16 * y] = acc[x][y];
}

// grid (chunk, head, tiles of [N, dv] + 1): the last z makes the scores of the chunk's groups, in the CTAs of the first heads
template <bool VEC, bool NORM>
__global__ void __launch_bounds__(THREADS, 5)
gated_gains_kernel(const Args a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ double L[CHUNK];
    __shared__ float w[CHUNK];
    float* K = smem;
    float* V = K + CHUNK * LDT;
    pdl_trigger();
    const int chunk = blockIdx.x, h = blockIdx.y, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const bool scores = blockIdx.z == gridDim.z - 1;
    const int row_tiles = (a.N + CHUNK - 1) / CHUNK;
    const int n0 = ((int)blockIdx.z % row_tiles) * CHUNK, c0 = ((int)blockIdx.z / row_tiles) * CHUNK;
    const int grp = h / (a.heads / a.groups);
    const int r = a.chunk_req[chunk], t0 = a.chunk_t0[chunk], n = min(CHUNK, a.q_len[r] - t0);
    const int token0 = a.q_start[r] + t0;
    const int nr = min(CHUNK, a.N - n0), nc = min(CHUNK, a.dv - c0);
    pdl_wait();
    if (scores) {
        if (h < a.groups) chunk_scores<VEC>(a, chunk, h, n, (size_t)token0, K, V);
        return;
    }
    stage_decays(a, h, token0, n, L, w);
    stage<VEC>(K, a.k + (size_t)token0 * a.k_stride + grp * a.N + n0, a.k_stride, n, nr);
    stage<VEC>(V, a.v + (size_t)token0 * a.v_stride + h * a.dv + c0, a.v_stride, n, nc);
    __syncthreads();
    if (threadIdx.x < CHUNK) w[threadIdx.x] *= expf((float)(L[CHUNK - 1] - L[threadIdx.x]));
    if (blockIdx.z == 0 && threadIdx.x == 0) a.chunk_decay[(size_t)chunk * a.heads + h] = expf((float)L[CHUNK - 1]);
    __syncthreads();
    float acc[2][4][4] = {};
    for (int i = 0; i < n; ++i) {
        const float wi = w[i];
        float4 v = *reinterpret_cast<const float4*>(V + i * LDT + 4 * tx);
        v.x *= wi; v.y *= wi; v.z *= wi; v.w *= wi;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const float4 k = *reinterpret_cast<const float4*>(K + i * LDT + 32 * half + 4 * ty);
            const float kv[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                acc[half][x][0] = fmaf(kv[x], v.x, acc[half][x][0]); acc[half][x][1] = fmaf(kv[x], v.y, acc[half][x][1]);
                acc[half][x][2] = fmaf(kv[x], v.z, acc[half][x][2]); acc[half][x][3] = fmaf(kv[x], v.w, acc[half][x][3]);
            }
        }
    }
    const size_t per_head = (size_t)a.N * a.dv + (NORM ? a.N : 0);
    float* out = a.blocks + ((size_t)chunk * a.heads + h) * per_head;
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int row = 32 * half + 4 * ty + x;
            if (row >= nr) continue;
            float* dst = out + (size_t)(n0 + row) * a.dv + c0 + 4 * tx;
            if (VEC) {
                if (4 * tx < nc) *reinterpret_cast<float4*>(dst) = make_float4(acc[half][x][0], acc[half][x][1], acc[half][x][2], acc[half][x][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (4 * tx + e < nc) dst[e] = acc[half][x][e];
            }
        }
    if (NORM && c0 == 0 && (int)threadIdx.x < nr) {
        float sum = 0.f;
        for (int i = 0; i < n; ++i) sum = fmaf(w[i], K[i * LDT + threadIdx.x], sum);
        out[(size_t)a.N * a.dv + n0 + threadIdx.x] = sum;
    }
}

// grid (requests, heads, elements / (256 VEC)): a thread owns VEC neighbouring elements of the head's [N * dv (+ N)] state
template <int VEC, bool NORM>
__global__ void __launch_bounds__(256)
gated_scan_kernel(const Args a) {
    pdl_trigger();
    const int r = blockIdx.x, h = blockIdx.y, e = (blockIdx.z * 256 + threadIdx.x) * VEC;
    const int matrix = a.N * a.dv, per_head = matrix + (NORM ? a.N : 0);
    const int n_all = a.q_len[r];
    pdl_wait();
    if (n_all < a.least || e >= per_head) return;
    float* row = a.state + (size_t)a.req_slot[r] * a.state_stride;
    float* kept = e < matrix ? row + (size_t)h * matrix + e : row + (size_t)a.heads * matrix + (size_t)h * a.N + (e - matrix);
    float S[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) S[j] = kept[j];
    const int chunk0 = a.req_chunk0[r], chunks = (n_all + CHUNK - 1) / CHUNK;
    const size_t step = (size_t)a.heads * per_head;
    float* block = a.blocks + ((size_t)chunk0 * a.heads + h) * per_head + e;
    const float* decay = a.chunk_decay + (size_t)chunk0 * a.heads + h;
    // the walk itself is one multiply-add per chunk: it goes as fast as the gains arrive, so AHEAD of them are asked for
    // together, and the next ones before the ones at hand are used
    constexpr int AHEAD = 8;
    float gain[AHEAD][VEC], f[AHEAD];
    const auto fetch = [&](int c0) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const bool in = c0 + u < chunks;
            f[u] = in ? decay[(size_t)(c0 + u) * a.heads] : 0.f;
            if (VEC == 2) {
                const float2 x = in ? *reinterpret_cast<const float2*>(block + (size_t)(c0 + u) * step) : make_float2(0.f, 0.f);
                gain[u][0] = x.x; gain[u][1 % VEC] = x.y;
            } else gain[u][0] = in ? block[(size_t)(c0 + u) * step] : 0.f;
        }
    };
    fetch(0);
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float now[AHEAD][VEC], fn[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            fn[u] = f[u];
#pragma unroll
            for (int j = 0; j < VEC; ++j) now[u][j] = gain[u][j];
        }
        if (c0 + AHEAD < chunks) fetch(c0 + AHEAD);
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (c0 + u < chunks) {
                float* at = block + (size_t)(c0 + u) * step;
                if (VEC == 2) *reinterpret_cast<float2*>(at) = make_float2(S[0], S[1 % VEC]);
                else at[0] = S[0];
#pragma unroll
                for (int j = 0; j < VEC; ++j) S[j] = fmaf(fn[u], S[j], now[u][j]);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) kept[j] = S[j];
}

// acc[x][y] += sum_k A[ty + 8 x][k] B[k][4 tx + y] over the first 4 * k4s rows of B
__device__ __forceinline__ void tile_product(const float* A, const float* B, int tx, int ty, int k4s, float (&acc)[8][4]) {
    for (int k4 = 0; k4 < k4s; ++k4) {
        float4 b[4];
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) b[kk] = *reinterpret_cast<const float4*>(B + (4 * k4 + kk) * LDT + 4 * tx);
#pragma unroll
        for (int x = 0; x < 8; ++x) {
            const float4 av = *reinterpret_cast<const float4*>(A + (ty + 8 * x) * LDT + 4 * k4);
            const float f[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                acc[x][0] = fmaf(f[kk], b[kk].x, acc[x][0]); acc[x][1] = fmaf(f[kk], b[kk].y, acc[x][1]);
                acc[x][2] = fmaf(f[kk], b[kk].z, acc[x][2]); acc[x][3] = fmaf(f[kk], b[kk].w, acc[x][3]);
            }
        }
    }
}

template <bool VEC, bool NORM>
__global__ void __launch_bounds__(THREADS, 5)
gated_reads_kernel(const Args a) {
    extern __shared__ __align__(16) float smem[];
    __shared__ double L[CHUNK];
    __shared__ float gain[CHUNK], carried[CHUNK], nvec[CHUNK];
    float* A = smem;
    float* B = A + CHUNK * LDT;
    pdl_trigger();
    const int chunk = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CHUNK, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int grp = h / (a.heads / a.groups);
    const int r = a.chunk_req[chunk], t0 = a.chunk_t0[chunk], n = min(CHUNK, a.q_len[r] - t0);
    const int token0 = a.q_start[r] + t0, nc = min(CHUNK, a.dv - c0);
    const size_t per_head = (size_t)a.N * a.dv + (NORM ? a.N : 0);
    const float* block = a.blocks + ((size_t)chunk * a.heads + h) * per_head;
    const bool norm_here = NORM && c0 == 0;
    const int nt = tid >> 1, nhalf = (tid & 1) * 32;          // normaliser: two threads per token, half a row each
    float norm = 0.f;
    pdl_wait();
    stage_decays(a, h, token0, n, L, gain);
    float acc[8][4] = {};
    for (int n0 = 0; n0 < a.N; n0 += CHUNK) {
        const int nr = min(CHUNK, a.N - n0);
        if (n0) __syncthreads();
        stage<VEC>(A, a.q + (size_t)token0 * a.q_stride + grp * a.N + n0, a.q_stride, n, nr);
        stage<VEC>(B, block + (size_t)n0 * a.dv + c0, a.dv, nr, nc);
        if (norm_here && tid < CHUNK) nvec[tid] = tid < nr ? block[(size_t)a.N * a.dv + n0 + tid] : 0.f;
        __syncthreads();
        tile_product(A, B, tx, ty, (nr + 3) >> 2, acc);
        if (norm_here)
            for (int i = 0; i < 32; ++i) norm = fmaf(A[nt * LDT + nhalf + i], nvec[nhalf + i], norm);
    }
    if (tid < CHUNK) carried[tid] = expf((float)L[tid]);
    __syncthreads();
#pragma unroll
    for (int x = 0; x < 8; ++x) {
        const float f = carried[ty + 8 * x];
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] *= f;
    }
    norm *= carried[nt];
    stage<VEC>(B, a.v + (size_t)token0 * a.v_stride + h * a.dv + c0, a.v_stride, n, nc);
    const float* G = a.scores + ((size_t)chunk * a.groups + grp) * CHUNK * CHUNK;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
        const int i4 = tid + u * THREADS, t = i4 >> 4, i = (i4 & 15) * 4;
        const float4 raw = *reinterpret_cast<const float4*>(G + t * CHUNK + i);
        const float sc[4] = {raw.x, raw.y, raw.z, raw.w};
        float p[4];
        const double Lt = L[t];
#pragma unroll
        for (int e = 0; e < 4; ++e) p[e] = i + e <= t ? sc[e] * gain[i + e] * expf((float)(Lt - L[i + e])) : 0.f;
        *reinterpret_cast<float4*>(A + t * LDT + i) = make_float4(p[0], p[1], p[2], p[3]);
    }
    __syncthreads();
    tile_product(A, B, tx, ty, CHUNK / 4, acc);
    if (norm_here) {
        for (int i = 0; i < 32; ++i) norm += A[nt * LDT + nhalf + i];
        norm += __shfl_xor_sync(0xffffffffu, norm, 1);
        if (nhalf == 0 && nt < n) a.yn[(size_t)(token0 + nt) * a.heads + h] = norm * a.q_scale;
    }
#pragma unroll
    for (int x = 0; x < 8; ++x) {
        const int t = ty + 8 * x;
        if (t >= n) continue;
        float* dst = a.y + ((size_t)(token0 + t) * a.heads + h) * a.dv + c0 + 4 * tx;
        if (VEC) {
            if (4 * tx < nc) *reinterpret_cast<float4*>(dst) = make_float4(acc[x][0] * a.q_scale, acc[x][1] * a.q_scale, acc[x][2] * a.q_scale, acc[x][3] * a.q_scale);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (4 * tx + e < nc) dst[e] = acc[x][e] * a.q_scale;
        }
    }
}

template <int ROWS, int VEC, bool NORM>
int launch_walk(const Args& a, int n_req, cudaStream_t s) {
    constexpr int NP = 16 * ROWS, COLS = 16 * VEC;
    const size_t smem = sizeof(float) * ((size_t)TB * (2 * NP + COLS + 2) + 8 * TB * COLS + 8 * TB);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(gated_walk_kernel<ROWS, VEC, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    return launch_kernel(gated_walk_kernel<ROWS, VEC, NORM>, dim3(n_req, a.heads, (a.dv + COLS - 1) / COLS), dim3(256), smem, s, g_pdl, a);
}
template <int VEC, bool NORM>
int walk(const Args& a, int n_req, cudaStream_t s) {
    if (a.N <= 64) return launch_walk<4, VEC, NORM>(a, n_req, s);
    if (a.N <= 128) return launch_walk<8, VEC, NORM>(a, n_req, s);
    if (a.N <= 256) return launch_walk<16, VEC, NORM>(a, n_req, s);
    return launch_walk<32, VEC, NORM>(a, n_req, s);
}

template <bool VEC, bool NORM>
int chunks(const Args& a, int n_req, int n_chunks, cudaStream_t s) {
    const size_t smem = sizeof(float) * 2 * CHUNK * LDT;       // 34 KB: within the default limit
    const int row_tiles = (a.N + CHUNK - 1) / CHUNK, col_tiles = (a.dv + CHUNK - 1) / CHUNK;
    static bool configured = false;
    if (!configured) {       // five CTAs per SM want more shared memory than the default split gives
        cudaError_t e = cudaFuncSetAttribute(gated_gains_kernel<VEC, NORM>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(gated_reads_kernel<VEC, NORM>, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    int st = launch_kernel(gated_gains_kernel<VEC, NORM>, dim3(n_chunks, a.heads, row_tiles * col_tiles + 1), dim3(THREADS), smem, s, g_pdl, a);
    if (st) return st;
    const int elements = a.N * a.dv + (NORM ? a.N : 0);
    // two elements per thread where every block and every state row begins on 8 bytes and no pair straddles matrix and normaliser
    const bool pairs = VEC && a.state_stride % 2 == 0 && !((uintptr_t)a.state & 7);
    if (pairs) st = launch_kernel(gated_scan_kernel<2, NORM>, dim3(n_req, a.heads, (elements / 2 + 255) / 256), dim3(256), 0, s, g_pdl, a);
    else st = launch_kernel(gated_scan_kernel<1, NORM>, dim3(n_req, a.heads, (elements + 255) / 256), dim3(256), 0, s, g_pdl, a);
    if (st) return st;
    return launch_kernel(gated_reads_kernel<VEC, NORM>, dim3(n_chunks, a.heads, col_tiles), dim3(THREADS), smem, s, g_pdl, a);
}
}  // namespace

// The recurrence for a step: the requests that bring at least `least` tokens run chunk by chunk (`n_chunks` chunks listed in
// chunk_req / chunk_t0, a request's first one in req_chunk0), the `n_short` others token by token; least <= 0: every request token by token.
// yn null: no normaliser.
CISR_EXPORT int cisr_gated_recurrence(const float* q, int q_stride, const float* k, int k_stride, const float* v, int v_stride, const float* la,
                                      const float* g, float* state, long long state_stride, const int* req_slot, const int* q_start,
                                      const int* q_len, float* y, float* yn, float q_scale, int heads, int groups, int N, int dv, int n_req,
                                      int least, int n_chunks, int n_short, const int* chunk_req, const int* chunk_t0, const int* req_chunk0,
                                      float* scores, float* blocks, float* chunk_decay, void* stream) {
    if (n_req <= 0) return 0;
    if (heads <= 0 || groups <= 0 || heads % groups || N <= 0 || N > MAX_ROWS || dv <= 0) return -2;
    Args a;
    a.q = q; a.k = k; a.v = v; a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride; a.la = la; a.g = g; a.state = state;
    a.state_stride = state_stride; a.req_slot = req_slot; a.q_start = q_start; a.q_len = q_len; a.chunk_req = chunk_req; a.chunk_t0 = chunk_t0;
    a.req_chunk0 = req_chunk0; a.scores = scores; a.blocks = blocks; a.chunk_decay = chunk_decay; a.y = y; a.yn = yn; a.q_scale = q_scale;
    a.heads = heads; a.groups = groups; a.N = N; a.dv = dv;
    cudaStream_t s = (cudaStream_t)stream;
    const bool chunked = least > 0 && n_chunks > 0;
    a.least = chunked ? least : 0;
    int st = 0;
    if (chunked) {
        if (!chunk_req || !chunk_t0 || !req_chunk0 || !scores || !blocks || !chunk_decay) return -2;
        const bool vec = N % 4 == 0 && dv % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && v_stride % 4 == 0 &&
                         !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)blocks | (uintptr_t)y) & 15);
        if (vec) st = yn ? chunks<true, true>(a, n_req, n_chunks, s) : chunks<true, false>(a, n_req, n_chunks, s);
        else st = yn ? chunks<false, true>(a, n_req, n_chunks, s) : chunks<false, false>(a, n_req, n_chunks, s);
        if (st) return st;
    }
    if (!chunked || n_short > 0) {
        const bool vec = dv % 4 == 0 && state_stride % 4 == 0 && !((uintptr_t)state & 15);
        if (vec) st = yn ? walk<4, true>(a, n_req, s) : walk<4, false>(a, n_req, s);
        else st = yn ? walk<1, true>(a, n_req, s) : walk<1, false>(a, n_req, s);
    }
    return st;
}
