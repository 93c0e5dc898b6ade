// The real-gated linear recurrence of a recurrent block: per channel c (part b = c / block of `blocks` equal parts)
//
//   r = sigmoid(R_b u_b + rb),  i = sigmoid(I_b u_b + ib)          R_b, I_b square [block, block], [out, in]
//   la = -factor * r * softplus(lam);   S <- exp(la) S + sqrt(1 - exp(2 la)) i u
//   out = S * gelu(gate + gate_bias)                                gelu in its tanh form; out: operand of the output projection
//
// u float [tokens, width] (after the short convolution), gate float columns of the input projection.  Everything here is
// float: the block products take u as float (the gates decide what a recurrence keeps for thousands of tokens), and
// 1 - exp(2 la) keeps its digits where the decay is nearly one (a power series there).
//   gates   a warp per channel, up to 16 tokens: both products of a channel with the tokens' parts (weights read once,
//           16 tokens' u in shared memory), the sums brought to one lane per token by a transposing reduction.  FUSED (a step of at
//           most 16 tokens): the recurrence and the output follow in the same kernel, tokens in order across the lanes.
//           Otherwise the sums are written: pre [blocks][rows][2 block] (a part's r sums, then its i sums), the
//           layout that the grouped tensor-core product has when that makes them.
//   scan    any portions: a cluster of 1 to 8 CTAs per (request, 32 channels), a warp per segment of 8 tokens.  Each warp
//           forms its tokens' decays and inputs and its segment's (decay, end value); the segments are chained through
//           shared memory, the CTAs' shares through one another's; then each warp walks its tokens again from the state
//           before them and writes their outputs.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_rglru_set_pdl(int on) { g_pdl = on != 0; }

namespace {
constexpr int GT_MAX = 16;           // tokens per tile of the gates kernel (eight where a step has no more)
constexpr int GATE_WARPS = 8;
constexpr int KT = 256;              // u columns staged at once

__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.f, 1.f + expf(-z)); }      // beyond z = -87 the divisor is infinite and the result 0
// A token's log decay, decay and input.  1 - exp(x), x = 2 la <= 0: for x above -1/4 the series -x (1 + x/2 (1 + x/3 (1 + ...)))
// up to x^7 (what is left out is below 2^-29 of it), else one minus the decay's square, which is at most 0.78 then.
__device__ __forceinline__ void decay_and_input(float pre_r, float pre_i, float u, float rate, float& la, float& dec, float& in) {
    la = rate * sigmoid_f(pre_r);                                  // rate = -factor softplus(lam)
    dec = expf(la);
    const float x = 2.f * la;
    float p = fmaf(x, 1.f / 7.f, 1.f);
    p = fmaf(x * p, 1.f / 6.f, 1.f);
    p = fmaf(x * p, 1.f / 5.f, 1.f);
    p = fmaf(x * p, 1.f / 4.f, 1.f);
    p = fmaf(x * p, 1.f / 3.f, 1.f);
    p = fmaf(x * p, 1.f / 2.f, 1.f);
    const float gone = x > -0.25f ? -x * p : fmaf(-dec, dec, 1.f);
    float root;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(root) : "f"(gone));       // within 2^-23 of it
    in = root * sigmoid_f(pre_i) * u;
}

__device__ __forceinline__ float4 weights4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 weights4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
}

struct GateArgs {
    const float* u; const void* w; const float* bias;              // w [blocks][2 block][block]; bias [blocks][2 block]
    float* pre; long long rows;
    int tokens, width, block;
    const float* rate; float* state; long long state_stride, s_offset;
    const int* token_req; const int* req_slot; const int* q_start; const int* q_len;
    const float* gate; int gate_stride, gate_col; const float* gate_bias; void* out; int out_stride;
};

// VEC: block is a multiple of 4 (16-byte rows of u, 8-byte groups of weights).  GT: tokens per tile
template <typename WT, typename OT, bool VEC, bool FUSED, int GT>
__global__ void __launch_bounds__(32 * GATE_WARPS)
rglru_gates_kernel(const GateArgs a) {
    __shared__ __align__(16) float us[GT][KT];
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int part = blockIdx.x, ch = blockIdx.y * GATE_WARPS + warp, t0 = blockIdx.z * GT;
    const bool live = ch < a.block;
    const int count = min(GT, a.tokens - t0), c = part * a.block + ch;
    const WT* wr = reinterpret_cast<const WT*>(a.w) + ((size_t)part * 2 * a.block + (live ? ch : 0)) * a.block;
    const WT* wi = wr + (size_t)a.block * a.block;
    float acc[2 * GT];
#pragma unroll
    for (int j = 0; j < 2 * GT; ++j) acc[j] = 0.f;
    float4 r0[KT / 128], i0[KT / 128];       // the weights come from no kernel: the first KT columns are asked for before the wait
    if (VEC) {
#pragma unroll
        for (int s = 0; s < KT / 128; ++s) {
            const int k = 4 * lane + 128 * s;
            r0[s] = k < a.block ? weights4(wr + k) : make_float4(0.f, 0.f, 0.f, 0.f);
            i0[s] = k < a.block ? weights4(wi + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    pdl_wait();
    // FUSED: lane l finishes token l; what it needs besides the sums is on its way during the products
    const bool mine = FUSED && live && lane < count;
    bool first = true, last = true;
    float* kept = nullptr;
    float S = 0.f, u_own = 0.f, y_own = 0.f, rate = 0.f;
    if (mine) {
        const int t = t0 + lane, r = a.token_req[t], q0 = a.q_start[r];
        first = t == q0;
        last = t == q0 + a.q_len[r] - 1;
        kept = a.state + (size_t)a.req_slot[r] * a.state_stride + a.s_offset + c;
        if (first) S = *kept;                                      // the state before this lane's token, where a portion begins
        u_own = a.u[(size_t)t * a.width + c];
        y_own = a.gate[(size_t)t * a.gate_stride + a.gate_col + c] + a.gate_bias[c];
        rate = a.rate[c];
    }
    for (int k0 = 0; k0 < a.block; k0 += KT) {
        const int kc = min(KT, a.block - k0);
        if (k0) __syncthreads();
        for (int i = threadIdx.x; i < GT * KT; i += 32 * GATE_WARPS) {
            const int t = i / KT, k = i - t * KT;
            us[t][k] = (t < count && k < kc) ? a.u[(size_t)(t0 + t) * a.width + part * a.block + k0 + k] : 0.f;
        }
        __syncthreads();
        if (VEC) {
#pragma unroll
            for (int s = 0; s < KT / 128; ++s) {
                const int k = 4 * lane + 128 * s;
                if (k >= kc) break;                                // kc is a multiple of 4: a group is whole or beyond
                const float4 r = k0 ? weights4(wr + k0 + k) : r0[s], i = k0 ? weights4(wi + k0 + k) : i0[s];
#pragma unroll
                for (int t = 0; t < GT; ++t) {
                    const float4 x = *reinterpret_cast<const float4*>(&us[t][k]);
                    acc[t] = fmaf(r.x, x.x, fmaf(r.y, x.y, fmaf(r.z, x.z, fmaf(r.w, x.w, acc[t]))));
                    acc[GT + t] = fmaf(i.x, x.x, fmaf(i.y, x.y, fmaf(i.z, x.z, fmaf(i.w, x.w, acc[GT + t]))));
                }
            }
        } else {
            for (int k = lane; k < kc; k += 32) {
                const float r = to_float(wr[k0 + k]), i = to_float(wi[k0 + k]);
#pragma unroll
                for (int t = 0; t < GT; ++t) { acc[t] = fmaf(r, us[t][k], acc[t]); acc[GT + t] = fmaf(i, us[t][k], acc[GT + t]); }
            }
        }
    }
    // transposing reduction: lane l ends up with the warp's sum of acc[l % (2 GT)] (r of token l below GT, i of token l - GT from GT on)
#pragma unroll
    for (int off = GT; off; off >>= 1) {
        const bool high = lane & off;
#pragma unroll
        for (int j = 0; j < off; ++j) {
            const float send = high ? acc[j] : acc[j + off], keep = high ? acc[j + off] : acc[j];
            acc[j] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
    }
    if (GT < 16) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 16);
    const float* bias = a.bias + (size_t)part * 2 * a.block + (live ? ch : 0);
    const bool is_r = !(lane & GT);
    const float sum = acc[0] + (is_r ? bias[0] : bias[a.block]);
    const int t = t0 + (lane & (GT - 1));
    if (!FUSED) {
        if (live && lane < 2 * GT && t < a.tokens) a.pre[((size_t)part * a.rows + t) * 2 * a.block + (is_r ? ch : a.block + ch)] = sum;
        return;
    }
    const float pre_i = __shfl_sync(0xffffffffu, sum, (lane + GT) & 31);
    float la = 0.f, dec = 1.f, in = 0.f;
    if (mine) decay_and_input(sum, pre_i, u_own, rate, la, dec, in);
    for (int j = 0; j < count; ++j) {                              // tokens in order; lane j takes lane j - 1's state unless its portion begins
        const float before = __shfl_sync(0xffffffffu, S, j ? j - 1 : 0);
        if (lane == j) S = fmaf(dec, first ? S : before, in);
    }
    if (mine) {
        if (last) *kept = S;
        reinterpret_cast<OT*>(a.out)[(size_t)t * a.out_stride + c] = from_float<OT>(S * gelu_tanh(y_own));
    }
}

// ------------------------------------------------------------------ scan
constexpr int SEG = 8;               // tokens per segment (one warp's share of a round)
constexpr int SCAN_SEGS = 8;         // most segments per CTA
constexpr int MAX_CLUSTER = 8;       // most CTAs that share a request's tokens

struct ScanArgs {
    const float* pre; long long rows; const float* bias;           // bias null: pre holds it already
    const float* u; int width, block;
    const float* rate; float* state; long long state_stride, s_offset;
    const int* req_slot; const int* q_start; const int* q_len;
    const float* gate; int gate_stride, gate_col; const float* gate_bias; void* out; int out_stride;
    int cluster;
};

// a float of another CTA's shared memory: the address of `mine` as CTA `rank` of the cluster has it
__device__ __forceinline__ void store_to_cta(float* mine, int rank, float v) {
    uint32_t remote;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"((uint32_t)__cvta_generic_to_shared(mine)), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
}

// grid (requests, channels / 32, cluster): the CTAs of a cluster share a request's tokens.  In a round a cluster takes
// cluster * segs * SEG neighbouring tokens; one more warp per CTA chains.  A segment, a CTA's share and a round are each a map S -> decay S + end; the
// CTAs write theirs into one another's shared memory, so one cluster barrier per round chains them.
template <typename OT>
__global__ void __launch_bounds__(32 * (SCAN_SEGS + 1), 2)
rglru_scan_kernel(const ScanArgs a) {
    __shared__ float seg_decay[2][SCAN_SEGS][32], seg_end[2][SCAN_SEGS][32];
    __shared__ float cta_decay[2][MAX_CLUSTER][32], cta_end[2][MAX_CLUSTER][32];
    pdl_trigger();
    const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5, segs = (blockDim.x >> 5) - 1, rank = blockIdx.z;
    const int r = blockIdx.x, c = blockIdx.y * 32 + lane;
    const bool live = c < a.width;
    const int n = a.q_len[r];
    const size_t first = (size_t)a.q_start[r];
    pdl_wait();
    if (n <= 0) return;                                            // the whole cluster alike
    const int part = live ? c / a.block : 0, ch = c - part * a.block;
    float* kept = a.state + (size_t)a.req_slot[r] * a.state_stride + a.s_offset + c;
    float S0 = 0.f, rate = 0.f, gate_bias = 0.f, rb = 0.f, ib = 0.f;
    if (live) {
        S0 = *kept; rate = a.rate[c]; gate_bias = a.gate_bias[c];
        if (a.bias) { rb = a.bias[(size_t)part * 2 * a.block + ch]; ib = a.bias[(size_t)part * 2 * a.block + a.block + ch]; }
    }
    const float* pre = a.pre + ((size_t)part * a.rows + first) * 2 * a.block + ch;
    const float* u = a.u + first * a.width + c;
    const float* gate = a.gate + first * a.gate_stride + a.gate_col + c;
    OT* out = reinterpret_cast<OT*>(a.out) + first * a.out_stride + c;
    const size_t pre_stride = (size_t)2 * a.block;
    const int share = segs * SEG, round = a.cluster * share;
    float nr[SEG], ni[SEG], nu[SEG];
    const auto fetch = [&](int t0) {
#pragma unroll
        for (int j = 0; j < SEG; ++j) {
            const int t = t0 + j;
            const bool in = live && t < n;
            nr[j] = in ? pre[(size_t)t * pre_stride] : 0.f;
            ni[j] = in ? pre[(size_t)t * pre_stride + a.block] : 0.f;
            nu[j] = in ? u[(size_t)t * a.width] : 0.f;
        }
    };
    if (a.cluster > 1) asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    const bool chains = seg == segs;                               // the last warp has no tokens
    if (!chains) fetch(rank * share + seg * SEG);
    if (a.cluster > 1) asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");      // every CTA of the cluster runs: its shared memory may be written
    for (int base = 0, turn = 0; base < n; base += round, turn ^= 1) {
        const int t0 = base + rank * share + seg * SEG;
        float dec[SEG], in[SEG], y[SEG], sum = 0.f, end = 0.f;
        if (!chains) {
#pragma unroll
            for (int j = 0; j < SEG; ++j) {
                float la;
                decay_and_input(nr[j] + rb, ni[j] + ib, nu[j], rate, la, dec[j], in[j]);      // u is zero beyond the portion, and so is the input
                const bool inside = t0 + j < n;
                y[j] = (live && inside) ? gate[(size_t)(t0 + j) * a.gate_stride] : 0.f;      // on its way during the chaining
                if (!inside) { la = 0.f; dec[j] = 1.f; }           // the state passes as it is
                sum += la;
                end = fmaf(dec[j], end, in[j]);
            }
            if (base + round < n) fetch(t0 + round);               // the next round's operands are on their way during the chaining
            seg_decay[turn][seg][lane] = expf(sum);
            seg_end[turn][seg][lane] = end;
        }
        __syncthreads();
        // the segments before this one as one map (for the chaining warp: the CTA's whole share)
        float A = 1.f, E = 0.f;
        for (int s = 0; s < seg; ++s) {
            const float d = seg_decay[turn][s][lane];
            E = fmaf(d, E, seg_end[turn][s][lane]);
            A *= d;
        }
        float before = S0;
        if (a.cluster > 1) {
            // Only the chaining warp has something to release; the others' loads and stores in flight need not be waited for.
            if (chains) {
                for (int k = 0; k < a.cluster; ++k) {
                    store_to_cta(&cta_decay[turn][rank][lane], k, A);
                    store_to_cta(&cta_end[turn][rank][lane], k, E);
                }
                asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
            } else {
                asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");
            }
            asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
            float S = S0;
            for (int k = 0; k < a.cluster; ++k) {
                if (k == rank) before = S;
                S = fmaf(cta_decay[turn][k][lane], S, cta_end[turn][k][lane]);
            }
            S0 = S;                                                // every warp knows the state behind the round
        } else {
            float S = S0;
            for (int s = 0; s < segs; ++s) S = fmaf(seg_decay[turn][s][lane], S, seg_end[turn][s][lane]);
            S0 = S;
        }
        if (chains) continue;
        float S = fmaf(A, before, E);
#pragma unroll
        for (int j = 0; j < SEG; ++j) {
            S = fmaf(dec[j], S, in[j]);
            const float o = S * gelu_tanh(y[j] + gate_bias);
            if (live && t0 + j < n) out[(size_t)(t0 + j) * a.out_stride] = from_float<OT>(o);
        }
    }
    if (live && chains && rank == 0) *kept = S0;
}
}  // namespace

CISR_EXPORT int cisr_rglru_fused_tokens() { return GT_MAX; }

// pre null: the whole block for a step of at most 16 tokens; else only the gates' sums (any number of tokens).
CISR_EXPORT int cisr_rglru_gates(const float* u, const void* w, int w_dtype, const float* bias, float* pre, long long rows, int tokens, int width,
                                 int block, const float* rate, float* state, long long state_stride, long long s_offset,
                                 const int* token_req, const int* req_slot, const int* q_start, const int* q_len, const float* gate,
                                 int gate_stride, int gate_col, const float* gate_bias, void* out, int out_dtype, int out_stride, void* stream) {
    if (tokens <= 0) return 0;
    if (width <= 0 || block <= 0 || width % block || (!pre && tokens > GT_MAX) || (pre && rows < tokens)) return -2;
    GateArgs a;
    a.u = u; a.w = w; a.bias = bias; a.pre = pre; a.rows = rows; a.tokens = tokens; a.width = width; a.block = block; a.rate = rate; a.state = state;
    a.state_stride = state_stride; a.s_offset = s_offset; a.token_req = token_req; a.req_slot = req_slot; a.q_start = q_start; a.q_len = q_len;
    a.gate = gate; a.gate_stride = gate_stride; a.gate_col = gate_col; a.gate_bias = gate_bias; a.out = out; a.out_stride = out_stride;
    const dim3 grid(width / block, (block + GATE_WARPS - 1) / GATE_WARPS, (tokens + GT_MAX - 1) / GT_MAX), threads(32 * GATE_WARPS);
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = block % 4 == 0 && !((uintptr_t)w & 15);
#define CISR_GATES(WT, OT)                                                                                              \
    do {                                                                                                                \
        if (pre) return vec ? launch_kernel(rglru_gates_kernel<WT, OT, true, false, 16>, grid, threads, 0, s, g_pdl, a) \
                            : launch_kernel(rglru_gates_kernel<WT, OT, false, false, 16>, grid, threads, 0, s, g_pdl, a); \
        if (tokens <= 8) return vec ? launch_kernel(rglru_gates_kernel<WT, OT, true, true, 8>, grid, threads, 0, s, g_pdl, a) \
                                    : launch_kernel(rglru_gates_kernel<WT, OT, false, true, 8>, grid, threads, 0, s, g_pdl, a); \
        return vec ? launch_kernel(rglru_gates_kernel<WT, OT, true, true, 16>, grid, threads, 0, s, g_pdl, a)           \
                   : launch_kernel(rglru_gates_kernel<WT, OT, false, true, 16>, grid, threads, 0, s, g_pdl, a);         \
    } while (0)
    if (w_dtype == CISR_BF16) CISR_GATES(__nv_bfloat16, __nv_bfloat16);
    CISR_GATES(float, float);
#undef CISR_GATES
}

// `longest`: a bound on the portions of the step (the number of segments a CTA is launched with; any value is right).
CISR_EXPORT int cisr_rglru_scan(const float* pre, long long rows, const float* bias, const float* u, int width, int block, const float* rate,
                                float* state, long long state_stride, long long s_offset, const int* req_slot, const int* q_start,
                                const int* q_len, const float* gate, int gate_stride, int gate_col, const float* gate_bias, void* out,
                                int out_dtype, int out_stride, int n_req, int longest, void* stream) {
    if (n_req <= 0) return 0;
    if (width <= 0 || block <= 0 || width % block) return -2;
    ScanArgs a;
    a.pre = pre; a.rows = rows; a.bias = bias; a.u = u; a.width = width; a.block = block; a.rate = rate; a.state = state; a.state_stride = state_stride;
    a.s_offset = s_offset; a.req_slot = req_slot; a.q_start = q_start; a.q_len = q_len; a.gate = gate; a.gate_stride = gate_stride;
    a.gate_col = gate_col; a.gate_bias = gate_bias; a.out = out; a.out_stride = out_stride;
    int segs = (longest + SEG - 1) / SEG;
    segs = segs < 1 ? 1 : segs > SCAN_SEGS ? SCAN_SEGS : segs;
    // long portions: as many CTAs of a cluster as one round of the longest portion fills
    int cluster = 1;
    while (cluster < MAX_CLUSTER && cluster * SCAN_SEGS * SEG < longest) cluster *= 2;
    a.cluster = cluster;
    const dim3 grid(n_req, (width + 31) / 32, cluster), threads(32 * (segs + 1));
    cudaStream_t s = (cudaStream_t)stream;
    if (out_dtype == CISR_BF16) return launch_kernel_cluster(rglru_scan_kernel<__nv_bfloat16>, grid, threads, 0, s, g_pdl, cluster, a);
    return launch_kernel_cluster(rglru_scan_kernel<float>, grid, threads, 0, s, g_pdl, cluster, a);
}
