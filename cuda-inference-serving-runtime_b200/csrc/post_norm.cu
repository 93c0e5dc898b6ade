// The seam between two sub-blocks of a layer that norms before AND after each of them: one kernel brings the output of
// the sub-block before into the residual stream through its own norm and forms the normed input of the next.
//
//   for row r (source token src = rows ? rows[r] : r), channel d:
//     v[d] = x[src][d] + norm_post(y[src])[d] * post_w[d] + (extra ? extra[src][d] : 0) + (vec ? vec[d] : 0)
//     x_out[src][d] = v[d]                              (when `store`)
//     h[r][d] = norm_pre(v)[d] * pre_w[d]               (h null: the stream only)
//   (pre_kind 2: h[r][d] = v[d], for a layer that norms its sub-blocks' outputs only)
//   norm(u) = (u - mean) / sqrt(var + eps) with var the mean squared deviation (kind 0), or u / sqrt(mean(u^2) + eps) (kind 1)
//
// y null: nothing is pending.  post_w is the output norm's weight, times the layer scale where a layer has one.  `extra` is
// a tensor of the stream's shape (the embedding output that a repeated pass adds again), `vec` one vector for all tokens.
// Everything is float; a row is held in registers, its statistics are summed in a fixed order (so a row does not depend
// on the batch), and h is rounded once to its storage type.
#include "common.cuh"

static bool g_pdl = false;
CISR_EXPORT void cisr_post_norm_set_pdl(int on) { g_pdl = on != 0; }

namespace {
struct RowArgs {
    const float* x; float* x_out; const float* y; const float* post_w; const float* extra; const float* vec; const float* pre_w;
    void* h; const int* rows;
    float post_eps, pre_eps; int post_kind, pre_kind, n_rows, hidden, store;
};

template <int VEC> struct Run { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Run<VEC> load_run(const float* p) {
    Run<VEC> r;
    if (VEC == 4) { const float4 f = *reinterpret_cast<const float4*>(p); r.v[0] = f.x; r.v[1 % VEC] = f.y; r.v[2 % VEC] = f.z; r.v[3 % VEC] = f.w; }
    else r.v[0] = p[0];
    return r;
}
template <int VEC> __device__ __forceinline__ void store_run(float* p, const Run<VEC>& r) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
    else p[0] = r.v[0];
}
template <int VEC> __device__ __forceinline__ void store_run(__nv_bfloat16* p, const Run<VEC>& r) {
    if (VEC == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(r.v[0], r.v[1 % VEC]), hi = __floats2bfloat162_rn(r.v[2 % VEC], r.v[3 % VEC]);
        uint2 raw;
        raw.x = *reinterpret_cast<const uint32_t*>(&lo); raw.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    } else p[0] = __float2bfloat16_rn(r.v[0]);
}

constexpr int WARP_ROWS = 4;      // rows per CTA where a warp takes a row

// WARP: a warp per row; else a CTA of at most MAXT threads per row.  A thread holds PER runs of VEC neighbouring channels.
template <typename OT, int VEC, int PER, bool WARP, int MAXT>
__global__ void __launch_bounds__(MAXT)
post_norm_kernel(const RowArgs a) {
    __shared__ float scratch[32];
    pdl_trigger();
    const int lane = WARP ? (threadIdx.x & 31) : threadIdx.x, width = WARP ? 32 : blockDim.x;
    const int r = WARP ? blockIdx.x * WARP_ROWS + (threadIdx.x >> 5) : blockIdx.x;
    const bool live = r < a.n_rows;
    const int hidden = a.hidden, runs = hidden / VEC;
    constexpr bool EARLY = PER <= 2;     // the weights come from no kernel: where registers allow, they are fetched before the wait
    Run<VEC> pw[EARLY ? PER : 1], nw[EARLY ? PER : 1];
    if (EARLY) {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + width * i;
            if (live && d < runs) {
                if (a.y) pw[EARLY ? i : 0] = load_run<VEC>(a.post_w + (size_t)d * VEC);
                if (a.h && a.pre_w) nw[EARLY ? i : 0] = load_run<VEC>(a.pre_w + (size_t)d * VEC);
            }
        }
    }
    pdl_wait();
    if (WARP && !live) return;
    const size_t src = (size_t)(a.rows ? a.rows[r] : r) * hidden;
    auto total = [&](float v) { return WARP ? warp_sum(v) : block_sum(v, scratch); };
    Run<VEC> v[PER], y[PER];
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + width * i;
        const bool in = d < runs;
#pragma unroll
        for (int e = 0; e < VEC; ++e) { v[i].v[e] = 0.f; y[i].v[e] = 0.f; }
        if (in) {
            v[i] = load_run<VEC>(a.x + src + (size_t)d * VEC);
            if (a.y) y[i] = load_run<VEC>(a.y + src + (size_t)d * VEC);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) sum += y[i].v[e];
    }
    if (a.y) {
        const float mean = a.post_kind == 0 ? total(sum) / (float)hidden : 0.f;
        float sq = 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            if (lane + width * i < runs) {
#pragma unroll
                for (int e = 0; e < VEC; ++e) { const float c = y[i].v[e] - mean; sq += c * c; }
            }
        }
        const float inv = 1.f / sqrtf(total(sq) / (float)hidden + a.post_eps);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + width * i;
            if (d < runs) {
                const Run<VEC> w = EARLY ? pw[EARLY ? i : 0] : load_run<VEC>(a.post_w + (size_t)d * VEC);
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[i].v[e] += (y[i].v[e] - mean) * inv * w.v[e];
            }
        }
    }
    sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + width * i;
        if (d < runs) {
            if (a.extra) {
                const Run<VEC> x = load_run<VEC>(a.extra + src + (size_t)d * VEC);
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[i].v[e] += x.v[e];
            }
            if (a.vec) {
                const Run<VEC> x = load_run<VEC>(a.vec + (size_t)d * VEC);
#pragma unroll
                for (int e = 0; e < VEC; ++e) v[i].v[e] += x.v[e];
            }
            if (a.store) store_run<VEC>(a.x_out + src + (size_t)d * VEC, v[i]);
#pragma unroll
            for (int e = 0; e < VEC; ++e) sum += v[i].v[e];
        }
    }
    if (!a.h) return;
    OT* out = reinterpret_cast<OT*>(a.h) + (size_t)r * hidden;
    if (a.pre_kind == 2) {
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int d = lane + width * i;
            if (d < runs) store_run<VEC>(out + (size_t)d * VEC, v[i]);
        }
        return;
    }
    const float mean = a.pre_kind == 0 ? total(sum) / (float)hidden : 0.f;
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        if (lane + width * i < runs) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) { const float c = v[i].v[e] - mean; sq += c * c; }
        }
    }
    const float inv = 1.f / sqrtf(total(sq) / (float)hidden + a.pre_eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = lane + width * i;
        if (d < runs) {
            const Run<VEC> w = EARLY ? nw[EARLY ? i : 0] : load_run<VEC>(a.pre_w + (size_t)d * VEC);
            Run<VEC> o;
#pragma unroll
            for (int e = 0; e < VEC; ++e) o.v[e] = (v[i].v[e] - mean) * inv * w.v[e];
            store_run<VEC>(out + (size_t)d * VEC, o);
        }
    }
}

template <typename OT, int VEC>
int launch_rows(const RowArgs& a, cudaStream_t s) {
    const int runs = a.hidden / VEC;
#define CISR_POST(PER, WARP, MAXT, GRID, BLOCK) launch_kernel(post_norm_kernel<OT, VEC, PER, WARP, MAXT>, dim3(GRID), dim3(BLOCK), 0, s, g_pdl, a)
    // many short rows: a warp per row, no barrier
    if (runs <= 256 && a.n_rows > 64) {
        const int grid = (a.n_rows + WARP_ROWS - 1) / WARP_ROWS;
        if (runs <= 64) return CISR_POST(2, true, 32 * WARP_ROWS, grid, 32 * WARP_ROWS);
        return CISR_POST(8, true, 32 * WARP_ROWS, grid, 32 * WARP_ROWS);
    }
    const auto threads = [&](int per) { return ((runs + per - 1) / per + 31) / 32 * 32; };
    // few rows: as many threads as the row has runs, so that all its loads are in flight together; many rows: four per thread
    if (runs <= 1024 && a.n_rows <= 64) return CISR_POST(1, false, 1024, a.n_rows, threads(1));
    if (runs <= 1024) return CISR_POST(4, false, 256, a.n_rows, threads(4));
    if (runs <= 4096) return CISR_POST(8, false, 512, a.n_rows, threads(8));
    if (runs <= 8192) return CISR_POST(8, false, 1024, a.n_rows, 1024);
#undef CISR_POST
    return -3;
}
}  // namespace

CISR_EXPORT int cisr_post_norm(const float* x, float* x_out, const float* y, const float* post_w, float post_eps, int post_kind,
                               const float* extra, const float* vec, const float* pre_w, float pre_eps, int pre_kind, void* h, int h_dtype,
                               const int* rows, int n_rows, int hidden, int store, void* stream) {
    if (n_rows <= 0) return 0;
    if (hidden <= 0 || (y && !post_w) || (h && !pre_w && pre_kind != 2) || post_kind < 0 || post_kind > 1 || pre_kind < 0 || pre_kind > 2) return -2;
    RowArgs a;
    a.x = x; a.x_out = x_out; a.y = y; a.post_w = post_w; a.extra = extra; a.vec = vec; a.pre_w = pre_w; a.h = h; a.rows = rows;
    a.post_eps = post_eps; a.pre_eps = pre_eps; a.post_kind = post_kind; a.pre_kind = pre_kind; a.n_rows = n_rows; a.hidden = hidden; a.store = store;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)post_w | (uintptr_t)extra | (uintptr_t)vec | (uintptr_t)pre_w | (uintptr_t)h;
    const bool wide = hidden % 4 == 0 && !(all & 15);
    cudaStream_t s = (cudaStream_t)stream;
    if (h_dtype == CISR_BF16) return wide ? launch_rows<__nv_bfloat16, 4>(a, s) : launch_rows<__nv_bfloat16, 1>(a, s);
    return wide ? launch_rows<float, 4>(a, s) : launch_rows<float, 1>(a, s);
}
