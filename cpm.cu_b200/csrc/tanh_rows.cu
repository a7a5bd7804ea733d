// Row-wise kernels of dynamic-tanh models: norms, token shift, residual sums, clamped gate, token side input, output norm
// and gate of recurrences.  Everything is computed in fp32; T is the dtype of the activations.
#include <algorithm>

#include "ptx.cuh"
#include "row_ops.cuh"

namespace {

__device__ __forceinline__ float tanh_norm(float x, float alpha, float w, float b) { return tanhf(alpha * x) * w + b; }

__device__ __forceinline__ void tanh_norm8(const float* x, const DynTanh& n, int c, float* h) {
    float w[8], b[8];
    load_vec<8>(n.w + c, w);
    load_vec<8>(n.b + c, b);
#pragma unroll
    for (int e = 0; e < 8; ++e) h[e] = tanh_norm(x[e], n.alpha, w[e], b[e]);
}

// the mixes of row r, columns c .. c + 7, from its h and the h before it
template <typename T>
__device__ __forceinline__ void store_mixes(const TokenShift& t, int r, int ld, int c, const float* h, const float* before) {
#pragma unroll
    for (int m = 0; m < kMixes; ++m) {
        float mu[8], f[8];
        load_vec<8>(t.mu + static_cast<size_t>(m) * ld + c, mu);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = h[e] + (before[e] - h[e]) * mu[e];
        store_vec<8>(static_cast<T*>(t.out) + m * t.stride + static_cast<size_t>(r) * ld + c, f);
    }
}

// columns c .. c + 7 of the h before the first row
__device__ __forceinline__ void load_before(const TokenShift& t, int c, float* before) {
    if (*t.kv_len + t.kv_off == 0) {
#pragma unroll
        for (int e = 0; e < 8; ++e) before[e] = 0.f;
    } else {
        load_vec<8>(t.prev + c, before);
    }
}

// CTA b takes row b; with mixes the last row belongs to CTA 0 as well, which has then read `prev` before it is written.
template <typename T>
__global__ void tanh_norm_kernel(const float* __restrict__ x32, const int32_t* __restrict__ rows_idx, const DynTanh n, T* __restrict__ hout,
                                 const TokenShift t, int rows, int ld) {
    grid_dependency_sync();
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8; c < ld; c += gridDim.y * blockDim.x * 8) {
        for (int r = blockIdx.x; r < rows; r += rows - 1 > 0 && blockIdx.x == 0 && t.mu != nullptr ? rows - 1 : rows) {
            const size_t at = static_cast<size_t>(rows_idx ? rows_idx[r] : r) * ld + c;
            float x[8], h[8];
            load_vec<8>(x32 + at, x);
            tanh_norm8(x, n, c, h);
            store_vec<8>(hout + static_cast<size_t>(r) * ld + c, h);
            if (t.mu == nullptr) continue;
            float before[8];
            if (r == 0) {
                load_before(t, c, before);
            } else {
                load_vec<8>(x32 + at - ld, x);
                tanh_norm8(x, n, c, before);
            }
            store_mixes<T>(t, r, ld, c, h, before);
            if (r == rows - 1) store_vec<8>(t.prev + c, h);
        }
    }
}

template <typename T>
__global__ void tanh_residual_kernel(float* __restrict__ x32, const T* __restrict__ delta, const DynTanh post, const DynTanh next,
                                     T* __restrict__ out, int rows, int ld) {
    grid_dep_trigger();
    {
        const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
        if (rows < 64 && c < ld && threadIdx.x % 8 == 0) {
            prefetch_l2(post.w + c);
            prefetch_l2(post.b + c);
            if (next.w != nullptr) {
                prefetch_l2(next.w + c);
                prefetch_l2(next.b + c);
            }
        }
    }
    grid_dep_wait();
    const size_t base = static_cast<size_t>(blockIdx.x) * ld;
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8; c < ld; c += gridDim.y * blockDim.x * 8) {
        float x[8], d[8], y[8];
        load_vec<8>(x32 + base + c, x);
        load_vec<8>(delta + base + c, d);
        tanh_norm8(d, post, c, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] += y[e];
        store_vec<8>(x32 + base + c, x);
        if (next.w != nullptr) tanh_norm8(x, next, c, x);
        store_vec<8>(out + base + c, x);
    }
}

template <typename T>
__global__ void clamped_gate_kernel(const T* __restrict__ gu, int ld_gu, T* __restrict__ act, int ld_act, int ff, float limit, float alpha,
                                    int interleaved) {
    grid_dependency_sync();
    const T* g = gu + static_cast<size_t>(blockIdx.x) * ld_gu;
    for (int c = threadIdx.x * 8; c < ff; c += blockDim.x * 8) {   // ff is a multiple of 64
        const int at = interleaved ? (c >> 6) * 128 + (c & 63) : c;
        float gv[8], uv[8];
        load_vec<8>(g + at, gv);
        load_vec<8>(g + at + (interleaved ? 64 : ff), uv);
#pragma unroll
        for (int e = 0; e < 8; ++e) gv[e] = clamped_gate(gv[e], uv[e], limit, alpha);
        store_vec<8>(act + static_cast<size_t>(blockIdx.x) * ld_act + c, gv);
    }
}

__device__ __forceinline__ float gelu_tanh(float z) {
    return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename T>
__global__ void side_gate_kernel(const T* __restrict__ z, int ld, const int32_t* __restrict__ ids, const bf16* __restrict__ table, int table_ld,
                                 int col0, int dim, int vocab, T* __restrict__ g) {
    grid_dependency_sync();
    int id = ids[blockIdx.x];
    if (id < 0 || id >= vocab) id = 0;   // reported by the embedding
    const bf16* e = table + static_cast<size_t>(id) * table_ld + col0;
    const size_t base = static_cast<size_t>(blockIdx.x) * ld;
    for (int c = threadIdx.x; c < ld; c += blockDim.x) {
        g[base + c] = from_float<T>(c < dim ? gelu_tanh(to_float<T>(z[base + c])) * __bfloat162float(e[c]) : 0.f);
    }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(512)
side_add_kernel(float* __restrict__ x32, const T* __restrict__ y, const bf16* __restrict__ w, const DynTanh next, T* __restrict__ hout,
                const TokenShift t, int width, int ld, float eps) {
    grid_dependency_sync();
    __shared__ float sh[64];
    const size_t base = static_cast<size_t>(blockIdx.x) * ld;
    float yv[VPT][8], ss = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c >= ld) continue;
        load_vec<8>(y + base + c, yv[j]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += yv[j][e] * yv[j][e];   // padding columns are zero
    }
    const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / width + eps);
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c >= ld) continue;
        float x[8], wv[8];
        load_vec<8>(x32 + base + c, x);
        load_vec<8>(w + c, wv);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] += yv[j][e] * rs * wv[e];
        store_vec<8>(x32 + base + c, x);
        if (next.w == nullptr) continue;
        float h[8];
        tanh_norm8(x, next, c, h);
        store_vec<8>(hout + base + c, h);
        if (t.mu != nullptr) {   // a single row
            float before[8];
            load_before(t, c, before);
            store_mixes<T>(t, 0, ld, c, h, before);
            store_vec<8>(t.prev + c, h);
        }
    }
}

// ---------------------------------------------------------------- one row through the token side input
constexpr int SIDE_CTAS = 16, SIDE_THREADS = 512;   // at most; a cluster of 16 is above the portable size

// element (row, k) of a matrix with K columns: tile-major (linear_weight_elems) or row-major
template <typename T>
__device__ __forceinline__ size_t weight_at(int row, int k, int K) {
    if constexpr (sizeof(T) == 2) {
        return (static_cast<size_t>(row >> 7) * (K >> 6) + (k >> 6)) * (128 * 64) + static_cast<size_t>(row & 127) * 64 + (k & 63);
    } else {
        return static_cast<size_t>(row) * K + k;
    }
}

// One cluster of SIDE_CTAS CTAs.  Every CTA takes the residual sum of the whole row; it computes its share of the gate's rows,
// which go to all CTAs, then its share of the projection's rows = columns of the stream.
template <typename T>
__global__ void __launch_bounds__(SIDE_THREADS)
side_step_kernel(const SideStepArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float sh[64];
    __shared__ float s_sum[SIDE_CTAS];
    const int dim_p = (a.dim + 63) / 64 * 64;
    float* xs = sm;                // [ld] the stream
    float* sg = xs + a.ld;         // [dim_p] gated side input
    float* ys = sg + dim_p;        // this CTA's columns of the projection
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int rank = static_cast<int>(ptx::cluster_ctarank());
    const int ctas = gridDim.x;
    const int whole = (a.ld / 8 + ctas - 1) / ctas * 8, col0 = min(rank * whole, a.ld), share = min(whole, a.ld - col0);
    const int per = (a.dim + ctas - 1) / ctas, g0 = rank * per, g1 = min(g0 + per, a.dim);
    grid_dep_trigger();
    {
        const int kb = a.ld / 64, lines = max(g1 - g0, 0) * kb;
        for (int i = tid; i < lines; i += SIDE_THREADS) prefetch_l2(a.gate + weight_at<T>(g0 + i / kb, (i % kb) * 64, a.ld));
        const int pb = dim_p / 64, plines = max(min(share, a.width - col0), 0) * pb;
        for (int i = tid; i < plines; i += SIDE_THREADS) prefetch_l2(a.proj + weight_at<T>(col0 + i / pb, (i % pb) * 64, dim_p));
        for (int c = tid * 64; c < a.ld; c += SIDE_THREADS * 64) {
            prefetch_l2(a.post.w + c);
            prefetch_l2(a.post.b + c);
        }
    }
    for (int k = tid; k < dim_p; k += SIDE_THREADS) sg[k] = 0.f;
    // what this thread's columns need at the end (all weights, and the mixer input of the step before, which the host has waited for)
    const int mine = col0 + tid * 8;
    const bool has = tid * 8 < share;
    uint4 w_norm, w_next, b_next, w_mu[kMixes];
    float prev[8];
    w_norm = w_next = b_next = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int m = 0; m < kMixes; ++m) w_mu[m] = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int e = 0; e < 8; ++e) prev[e] = 0.f;
    if (has) {
        w_norm = *reinterpret_cast<const uint4*>(a.norm + mine);
        if (a.next.w != nullptr) {
            w_next = *reinterpret_cast<const uint4*>(a.next.w + mine);
            b_next = *reinterpret_cast<const uint4*>(a.next.b + mine);
        }
        if (a.shift.mu != nullptr) {
#pragma unroll
            for (int m = 0; m < kMixes; ++m) w_mu[m] = *reinterpret_cast<const uint4*>(a.shift.mu + static_cast<size_t>(m) * a.ld + mine);
            load_vec<8>(a.shift.prev + mine, prev);
        }
    }
    grid_dep_wait();
    for (int c = tid * 8; c < a.ld; c += SIDE_THREADS * 8) {
        float x[8], d[8], y[8];
        load_vec<8>(a.x32 + c, x);
        load_vec<8>(static_cast<const T*>(a.delta) + c, d);
        tanh_norm8(d, a.post, c, y);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] += y[e];
        store_vec<8>(xs + c, x);
    }
    int id = a.ids[0];
    if (id < 0 || id >= a.vocab) id = 0;   // reported by the embedding
    const bf16* side = a.table + static_cast<size_t>(id) * a.table_ld + a.col0;
    ptx::cluster_sync();   // xs here; sg zeroed in every CTA
    for (int row = g0 + warp; row < g1; row += SIDE_THREADS / 32) {
        float z = 0.f;
#pragma unroll 8
        for (int k = lane * 8; k < a.ld; k += 256) {
            float w[8], x[8];
            load_vec<8>(a.gate + weight_at<T>(row, k, a.ld), w);
            load_vec<8>(xs + k, x);
#pragma unroll
            for (int e = 0; e < 8; ++e) z = fmaf(w[e], to_float<T>(from_float<T>(x[e])), z);
        }
        z = to_float<T>(from_float<T>(warp_sum(z)));
        const float g = to_float<T>(from_float<T>(gelu_tanh(z) * __bfloat162float(side[row])));
        if (lane < ctas) ptx::st_cluster_f32(ptx::cluster_map(ptx::smem_u32(sg + row), lane), g);
    }
    ptx::cluster_sync();
    int lpr = 8;           // lanes per row of the projection
    while (lpr < 32 && lpr * 8 < dim_p) lpr *= 2;
    const int sub = lane / lpr, sl = lane % lpr, rpw = 32 / lpr;
    float ss = 0.f;
    constexpr int B = 8;   // rows in flight per group of lanes
    for (int r0 = warp * rpw * B; r0 < share; r0 += SIDE_THREADS / 32 * rpw * B) {   // uniform within a warp
        float y[B] = {};
        for (int k = sl * 8; k < dim_p; k += lpr * 8) {
            float g[8];
            load_vec<8>(sg + k, g);
            uint4 w[B];
#pragma unroll
            for (int n = 0; n < B; ++n) {
                const int r = r0 + n * rpw + sub;
                w[n] = make_uint4(0, 0, 0, 0);
                if (r < share && col0 + r < a.width) w[n] = __ldg(reinterpret_cast<const uint4*>(a.proj + weight_at<T>(col0 + r, k, dim_p)));
            }
#pragma unroll
            for (int n = 0; n < B; ++n) {
                const bf16* e8 = reinterpret_cast<const bf16*>(&w[n]);
#pragma unroll
                for (int e = 0; e < 8; ++e) y[n] = fmaf(__bfloat162float(e8[e]), g[e], y[n]);
            }
        }
#pragma unroll
        for (int n = 0; n < B; ++n) {
            for (int o = lpr / 2; o > 0; o >>= 1) y[n] += __shfl_xor_sync(0xffffffffu, y[n], o);
            y[n] = to_float<T>(from_float<T>(y[n]));
            const int r = r0 + n * rpw + sub;
            if (sl == 0 && r < share) {
                ys[r] = y[n];
                ss += y[n] * y[n];
            }
        }
    }
    ss = block_sum2(ss, 0.f, sh).x;
    if (tid < ctas) ptx::st_cluster_f32(ptx::cluster_map(ptx::smem_u32(s_sum + rank), tid), ss);
    ptx::cluster_sync();
    float sum = 0.f;
    for (int i = 0; i < ctas; ++i) sum += s_sum[i];
    const float rs = rsqrtf(sum / a.width + a.eps);
    if (!has) return;   // share <= 8 * SIDE_THREADS
    auto bf8 = [](const uint4& u, int e) { return __bfloat162float(reinterpret_cast<const bf16*>(&u)[e]); };
    float x[8], y[8], h[8];
    load_vec<8>(xs + mine, x);
    load_vec<8>(ys + tid * 8, y);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] += y[e] * rs * bf8(w_norm, e);
    store_vec<8>(a.x32 + mine, x);
    if (a.next.w == nullptr) return;
#pragma unroll
    for (int e = 0; e < 8; ++e) h[e] = tanh_norm(x[e], a.next.alpha, bf8(w_next, e), bf8(b_next, e));
    store_vec<8>(static_cast<T*>(a.h) + mine, h);
    if (a.shift.mu == nullptr) return;
    const bool first = *a.shift.kv_len + a.shift.kv_off == 0;
#pragma unroll
    for (int m = 0; m < kMixes; ++m) {
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = h[e] + ((first ? 0.f : prev[e]) - h[e]) * bf8(w_mu[m], e);
        store_vec<8>(static_cast<T*>(a.shift.out) + m * a.shift.stride + mine, f);
    }
    store_vec<8>(a.shift.prev + mine, h);
}

// ROWS tokens x 256 channels per CTA, two neighbouring channels per thread.
constexpr int DECAY_THREADS = 128;

template <typename T, int ROWS>
__global__ void __launch_bounds__(DECAY_THREADS)
decay_kernel(const T* __restrict__ x, int ld_x, const bf16* __restrict__ w2, const bf16* __restrict__ w0, int rank, int channels,
             float* __restrict__ out, int ld_out, int rows) {
    extern __shared__ __align__(16) float inner[];   // [rank][ROWS]
    const int row0 = blockIdx.y * ROWS, n = min(ROWS, rows - row0);
    const int c = (blockIdx.x * DECAY_THREADS + threadIdx.x) * 2;
    const bool one = c < channels, two = c + 1 < channels;
    const float b0 = one ? __bfloat162float(w0[c]) : 0.f, b1 = two ? __bfloat162float(w0[c + 1]) : 0.f;
    grid_dependency_sync();
    for (int i = threadIdx.x; i < ROWS * rank; i += DECAY_THREADS) {
        const int t = i / rank, k = i - t * rank;
        inner[k * ROWS + t] = t < n ? tanhf(to_float<T>(x[static_cast<size_t>(row0 + t) * ld_x + k])) : 0.f;
    }
    __syncthreads();
    if (!one) return;
    f32x2 z[2][ROWS / 2];
#pragma unroll
    for (int t = 0; t < ROWS / 2; ++t) {
        z[0][t] = pair(b0, b0);
        z[1][t] = pair(b1, b1);
    }
    auto add = [&](float a, float b, int k) {
        const f32x2 wa = pair(a, a), wb = pair(b, b);
#pragma unroll
        for (int t = 0; t < ROWS / 2; t += 2) {
            const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(inner + k * ROWS + 2 * t);
            z[0][t] = fma2(wa, v.x, z[0][t]);
            z[0][t + 1] = fma2(wa, v.y, z[0][t + 1]);
            z[1][t] = fma2(wb, v.x, z[1][t]);
            z[1][t + 1] = fma2(wb, v.y, z[1][t + 1]);
        }
    };
    const bf16* w = w2 + c;
    if (channels % 2 == 0) {
        int k = 0;
        for (; k + 8 <= rank; k += 8) {
            __nv_bfloat162 f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = *reinterpret_cast<const __nv_bfloat162*>(w + static_cast<size_t>(k + e) * channels);
#pragma unroll
            for (int e = 0; e < 8; ++e) add(__low2float(f[e]), __high2float(f[e]), k + e);
        }
        for (; k < rank; ++k) {
            const __nv_bfloat162 f = *reinterpret_cast<const __nv_bfloat162*>(w + static_cast<size_t>(k) * channels);
            add(__low2float(f), __high2float(f), k);
        }
    } else {
        for (int k = 0; k < rank; ++k) {
            const bf16* q = w + static_cast<size_t>(k) * channels;
            add(__bfloat162float(q[0]), two ? __bfloat162float(q[1]) : 0.f, k);
        }
    }
#pragma unroll
    for (int t = 0; t < ROWS / 2; ++t) {
        const float2 f = unpair(z[0][t]), g = unpair(z[1][t]);
        float* o = out + static_cast<size_t>(row0 + 2 * t) * ld_out + c;
        if (2 * t < n) {
            o[0] = expf(-expf(f.x));
            if (two) o[1] = expf(-expf(g.x));
        }
        if (2 * t + 1 < n) {
            o[ld_out] = expf(-expf(f.y));
            if (two) o[ld_out + 1] = expf(-expf(g.y));
        }
    }
}

// One CTA per row; one warp per group, or the whole CTA for a single group.
template <typename T>
__global__ void norm_gate_kernel(const float* __restrict__ o, int ld_o, int groups, int group, const bf16* __restrict__ w,
                                 const T* __restrict__ gate, int ld_gate, int silu, float eps, float scale, T* __restrict__ out, int ld_out) {
    grid_dependency_sync();
    __shared__ float sh[64];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    o += static_cast<size_t>(blockIdx.x) * ld_o;
    gate += static_cast<size_t>(blockIdx.x) * ld_gate;
    out += static_cast<size_t>(blockIdx.x) * ld_out;
    auto finish = [&](int c, float rs) {
        const float g = to_float<T>(gate[c]), s = 1.f / (1.f + expf(-g));
        out[c] = from_float<T>(o[c] * rs * __bfloat162float(w[c]) * (silu ? g * s : s) * scale);
    };
    if (groups == 1) {
        float ss = 0.f;
        for (int c = threadIdx.x; c < group; c += blockDim.x) ss += o[c] * o[c];
        const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / group + eps);
        for (int c = threadIdx.x; c < group; c += blockDim.x) finish(c, rs);
    } else {
        for (int g = warp; g < groups; g += blockDim.x >> 5) {
            float ss = 0.f;
            for (int c = g * group + lane; c < (g + 1) * group; c += 32) ss += o[c] * o[c];
            const float rs = rsqrtf(warp_sum(ss) / group + eps);
            for (int c = g * group + lane; c < (g + 1) * group; c += 32) finish(c, rs);
        }
    }
}

// The same with 8 columns per thread: `lanes` neighbouring threads hold a group (a power of two, at most a warp), or the CTA holds
// the single group, at most 8 * VPT columns per thread.
template <typename T, int VPT>
__global__ void __launch_bounds__(256)
norm_gate8_kernel(const float* __restrict__ o, int ld_o, int lanes, int cols, int group, const bf16* __restrict__ w, const T* __restrict__ gate,
                  int ld_gate, int silu, float eps, float scale, T* __restrict__ out, int ld_out) {
    grid_dependency_sync();
    __shared__ float sh[64];
    o += static_cast<size_t>(blockIdx.x) * ld_o;
    gate += static_cast<size_t>(blockIdx.x) * ld_gate;
    out += static_cast<size_t>(blockIdx.x) * ld_out;
    float v[VPT][8], g[VPT][8], wv[VPT][8], ss[VPT], sum = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        ss[j] = 0.f;
        if (c >= cols) continue;
        load_vec<8>(o + c, v[j]);
        load_vec<8>(gate + c, g[j]);
        load_vec<8>(w + c, wv[j]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss[j] += v[j][e] * v[j][e];
        sum += ss[j];
    }
    if (lanes == 0) sum = block_sum2(sum, 0.f, sh).x;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        for (int m = lanes / 2; m > 0; m >>= 1) ss[j] += __shfl_xor_sync(0xffffffffu, ss[j], m);
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c >= cols) continue;
        const float rs = rsqrtf((lanes == 0 ? sum : ss[j]) / group + eps) * scale;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const float s = sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-g[j][e])) : 1.f / (1.f + expf(-g[j][e]));
            v[j][e] = v[j][e] * rs * wv[j][e] * (silu ? g[j][e] * s : s);
        }
        store_vec<8>(out + c, v[j]);
    }
}

// Grid and block of an element-wise kernel over rows of ld / 8 vectors: few rows spread over column blocks.
inline void row_grid(int rows, int ld, dim3& grid, dim3& block) {
    const int vecs = ld / 8;
    const int threads = std::min(rows < 64 ? 64 : 256, (vecs + 31) / 32 * 32);
    grid = dim3(rows, rows < 64 ? ceil_div(vecs, threads) : 1);
    block = dim3(threads);
}

}  // namespace

template <typename T>
void launch_tanh_norm(const float* x32, const int32_t* rows_idx, const DynTanh& n, T* h, const TokenShift& shift, int rows, int ld,
                      cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(ld % 64 == 0 && (shift.mu == nullptr || rows_idx == nullptr), "tanh_norm: bad arguments");
    dim3 grid, block;
    row_grid(rows, ld, grid, block);
    if (shift.mu != nullptr && rows > 1) grid.x = rows - 1;
    launch_kernel(tanh_norm_kernel<T>, grid, block, 0, s, x32, rows_idx, n, h, shift, rows, ld);
}

template <typename T>
void launch_tanh_residual(float* x32, const T* delta, const DynTanh& post, const DynTanh& next, T* out, int rows, int ld, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    dim3 grid, block;
    row_grid(rows, ld, grid, block);
    launch_kernel(tanh_residual_kernel<T>, grid, block, 0, s, x32, delta, post, next, out, rows, ld);
}

template <typename T>
void launch_clamped_gate(const T* gu, int ld_gu, T* act, int ld_act, int rows, int ff, float limit, float alpha, bool interleaved, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(ff % 64 == 0 && ld_act % 8 == 0 && ld_gu % 8 == 0, "clamped gate: widths must be multiples of 64");
    launch_kernel(clamped_gate_kernel<T>, dim3(rows), dim3(256), 0, s, gu, ld_gu, act, ld_act, ff, limit, alpha, interleaved ? 1 : 0);
}

template <typename T>
void launch_side_gate(const T* z, int ld, const int32_t* ids, const bf16* table, int table_ld, int col0, int dim, int vocab, T* g, int rows,
                      cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    launch_kernel(side_gate_kernel<T>, dim3(rows), dim3(64), 0, s, z, ld, ids, table, table_ld, col0, dim, vocab, g);
}

template <typename T>
void launch_side_add(float* x32, const T* y, const bf16* w, const DynTanh& next, T* h, const TokenShift& shift, int rows, int width, int ld,
                     float eps, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(ld % 64 == 0 && ld <= 512 * 8 * 4 && (shift.mu == nullptr || rows == 1), "side_add: bad arguments");
    const int vecs = ld / 8;
    const int threads = vecs >= 512 ? 512 : (vecs + 31) / 32 * 32;
    if (vecs <= 512) launch_kernel(side_add_kernel<T, 1>, dim3(rows), dim3(threads), 0, s, x32, y, w, next, h, shift, width, ld, eps);
    else launch_kernel(side_add_kernel<T, 4>, dim3(rows), dim3(threads), 0, s, x32, y, w, next, h, shift, width, ld, eps);
}

template <typename T>
void launch_side_step(const SideStepArgs& a, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(a.ld % 64 == 0 && a.ld <= 16384 && a.dim >= 1 && a.dim <= 4096, "side_step: unsupported sizes");
    static int ctas = 0;
    if (ctas == 0) {
        constexpr int kSmem = 96 * 1024;
        CUDA_CHECK(cudaFuncSetAttribute(side_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem));
        CUDA_CHECK(cudaFuncSetAttribute(side_step_kernel<T>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
        ctas = max_active_clusters(side_step_kernel<T>, dim3(SIDE_THREADS), kSmem, SIDE_CTAS) >= 1 ? SIDE_CTAS : 8;
    }
    const size_t smem = sizeof(float) * (a.ld + pad64(a.dim) + a.ld / 8);
    launch_kernel_cluster(side_step_kernel<T>, dim3(ctas), dim3(SIDE_THREADS), smem, s, ctas, a);
}
template void launch_side_step<bf16>(const SideStepArgs&, cudaStream_t);
template void launch_side_step<float>(const SideStepArgs&, cudaStream_t);

template <typename T>
void launch_decay(const T* x, int ld_x, const bf16* w2, const bf16* w0, int rank, int channels, float* out, int ld_out, int rows, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(rank >= 1 && rank <= 1024, "time mix: inner width of the decay must be in [1, 1024]");
    const int blocks = ceil_div(channels, 2 * DECAY_THREADS);
    auto run = [&](auto kernel, int n) {
        launch_kernel(kernel, dim3(blocks, ceil_div(rows, n)), dim3(DECAY_THREADS), rank * n * sizeof(float), s, x, ld_x, w2, w0, rank, channels, out,
                      ld_out, rows);
    };
    if (rows >= 256 && rank <= 512) run(decay_kernel<T, 16>, 16);
    else run(decay_kernel<T, 4>, 4);
}

template <typename T>
void launch_norm_gate(const float* o, int ld_o, int groups, int group, const bf16* w, const T* gate, int ld_gate, bool silu, float eps,
                      float scale, T* out, int ld_out, int rows, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    const int lanes = groups == 1 ? 0 : group / 8, cols = groups * group;
    const bool wide = group % 8 == 0 && (lanes & (lanes - 1)) == 0 && lanes <= 32 && ld_o % 4 == 0 && ld_gate % 8 == 0 && ld_out % 8 == 0 &&
                      reinterpret_cast<uintptr_t>(gate) % 16 == 0 && reinterpret_cast<uintptr_t>(out) % 16 == 0 && cols <= 4 * 256 * 8;
    if (wide) {
        auto run = [&](auto kernel) {
            launch_kernel(kernel, dim3(rows), dim3(256), 0, s, o, ld_o, lanes, cols, group, w, gate, ld_gate, silu ? 1 : 0, eps, scale, out, ld_out);
        };
        if (cols <= 256 * 8) run(norm_gate8_kernel<T, 1>);
        else if (cols <= 2 * 256 * 8) run(norm_gate8_kernel<T, 2>);
        else run(norm_gate8_kernel<T, 4>);
        return;
    }
    launch_kernel(norm_gate_kernel<T>, dim3(rows), dim3(256), 0, s, o, ld_o, groups, group, w, gate, ld_gate, silu ? 1 : 0, eps, scale, out,
                  ld_out);
}

#define CPM_INSTANTIATE(T)                                                                                                                  \
    template void launch_tanh_norm<T>(const float*, const int32_t*, const DynTanh&, T*, const TokenShift&, int, int, cudaStream_t);         \
    template void launch_tanh_residual<T>(float*, const T*, const DynTanh&, const DynTanh&, T*, int, int, cudaStream_t);                    \
    template void launch_clamped_gate<T>(const T*, int, T*, int, int, int, float, float, bool, cudaStream_t);                               \
    template void launch_side_gate<T>(const T*, int, const int32_t*, const bf16*, int, int, int, int, T*, int, cudaStream_t);               \
    template void launch_side_add<T>(float*, const T*, const bf16*, const DynTanh&, T*, const TokenShift&, int, int, int, float,            \
                                     cudaStream_t);                                                                                         \
    template void launch_decay<T>(const T*, int, const bf16*, const bf16*, int, int, float*, int, int, cudaStream_t);                       \
    template void launch_norm_gate<T>(const float*, int, int, int, const bf16*, const T*, int, bool, float, float, T*, int, int, cudaStream_t);
CPM_INSTANTIATE(bf16)
CPM_INSTANTIATE(float)
