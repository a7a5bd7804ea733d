// Row-wise kernels, plain attention and the fp32 matrix product of layered models (layered.cuh).  Norms, the residual
// sum, attention scores and weights are fp32 whatever T is.
#include <algorithm>

#include "row_ops.cuh"

namespace {

template <typename T>
__global__ void embed_rows_kernel(const int32_t* __restrict__ ids, const bf16* __restrict__ table, int vocab, float scale, float* __restrict__ x32,
                                  T* __restrict__ xh, int ld, const StateCheck check, int* __restrict__ error) {
    grid_dependency_sync();
    const size_t row = blockIdx.x;
    if (check.state_len != nullptr && row == 0 && threadIdx.x == 0) {
        const int first = *check.kv_len + check.kv_off;
        const bool ok = first == 0 || first == *check.state_len;
        if (!ok) atomicOr(error, ERR_STATE_POS);
        *check.state_len = ok ? first + static_cast<int>(gridDim.x) : -1;
    }
    int id = ids[row];
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicOr(error, ERR_BAD_TOKEN);
        id = 0;
    }
    const bf16* src = table + static_cast<size_t>(id) * ld;
    for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
        float f[8];
        load_vec<8>(src + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= scale;
        store_vec<8>(x32 + row * ld + c, f);
        store_vec<8>(xh + row * ld + c, f);
    }
}

// One CTA per token row.
template <typename T, int VEC>
__global__ void qkv_norm_append_kernel(const QkvNormArgs a) {
    grid_dependency_sync();
    __shared__ float sh[64];
    __shared__ float2 turn[256];   // cos, sin of the row's angles
    const int r = blockIdx.x;
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    const T* row = static_cast<const T*>(a.qkv) + static_cast<size_t>(r) * a.ld;
    const bool own_kv = a.k_cache != nullptr;
    const long long kv_row = own_kv ? static_cast<long long>(*a.kv_len) + a.kv_off + r : 0;
    const bool store_kv = own_kv && kv_row >= 0 && kv_row < a.cache_rows;
    if (own_kv && !store_kv && threadIdx.x == 0) atomicOr(a.error, ERR_KV_OVERFLOW);
    const int half = a.rot_dims / 2;
    if (half > 0) {
        const float pos = static_cast<float>(*a.kv_len + a.kv_off + r);
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            float sn, cs;
            sincosf(pos * a.inv_freq[i], &sn, &cs);
            turn[i] = make_float2(cs, sn);
        }
        __syncthreads();
    }
    float rq = 1.f, rk = 1.f;
    if (a.wq != nullptr) {
        float sq = 0.f, sk = 0.f, f[VEC];
        for (int c = threadIdx.x * VEC; c < nq; c += blockDim.x * VEC) {
            load_vec<VEC>(row + c, f);
#pragma unroll
            for (int e = 0; e < VEC; ++e) sq += f[e] * f[e];
        }
        if (own_kv) {
            for (int c = threadIdx.x * VEC; c < nk; c += blockDim.x * VEC) {
                load_vec<VEC>(row + nq + c, f);
#pragma unroll
                for (int e = 0; e < VEC; ++e) sk += f[e] * f[e];
            }
        }
        const float2 t = block_sum2(sq, sk, sh);
        rq = rsqrtf(t.x / nq + a.eps);
        if (own_kv) rk = rsqrtf(t.y / nk + a.eps);
    }
    auto place = [&](const T* src, const bf16* w, float rs, int n_heads, int d, int dp, T* dst, bool pad, int rot) {
        const int per = (pad ? dp : d) / VEC;
        for (int i = threadIdx.x; i < n_heads * per; i += blockDim.x) {
            const int h = i / per, c = (i - h * per) * VEC;
            float f[VEC];
            if (c < d) {
                load_vec<VEC>(src + h * d + c, f);
                if (w != nullptr) {
                    float g[VEC];
                    load_vec<VEC>(w + h * d + c, g);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) f[e] = f[e] * rs * g[e];
                }
                if (c < 2 * rot) {   // rot is a multiple of VEC
                    const bool upper = c >= rot;
                    const int other = upper ? c - rot : c + rot, i0 = upper ? c - rot : c;
                    float p[VEC];
                    load_vec<VEC>(src + h * d + other, p);
                    if (w != nullptr) {
                        float g[VEC];
                        load_vec<VEC>(w + h * d + other, g);
#pragma unroll
                        for (int e = 0; e < VEC; ++e) p[e] = p[e] * rs * g[e];
                    }
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        const float2 cs = turn[i0 + e];
                        f[e] = upper ? f[e] * cs.x + p[e] * cs.y : f[e] * cs.x - p[e] * cs.y;
                    }
                }
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) f[e] = 0.f;
            }
            store_vec<VEC>(dst + static_cast<size_t>(h) * dp + c, f);
        }
    };
    // the query buffer is shared by layers of different widths, so its padding is written; a cache's padding stays zero
    place(row, a.wq, rq, a.heads, a.dim, a.dim_p, static_cast<T*>(a.q_out) + static_cast<size_t>(r) * a.heads * a.dim_p, true, half);
    if (store_kv) {
        place(row + nq, a.wk, rk, a.kv_heads, a.dim, a.dim_p,
              static_cast<T*>(a.k_cache) + static_cast<size_t>(kv_row) * a.kv_heads * a.dim_p, false, half);
        place(row + nq + nk, nullptr, 1.f, a.kv_heads, a.vdim, a.vdim_p,
              static_cast<T*>(a.v_cache) + static_cast<size_t>(kv_row) * a.kv_heads * a.vdim_p, false, 0);
        (void)nv;
    }
}

template <typename T, int VPT, bool MIX>
__global__ void __launch_bounds__(512)
out_norm_kernel(float* __restrict__ x32, T* __restrict__ xh, const T* __restrict__ delta, const MoeMix mix, float mult,
                const bf16* __restrict__ w, int width, int ld, float eps) {
    grid_dep_trigger();
    __shared__ float sh[64];
    __shared__ int s_row[kMoeMaxTop];
    __shared__ float s_w[kMoeMaxTop];
    const size_t base = static_cast<size_t>(blockIdx.x) * ld;
    float wv[VPT][8];   // the weights never depend on the previous kernel
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c < ld) load_vec<8>(w + c, wv[j]);
    }
    grid_dep_wait();
    float xv[VPT][8], dv[VPT][8];
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c < ld) load_vec<8>(x32 + base + c, xv[j]);
    }
    if constexpr (MIX) {
        if (threadIdx.x < mix.top) {
            const size_t i = static_cast<size_t>(blockIdx.x) * mix.top + threadIdx.x;
            const int e = mix.expert[i];
            s_row[threadIdx.x] = e < mix.experts ? mix.offset[e] + mix.rank[i] : -1;
            s_w[threadIdx.x] = mix.weight[i];
        }
        __syncthreads();
        const float idw = mix.id_weight[blockIdx.x];
        const T* y = static_cast<const T*>(mix.y);
#pragma unroll
        for (int j = 0; j < VPT; ++j) {
            const int c = (threadIdx.x + j * blockDim.x) * 8;
            if (c >= ld) continue;
#pragma unroll
            for (int e = 0; e < 8; ++e) dv[j][e] = idw * xv[j][e];
#pragma unroll 4
            for (int k = 0; k < mix.top; ++k) {
                if (s_row[k] < 0) continue;
                float f[8];
                load_vec<8>(y + static_cast<size_t>(s_row[k]) * ld + c, f);
                const float wk = s_w[k];
#pragma unroll
                for (int e = 0; e < 8; ++e) dv[j][e] += wk * f[e];
            }
            if (mix.shared_row0 >= 0) {
                float f[8];
                load_vec<8>(y + (static_cast<size_t>(mix.shared_row0) + blockIdx.x) * ld + c, f);
#pragma unroll
                for (int e = 0; e < 8; ++e) dv[j][e] += f[e];
            }
        }
    } else {
#pragma unroll
        for (int j = 0; j < VPT; ++j) {
            const int c = (threadIdx.x + j * blockDim.x) * 8;
            if (c < ld) load_vec<8>(delta + base + c, dv[j]);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c < ld) {
#pragma unroll
            for (int e = 0; e < 8; ++e) ss += dv[j][e] * dv[j][e];   // padding columns are zero
        }
    }
    const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / width + eps);
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 8;
        if (c < ld) {
#pragma unroll
            for (int e = 0; e < 8; ++e) xv[j][e] += mult * (dv[j][e] * rs * (1.f + wv[j][e]));
            store_vec<8>(x32 + base + c, xv[j]);
            store_vec<8>(xh + base + c, xv[j]);
        }
    }
}

template <typename T>
__global__ void norm_rows_kernel(const float* __restrict__ x32, const int32_t* __restrict__ rows_idx, const bf16* __restrict__ w,
                                 T* __restrict__ y, int width, int ld, float eps) {
    grid_dependency_sync();
    __shared__ float sh[64];
    const float* x = x32 + static_cast<size_t>(rows_idx ? rows_idx[blockIdx.x] : blockIdx.x) * ld;
    float ss = 0.f, f[8], g[8];
    for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
        load_vec<8>(x + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
    }
    const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / width + eps);
    for (int c = threadIdx.x * 8; c < ld; c += blockDim.x * 8) {
        load_vec<8>(x + c, f);
        load_vec<8>(w + c, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = f[e] * rs * (1.f + g[e]);
        store_vec<8>(y + static_cast<size_t>(blockIdx.x) * ld + c, f);
    }
}

// One warp per (token, head): lanes take keys for the scores and value columns for the output.
constexpr int PA_WARPS = 4, PA_MAX_D = 512;

template <typename T>
__global__ void plain_attention_kernel(const PlainAttnArgs a) {
    grid_dependency_sync();
    __shared__ float sq[PA_WARPS][PA_MAX_D];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int item = blockIdx.x * PA_WARPS + warp;
    if (item >= a.tq * a.hq) return;
    const int t = item / a.hq, h = item - t * a.hq;
    const int g = h / (a.hq / a.hkv);
    const T* q = static_cast<const T*>(a.q) + static_cast<size_t>(item) * a.dk;
    for (int c = lane; c < a.dk; c += 32) sq[warp][c] = to_float<T>(q[c]);
    __syncwarp();
    const int i = *a.kv_len + a.kv_len_add - a.tq + t;   // position of this token
    const int lo = a.window > 0 ? max(i - a.window + 1, 0) : 0;
    const float slope = a.bias_exp > 0.f ? exp2f(-a.bias_exp * static_cast<float>(h + 1) / static_cast<float>(a.hq)) : 0.f;
    const T* kc = static_cast<const T*>(a.k_cache) + static_cast<size_t>(g) * a.dk;
    const T* vc = static_cast<const T*>(a.v_cache) + static_cast<size_t>(g) * a.dv;
    const size_t kld = static_cast<size_t>(a.hkv) * a.dk, vld = static_cast<size_t>(a.hkv) * a.dv;
    float m = -INFINITY, l = 0.f, acc[PA_MAX_D / 32];
#pragma unroll
    for (int c = 0; c < PA_MAX_D / 32; ++c) acc[c] = 0.f;
    for (int j0 = lo; j0 <= i; j0 += 32) {
        const int j = j0 + lane;
        float s = -INFINITY;
        if (j <= i) {
            const T* k = kc + static_cast<size_t>(j) * kld;
            float d = 0.f, f[8];
            for (int c = 0; c < a.dk; c += 8) {   // dk is padded to a multiple of 64
                load_vec<8>(k + c, f);
#pragma unroll
                for (int e = 0; e < 8; ++e) d += sq[warp][c + e] * f[e];
            }
            s = d * a.scale - slope * static_cast<float>(i - j);
        }
        float mx = s;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m, mx);
        const float alpha = expf(m - m_new);
        const float p = expf(s - m_new);
        l = l * alpha + warp_sum(p);
        m = m_new;
#pragma unroll
        for (int c = 0; c < PA_MAX_D / 32; ++c) acc[c] *= alpha;
        const int n = min(32, i - j0 + 1);
        for (int jj = 0; jj < n; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const T* v = vc + static_cast<size_t>(j0 + jj) * vld;
#pragma unroll
            for (int c = 0; c < PA_MAX_D / 32; ++c) {
                if (c * 32 + lane < a.out_cols) acc[c] += pj * to_float<T>(v[c * 32 + lane]);
            }
        }
    }
    T* out = static_cast<T*>(a.out) + static_cast<size_t>(t) * a.out_ld + static_cast<size_t>(h) * a.out_cols;
    if (a.sink != 0) l += expf(-m);
    const float inv = l > 0.f ? a.out_scale / l : 0.f;
#pragma unroll
    for (int c = 0; c < PA_MAX_D / 32; ++c) {
        if (c * 32 + lane < a.out_cols) out[c * 32 + lane] = from_float<T>(acc[c] * inv);
    }
}

// 64 x 64 output tile, 16 x 16 threads with 4 x 4 outputs each.
__global__ void __launch_bounds__(256)
linear_f32_kernel(const float* __restrict__ x, int ldx, const bf16* __restrict__ w, size_t w_stride, float* __restrict__ y, int ldy,
                  int M, int N, int K, const int4* __restrict__ entries, const int32_t* __restrict__ n_entries, int x_at_y) {
    grid_dependency_sync();
    constexpr int KT = 32;
    __shared__ float sx[KT][kF32Rows + 4], sw[KT][64 + 4];
    int x0 = blockIdx.y * kF32Rows, y0 = x0, rows = min(kF32Rows, M - x0);
    if (entries != nullptr) {
        if (static_cast<int>(blockIdx.z) >= *n_entries) return;
        const int4 e = entries[blockIdx.z];
        w += static_cast<size_t>(e.x) * w_stride;
        x0 = x_at_y ? e.z : e.y; y0 = e.z; rows = e.w;
    }
    const int n0 = blockIdx.x * 64;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += KT) {   // K is a multiple of 64
        for (int i = threadIdx.x; i < 64 * (KT / 4); i += 256) {
            const int r = i / (KT / 4), c = (i - r * (KT / 4)) * 4;
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < rows) v = *reinterpret_cast<const float4*>(x + static_cast<size_t>(x0 + r) * ldx + k0 + c);
            sx[c][r] = v.x; sx[c + 1][r] = v.y; sx[c + 2][r] = v.z; sx[c + 3][r] = v.w;
            bf16 b[4] = {};
            if (n0 + r < N) *reinterpret_cast<uint2*>(b) = *reinterpret_cast<const uint2*>(w + static_cast<size_t>(n0 + r) * K + k0 + c);
#pragma unroll
            for (int e = 0; e < 4; ++e) sw[c + e][r] = __bfloat162float(b[e]);
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < KT; ++k) {
            const float4 xv = *reinterpret_cast<const float4*>(&sx[k][ty * 4]);
            const float4 wv = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
            const float xs[4] = {xv.x, xv.y, xv.z, xv.w}, ws[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xs[i], ws[j], acc[i][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        if (ty * 4 + i >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (n0 + tx * 4 + j < N) y[static_cast<size_t>(y0 + ty * 4 + i) * ldy + n0 + tx * 4 + j] = acc[i][j];
        }
    }
}

__global__ void silu_f32_kernel(const float* __restrict__ gu, int ld_gu, float* __restrict__ act, int ld_act, int ff) {
    grid_dependency_sync();
    const float* g = gu + static_cast<size_t>(blockIdx.x) * ld_gu;
    float* o = act + static_cast<size_t>(blockIdx.x) * ld_act;
    for (int c = threadIdx.x; c < ff; c += blockDim.x) o[c] = g[c] / (1.f + expf(-g[c])) * g[ff + c];
}

}  // namespace

template <typename T>
void launch_embed_rows(const int32_t* ids, const bf16* table, int vocab, float scale, float* x32, T* xh, int ld, int rows,
                       const StateCheck& check, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    launch_kernel(embed_rows_kernel<T>, dim3(rows), dim3(128), 0, s, ids, table, vocab, scale, x32, xh, ld, check, runtime().d_error);
}

template <typename T>
void launch_qkv_norm_append(const QkvNormArgs& a, int rows, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(a.rot_dims % 2 == 0 && a.rot_dims <= a.dim && a.rot_dims <= 512, "layered model: bad number of rotated dimensions");
    const bool v8 = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0 && (a.rot_dims / 2) % 8 == 0;
    if (v8) launch_kernel(qkv_norm_append_kernel<T, 8>, dim3(rows), dim3(256), 0, s, a);
    else launch_kernel(qkv_norm_append_kernel<T, 1>, dim3(rows), dim3(256), 0, s, a);
}

template <typename T>
void launch_out_norm(float* x32, T* xh, const T* delta, const MoeMix& mix, float mult, const bf16* w, int rows, int width, int ld,
                     float eps, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    CPM_REQUIRE(ld % 64 == 0 && ld <= 512 * 8 * 4, "layered model: width above 16384 is not supported");
    CPM_REQUIRE(mix.top <= kMoeMaxTop, "mixture of experts: too many experts per token");
    const int vecs = ld / 8;
    const int threads = vecs >= 512 ? 512 : (vecs + 31) / 32 * 32;
    const bool mixed = mix.y != nullptr;
    auto run = [&](auto kernel) { launch_kernel(kernel, dim3(rows), dim3(threads), 0, s, x32, xh, delta, mix, mult, w, width, ld, eps); };
    if (vecs <= 512) {
        if (mixed) run(out_norm_kernel<T, 1, true>); else run(out_norm_kernel<T, 1, false>);
    } else {
        if (mixed) run(out_norm_kernel<T, 4, true>); else run(out_norm_kernel<T, 4, false>);
    }
}

template <typename T>
void launch_norm_rows(const float* x32, const int32_t* rows_idx, const bf16* w, T* y, int rows, int width, int ld, float eps,
                      cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    launch_kernel(norm_rows_kernel<T>, dim3(rows), dim3(256), 0, s, x32, rows_idx, w, y, width, ld, eps);
}

template <typename T>
void launch_plain_attention(const PlainAttnArgs& a, cudaStream_t s) {
    ProfileScope prof(KC_ATTENTION, s);
    CPM_REQUIRE(a.dk % 64 == 0 && a.dk <= PA_MAX_D && a.out_cols <= PA_MAX_D && a.hq % a.hkv == 0, "attention: head width above 512");
    launch_kernel(plain_attention_kernel<T>, dim3(ceil_div(a.tq * a.hq, PA_WARPS)), dim3(PA_WARPS * 32), 0, s, a);
}

void launch_linear_f32(const float* x, int ldx, const bf16* w, size_t w_stride, float* y, int ldy, int M, int N, int K,
                       const int4* entries, const int32_t* n_entries, int max_entries, bool x_at_y, cudaStream_t s) {
    ProfileScope prof(entries ? KC_MOE : KC_LINEAR, s);
    CPM_REQUIRE(K % 64 == 0 && ldx % 4 == 0, "linear_f32: K must be a multiple of 64");
    dim3 grid(ceil_div(N, 64), entries ? 1 : ceil_div(M, kF32Rows), entries ? max_entries : 1);
    launch_kernel(linear_f32_kernel, grid, dim3(256), 0, s, x, ldx, w, w_stride, y, ldy, M, N, K, entries, n_entries,
                  x_at_y ? 1 : 0);
}

void launch_silu_f32(const float* gu, int ld_gu, float* act, int ld_act, int rows, int ff, cudaStream_t s) {
    ProfileScope prof(KC_ROW, s);
    launch_kernel(silu_f32_kernel, dim3(rows), dim3(256), 0, s, gu, ld_gu, act, ld_act, ff);
}

#define CPM_INSTANTIATE(T)                                                                                                          \
    template void launch_embed_rows<T>(const int32_t*, const bf16*, int, float, float*, T*, int, int, const StateCheck&, cudaStream_t); \
    template void launch_qkv_norm_append<T>(const QkvNormArgs&, int, cudaStream_t);                                                 \
    template void launch_out_norm<T>(float*, T*, const T*, const MoeMix&, float, const bf16*, int, int, int, float, cudaStream_t);  \
    template void launch_norm_rows<T>(const float*, const int32_t*, const bf16*, T*, int, int, int, float, cudaStream_t);           \
    template void launch_plain_attention<T>(const PlainAttnArgs&, cudaStream_t);
CPM_INSTANTIATE(bf16)
CPM_INSTANTIATE(float)
