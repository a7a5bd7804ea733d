// Recurrences with an outer-product state (layered.cuh: ScanArgs) on the fp32 pipes.
//
// A warp holds 8 * KG rows (key channels) x 8 * (32 / KG) columns (value channels) of a head's state in registers, 8 x 8 per
// lane, and walks over the tokens; r, k, w, v of a few tokens at a time lie in shared memory.  The output of a token is a sum
// over the KG lanes of a column, folded so that every lane ends up with one column.
//
// Long portions are cut into chunks: scan_chunk_kernel adds up what every chunk alone would leave in the state (and its
// decay), scan_link_kernel runs over the chunks and replaces that by the state each chunk begins with, and scan_kernel then
// walks all chunks side by side.
#include <algorithm>

#include "row_ops.cuh"

namespace {

constexpr int kChunk = 64;   // tokens per chunk

template <int KG>
struct Shape {
    static constexpr int KP = 8 * KG;           // key channels, padded
    static constexpr int VG = 32 / KG;
    static constexpr int CW = 8 * VG;           // value columns per warp
    static constexpr int TT = KG >= 32 ? 8 : 16;  // tokens in shared memory
};

struct Geometry {
    int kg, warps, vblocks, kp, vp;
};
Geometry geometry(int dim, int vdim) {
    Geometry g;
    g.kg = dim <= 32 ? 4 : dim <= 64 ? 8 : dim <= 128 ? 16 : 32;
    const int cw = 8 * (32 / g.kg);
    g.warps = std::min(4, ceil_div(vdim, cw));
    g.vblocks = ceil_div(vdim, g.warps * cw);
    g.kp = 8 * g.kg;
    g.vp = g.vblocks * g.warps * cw;
    return g;
}

struct ScanParams {
    ScanArgs a;
    int vp;                  // columns of a state row
    int chunk;               // tokens per CTA in the token direction
    float* chunk_state;      // [chunks][heads][kp][vp]; null: the walk starts from and ends in a.state
    float* chunk_decay;      // [chunks][heads][kp]
    int chunks;
};

// tokens row0 .. row0 + n of one operand -> dst[t][width], zero where there is none
template <typename T>
__device__ __forceinline__ void stage(const void* src, int ld, int col0, int cols, int row0, int n, int width, bool silu, float* dst) {
    for (int i = threadIdx.x; i < n * width; i += blockDim.x) {
        const int t = i / width, c = i - t * width;
        float v = 0.f;
        if (c < cols) {
            v = to_float<T>(static_cast<const T*>(src)[static_cast<size_t>(row0 + t) * ld + col0 + c]);
            if (silu) v = silu_f32(v);
        }
        dst[i] = v;
    }
}

__device__ __forceinline__ void lds8(const float* p, int second, float* f) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + second);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

// Sum over the KG lanes of a column group.  Afterwards the lane holds the sums of columns fold_column() (+ 1 for KG = 4).
template <int KG>
__device__ __forceinline__ void fold(float* o, int lane) {
#pragma unroll
    for (int b = 0, n = 4; b < 3; ++b, n /= 2) {
        if ((1 << b) >= KG) break;
        const bool up = (lane >> b) & 1;
#pragma unroll
        for (int i = 0; i < n; ++i) {
            const float keep = up ? o[n + i] : o[i], give = up ? o[i] : o[n + i];
            o[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << b);
        }
    }
#pragma unroll
    for (int b = 8; b < KG; b *= 2) o[0] += __shfl_xor_sync(0xffffffffu, o[0], b);
}

template <typename T, int KG, bool CONST_DECAY>
__global__ void __launch_bounds__(128)
scan_kernel(const ScanParams p) {
    using S_ = Shape<KG>;
    constexpr int KP = S_::KP, TT = S_::TT;
    const ScanArgs& a = p.a;
    extern __shared__ float sm[];
    const int warps = blockDim.x >> 5, VB = warps * S_::CW;
    float* sr = sm;
    float* sk = sr + TT * KP;
    float* sw = sk + TT * KP;                          // no decays for CONST_DECAY
    float* sv = sw + (CONST_DECAY ? 0 : TT * KP);
    float* sb = sv + TT * VB;                          // bonus of a token: r . (u k)
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kg = lane % KG, vg = lane / KG;
    const int h = blockIdx.x, v0 = blockIdx.y * VB;
    const int begin = blockIdx.z * p.chunk, end = min(begin + p.chunk, a.rows);
    const int c_a = warp * S_::CW + vg * 4;            // this lane's columns: c_a .. + 3 and c_a + 4 VG .. + 3
    grid_dependency_sync();

    float S[8][8];
    float* state = (p.chunk_state != nullptr ? p.chunk_state + static_cast<size_t>(blockIdx.z) * a.heads * KP * p.vp : a.state) +
                   static_cast<size_t>(h) * KP * p.vp + v0 + c_a;
    auto k_of = [&](int i) { return (i >> 2) * 4 * KG + kg * 4 + (i & 3); };
    const bool fresh = p.chunk_state == nullptr && *a.kv_len + a.kv_off == 0;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        if (fresh) {
#pragma unroll
            for (int j = 0; j < 8; ++j) S[i][j] = 0.f;
        } else {
            const float* q = state + static_cast<size_t>(k_of(i)) * p.vp;
            const float4 x = *reinterpret_cast<const float4*>(q), y = *reinterpret_cast<const float4*>(q + 4 * S_::VG);
            S[i][0] = x.x; S[i][1] = x.y; S[i][2] = x.z; S[i][3] = x.w;
            S[i][4] = y.x; S[i][5] = y.y; S[i][6] = y.z; S[i][7] = y.w;
        }
    }
    const float lam = CONST_DECAY ? a.decay[h] : 0.f;
    for (int row0 = begin; row0 < end; row0 += TT) {
        const int n = min(TT, end - row0);
        __syncthreads();
        stage<T>(a.r, a.ld_r, h * a.dim, a.dim, row0, n, KP, a.silu, sr);
        stage<T>(a.k, a.ld_k, h * a.dim, a.dim, row0, n, KP, a.silu, sk);
        stage<T>(a.v, a.ld_v, h * a.vdim + v0, a.vdim - v0, row0, n, VB, a.silu, sv);
        if (!CONST_DECAY) stage<float>(a.w, a.ld_w, h * a.dim, a.dim, row0, n, KP, false, sw);
        __syncthreads();
        if (!CONST_DECAY) {
            for (int t = warp; t < n; t += warps) {
                float b = 0.f;
                for (int c = lane; c < a.dim; c += 32) b += sr[t * KP + c] * __bfloat162float(a.bonus[h * a.dim + c]) * sk[t * KP + c];
                b = warp_sum(b);
                if (lane == 0) sb[t] = b;
            }
            __syncthreads();
        }
        for (int t = 0; t < n; ++t) {
            float r[8], k[8], v[8], o[8];
            lds8(sr + t * KP + kg * 4, 4 * KG, r);
            lds8(sk + t * KP + kg * 4, 4 * KG, k);
            lds8(sv + t * VB + c_a, 4 * S_::VG, v);
            if (CONST_DECAY) {
#pragma unroll
                for (int i = 0; i < 8; ++i) {
#pragma unroll
                    for (int j = 0; j < 8; ++j) S[i][j] = fmaf(lam, S[i][j], k[i] * v[j]);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) o[j] = r[0] * S[0][j];
#pragma unroll
            for (int i = 1; i < 8; ++i) {
#pragma unroll
                for (int j = 0; j < 8; ++j) o[j] = fmaf(r[i], S[i][j], o[j]);
            }
            if (!CONST_DECAY) {
                float w[8];
                lds8(sw + t * KP + kg * 4, 4 * KG, w);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
#pragma unroll
                    for (int j = 0; j < 8; ++j) S[i][j] = fmaf(w[i], S[i][j], k[i] * v[j]);
                }
            }
            fold<KG>(o, lane);
            if (KG <= 8 || (lane & (KG - 1) & ~7) == 0) {
                const int j0 = KG == 4 ? (lane & 1) * 4 + ((lane >> 1) & 1) * 2 : (lane & 1) * 4 + ((lane >> 1) & 1) * 2 + ((lane >> 2) & 1);
#pragma unroll
                for (int e = 0; e < (KG == 4 ? 2 : 1); ++e) {
                    const int j = j0 + e, c = c_a + (j >> 2) * 4 * S_::VG + (j & 3);
                    float val = o[e];
                    if (!CONST_DECAY) val += sb[t] * sv[t * VB + c];
                    if (v0 + c < a.vdim) a.out[static_cast<size_t>(row0 + t) * a.ld_out + h * a.vdim + v0 + c] = val;
                }
            }
        }
    }
    if (p.chunk_state == nullptr) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            float* q = state + static_cast<size_t>(k_of(i)) * p.vp;
            *reinterpret_cast<float4*>(q) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
            *reinterpret_cast<float4*>(q + 4 * S_::VG) = make_float4(S[i][4], S[i][5], S[i][6], S[i][7]);
        }
    }
}

// What the tokens of one chunk leave in a state that was zero before it, and the decay over the chunk.
template <typename T, int KG, bool CONST_DECAY>
__global__ void __launch_bounds__(128)
scan_chunk_kernel(const ScanParams p) {
    using S_ = Shape<KG>;
    constexpr int KP = S_::KP, TT = S_::TT;
    const ScanArgs& a = p.a;
    extern __shared__ float sm[];
    const int warps = blockDim.x >> 5, VB = warps * S_::CW;
    float* sk = sm;
    float* sw = sk + TT * KP;
    float* sv = sw + (CONST_DECAY ? 0 : TT * KP);
    float* carry = sv + TT * VB;                       // decay from the tokens already added (later ones) to the chunk's end
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kg = lane % KG, vg = lane / KG;
    const int h = blockIdx.x, v0 = blockIdx.y * VB;
    const int begin = blockIdx.z * p.chunk, end = min(begin + p.chunk, a.rows);
    const int c_a = warp * S_::CW + vg * 4;
    grid_dependency_sync();
    const float lam = CONST_DECAY ? a.decay[h] : 0.f;
    for (int c = threadIdx.x; c < KP; c += blockDim.x) carry[c] = 1.f;
    float S[8][8] = {};
    for (int row1 = end; row1 > begin; row1 -= TT) {
        const int row0 = max(begin, row1 - TT), n = row1 - row0;
        __syncthreads();
        stage<T>(a.k, a.ld_k, h * a.dim, a.dim, row0, n, KP, a.silu, sk);
        stage<T>(a.v, a.ld_v, h * a.vdim + v0, a.vdim - v0, row0, n, VB, a.silu, sv);
        if (!CONST_DECAY) stage<float>(a.w, a.ld_w, h * a.dim, a.dim, row0, n, KP, false, sw);
        __syncthreads();
        for (int c = threadIdx.x; c < KP; c += blockDim.x) {
            float d = carry[c];
            for (int t = n - 1; t >= 0; --t) {
                sk[t * KP + c] *= d;
                d *= CONST_DECAY ? lam : sw[t * KP + c];
            }
            carry[c] = d;
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            float k[8], v[8];
            lds8(sk + t * KP + kg * 4, 4 * KG, k);
            lds8(sv + t * VB + c_a, 4 * S_::VG, v);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
#pragma unroll
                for (int j = 0; j < 8; ++j) S[i][j] = fmaf(k[i], v[j], S[i][j]);
            }
        }
    }
    float* state = p.chunk_state + (static_cast<size_t>(blockIdx.z) * a.heads + h) * KP * p.vp + v0 + c_a;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        float* q = state + static_cast<size_t>((i >> 2) * 4 * KG + kg * 4 + (i & 3)) * p.vp;
        *reinterpret_cast<float4*>(q) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        *reinterpret_cast<float4*>(q + 4 * S_::VG) = make_float4(S[i][4], S[i][5], S[i][6], S[i][7]);
    }
    if (blockIdx.y == 0) {
        for (int c = threadIdx.x; c < KP; c += blockDim.x) p.chunk_decay[(static_cast<size_t>(blockIdx.z) * a.heads + h) * KP + c] = carry[c];
    }
}

// chunk_state[c] becomes the state chunk c begins with; a.state the state after the last one.  One thread per four columns.
__global__ void scan_link_kernel(const ScanParams p, int kp) {
    grid_dependency_sync();
    const ScanArgs& a = p.a;
    const size_t n4 = static_cast<size_t>(a.heads) * kp * p.vp / 4, i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x;
    if (i >= n4) return;
    const size_t hk = i / (p.vp / 4);
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (*a.kv_len + a.kv_off != 0) s = reinterpret_cast<const float4*>(a.state)[i];
    float4* x = reinterpret_cast<float4*>(p.chunk_state) + i;
    const float* d = p.chunk_decay + hk;
    constexpr int B = 8;
    for (int c0 = 0; c0 < p.chunks; c0 += B) {
        float4 add[B];
        float dec[B];
#pragma unroll
        for (int c = 0; c < B; ++c) {
            if (c0 + c >= p.chunks) break;
            add[c] = x[(c0 + c) * n4];
            dec[c] = d[static_cast<size_t>(c0 + c) * a.heads * kp];
        }
#pragma unroll
        for (int c = 0; c < B; ++c) {
            if (c0 + c >= p.chunks) break;
            x[(c0 + c) * n4] = s;
            s.x = fmaf(dec[c], s.x, add[c].x);
            s.y = fmaf(dec[c], s.y, add[c].y);
            s.z = fmaf(dec[c], s.z, add[c].z);
            s.w = fmaf(dec[c], s.w, add[c].w);
        }
    }
    reinterpret_cast<float4*>(a.state)[i] = s;
}

template <typename T, int KG, bool CONST_DECAY>
void run_scan(const ScanParams& base, const Geometry& g, cudaStream_t s) {
    using S_ = Shape<KG>;
    ScanParams p = base;
    const ScanArgs& a = p.a;
    const int vb = g.warps * S_::CW;
    const size_t smem = sizeof(float) * (S_::TT * ((CONST_DECAY ? 2 : 3) * S_::KP + vb) + std::max<int>(S_::TT, S_::KP));
    static bool configured = false;
    if (!configured) {
        CUDA_CHECK(cudaFuncSetAttribute(scan_kernel<T, KG, CONST_DECAY>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
        CUDA_CHECK(cudaFuncSetAttribute(scan_chunk_kernel<T, KG, CONST_DECAY>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024));
        configured = true;
    }
    const dim3 block(g.warps * 32);
    if (a.rows > kChunk) {
        p.chunk = kChunk;
        p.chunks = ceil_div(a.rows, kChunk);
        launch_kernel(scan_chunk_kernel<T, KG, CONST_DECAY>, dim3(a.heads, g.vblocks, p.chunks), block, smem, s, p);
        const size_t n4 = static_cast<size_t>(a.heads) * g.kp * g.vp / 4;
        launch_kernel(scan_link_kernel, dim3(static_cast<unsigned>((n4 + 127) / 128)), dim3(128), 0, s, p, g.kp);
    } else {
        p.chunk = a.rows;
        p.chunks = 1;
        p.chunk_state = p.chunk_decay = nullptr;
    }
    launch_kernel(scan_kernel<T, KG, CONST_DECAY>, dim3(a.heads, g.vblocks, p.chunks), block, smem, s, p);
}

}  // namespace

bool scan_fits(int dim, int vdim) { return dim >= 1 && dim <= 256 && vdim >= 1 && vdim <= 512; }

size_t scan_state_floats(int heads, int dim, int vdim) {
    const Geometry g = geometry(dim, vdim);
    return static_cast<size_t>(heads) * g.kp * g.vp;
}

size_t scan_workspace_floats(int heads, int dim, int vdim, int rows) {
    const Geometry g = geometry(dim, vdim);
    return static_cast<size_t>(ceil_div(rows, kChunk)) * heads * g.kp * (g.vp + 1);
}

template <typename T>
void launch_scan(const ScanArgs& a, cudaStream_t s) {
    ProfileScope prof(KC_SCAN, s);
    CPM_REQUIRE(scan_fits(a.dim, a.vdim) && a.rows >= 1, "recurrence: head widths must be at most 256 (keys) and 512 (values)");
    CPM_REQUIRE((a.w != nullptr) != (a.decay != nullptr) && (a.w != nullptr) == (a.bonus != nullptr), "recurrence: decays per channel with a bonus, or per head");
    const Geometry g = geometry(a.dim, a.vdim);
    ScanParams p;
    p.a = a;
    p.vp = g.vp;
    p.chunk = p.chunks = 0;
    p.chunk_state = a.ws;
    p.chunk_decay = a.ws + static_cast<size_t>(ceil_div(a.rows, kChunk)) * a.heads * g.kp * g.vp;
    auto run = [&](auto kg) {
        constexpr int KG = decltype(kg)::value;
        if (a.decay != nullptr) run_scan<T, KG, true>(p, g, s);
        else run_scan<T, KG, false>(p, g, s);
    };
    switch (g.kg) {
        case 4: run(std::integral_constant<int, 4>()); break;
        case 8: run(std::integral_constant<int, 8>()); break;
        case 16: run(std::integral_constant<int, 16>()); break;
        default: run(std::integral_constant<int, 32>()); break;
    }
}
template void launch_scan<bf16>(const ScanArgs&, cudaStream_t);
template void launch_scan<float>(const ScanArgs&, cudaStream_t);
