// Recurrences with an outer-product state (layered.cuh: ScanArgs) on the fp32 pipes.
//
// A warp holds 16 * KG rows (key channels) x 4 * (32 / KG) columns (value channels) of a head's state in registers, 16 x 4 per
// lane as pairs of rows for the packed fp32 instructions, and walks over the tokens; r, k, w, v of a few tokens at a time lie
// in shared memory, the next ones on their way.  The output of a token is a sum over the KG lanes of a column, folded so that
// a lane ends up with one column (two for KG = 2).
//
// Long portions are cut into chunks: a first walk over every chunk alone, from a zero state and without outputs, leaves what
// the chunk adds to the state and its decay, scan_link_kernel runs over the chunks and replaces that by the state each chunk
// begins with, and a second walk over all chunks side by side gives the outputs.
//
// A single token takes scan_step_kernel, which streams the state and does what surrounds the recurrence as well.
#include <algorithm>
#include <vector>

#include "row_ops.cuh"

namespace {

constexpr int kMinChunk = 64;   // fewest tokens per chunk
constexpr int TT = 8;           // tokens in shared memory

template <int KG>
struct Shape {
    static constexpr int KP = 16 * KG;          // key channels, padded
    static constexpr int VG = 32 / KG;
    static constexpr int CW = 4 * VG;           // value columns per warp
};

struct Geometry {
    int kg, warps, vblocks, kp, vp;
};
Geometry geometry(int dim, int vdim) {
    Geometry g;
    g.kg = dim <= 32 ? 2 : dim <= 64 ? 4 : dim <= 128 ? 8 : 16;
    const int cw = 4 * (32 / g.kg);
    g.warps = std::min(4, ceil_div(vdim, cw));
    g.vblocks = ceil_div(vdim, g.warps * cw);
    g.kp = 16 * g.kg;
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
    int vec_k, vec_v;        // rows of r, k, w / of v can be copied 16 bytes at a time
};

__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))), "l"(src) : "memory");
}

// `n` rows of `cols` elements of a global matrix -> dst[t][width] in shared memory as they are
template <typename E>
__device__ __forceinline__ void copy_rows(E* dst, int width, const void* src, int ld, size_t row0, int col0, int cols, int n, int vec) {
    constexpr int PER = 16 / sizeof(E);
    const E* base = static_cast<const E*>(src) + row0 * ld + col0;
    if (vec) {
        const int per = cols / PER;
        for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
            const int t = i / per, c = (i - t * per) * PER;
            copy16(dst + t * width + c, base + static_cast<size_t>(t) * ld + c);
        }
    } else {
        for (int i = threadIdx.x; i < n * cols; i += blockDim.x) {
            const int t = i / cols, c = i - t * cols;
            dst[t * width + c] = base[static_cast<size_t>(t) * ld + c];
        }
    }
}

// raw rows -> fp32, zero from column `cols` on; width is a multiple of 8
template <typename T>
__device__ __forceinline__ void convert_rows(float* dst, const T* raw, int width, int cols, int n, bool silu) {
    for (int i = threadIdx.x * 8; i < n * width; i += blockDim.x * 8) {
        float f[8];
        load_vec<8>(raw + i, f);
        if (silu) {
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = silu_of<T>(f[e]);
        }
        if (cols != width) {
            const int c = i % width;
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                if (c + e >= cols) f[e] = 0.f;
            }
        }
        store_vec<8>(dst + i, f);
    }
}

// r and k of a batch at once, and own[t] = r . (u k)
template <typename T, int KP>
__device__ __forceinline__ void convert_keys(float* sr, float* sk, const T* raw_r, const T* raw_k, const float* su, float* own, int cols) {
    // whole warps stay together: TT * KP / 8 is a multiple of 32
    for (int i = threadIdx.x * 8; i < TT * KP; i += blockDim.x * 8) {
        const int c = i % KP;
        float r[8], k[8], u[8], b = 0.f;
        load_vec<8>(raw_r + i, r);
        load_vec<8>(raw_k + i, k);
        load_vec<8>(su + c, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            if (cols != KP && c + e >= cols) r[e] = k[e] = 0.f;
            b = fmaf(r[e] * u[e], k[e], b);
        }
        store_vec<8>(sr + i, r);
        store_vec<8>(sk + i, k);
#pragma unroll
        for (int o = KP / 16; o > 0; o >>= 1) b += __shfl_xor_sync(0xffffffffu, b, o);
        if (c == 0) own[i / KP] = b;
    }
}

// Sum over the KG lanes of a column group: afterwards the lane holds column fold_column() (and the next one for KG = 2).
template <int KG>
__device__ __forceinline__ void fold(float* o, int lane) {
#pragma unroll
    for (int b = 0, n = 2; b < 2; ++b, n /= 2) {
        if ((1 << b) >= KG) break;
        const bool up = (lane >> b) & 1;
#pragma unroll
        for (int i = 0; i < n; ++i) {
            const float keep = up ? o[n + i] : o[i], give = up ? o[i] : o[n + i];
            o[i] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << b);
        }
    }
#pragma unroll
    for (int b = 4; b < KG; b *= 2) o[0] += __shfl_xor_sync(0xffffffffu, o[0], b);
}
template <int KG>
__device__ __forceinline__ int fold_column(int lane) {
    return KG == 2 ? (lane & 1) * 2 : (lane & 1) * 2 + ((lane >> 1) & 1);
}

template <typename T, int KG, bool CONST_DECAY>
struct ScanSmem {
    static constexpr int KP = Shape<KG>::KP;
    // floats: r, k, v of the tokens being walked over, two rows of key channels, a number per token, decays of two batches; then
    // the raw rows of two batches
    static size_t bytes(int vb, bool out) {
        const int keys = out ? 2 : 1;
        return sizeof(float) * (TT * (keys * KP + vb + (CONST_DECAY ? 0 : 2 * KP)) + 2 * KP + TT) + sizeof(T) * 2 * TT * (keys * KP + vb);
    }
};

// OUT: outputs from the state a chunk (or the sequence) begins with; otherwise what a chunk alone leaves behind.
template <typename T, int KG, bool CONST_DECAY, bool OUT>
__global__ void __launch_bounds__(128, 4)
scan_kernel(const ScanParams p) {
    using S_ = Shape<KG>;
    constexpr int KP = S_::KP;
    const ScanArgs& a = p.a;
    extern __shared__ __align__(16) float sm[];
    const int warps = blockDim.x >> 5, VB = warps * S_::CW;
    float* sr = sm;
    float* sk = sr + (OUT ? TT * KP : 0);
    float* sv = sk + TT * KP;
    float* sd = sv + TT * VB;                          // [KP] decay over a batch, or the bonus
    float* stot = sd + KP;                             // [KP] decay over the chunk so far
    float* own = stot + KP;                            // [TT] r . (u k)
    float* sw = own + TT;                              // two batches
    T* raw = reinterpret_cast<T*>(sw + (CONST_DECAY ? 0 : 2 * TT * KP));
    const int raw_batch = TT * ((OUT ? 2 : 1) * KP + VB);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kg = lane % KG, vg = lane / KG;
    const int h = blockIdx.x, v0 = blockIdx.y * VB;
    const int begin = blockIdx.z * p.chunk, end = min(begin + p.chunk, a.rows);
    const int c_a = warp * S_::CW + vg * 4;            // this lane's columns: c_a .. + 3
    const int vcols = min(VB, a.vdim - v0);
    // columns of the raw rows that nothing is copied to: any finite value
    for (int i = threadIdx.x; i < 2 * raw_batch; i += blockDim.x) raw[i] = from_float<T>(0.f);
    if (!CONST_DECAY) {
        for (int i = threadIdx.x; i < 2 * TT * KP; i += blockDim.x) sw[i] = 0.f;
    }
    __syncthreads();
    grid_dependency_sync();

    auto fetch = [&](int batch, int row0) {
        const int n = min(TT, end - row0);
        T* dst = raw + (batch & 1) * raw_batch;
        if (OUT) copy_rows<T>(dst, KP, a.r, a.ld_r, row0, h * a.dim, a.dim, n, p.vec_k);
        copy_rows<T>(dst + (OUT ? TT * KP : 0), KP, a.k, a.ld_k, row0, h * a.dim, a.dim, n, p.vec_k);
        copy_rows<T>(dst + (OUT ? 2 : 1) * TT * KP, VB, a.v, a.ld_v, row0, h * a.vdim + v0, vcols, n, p.vec_v);
        if (!CONST_DECAY) copy_rows<float>(sw + (batch & 1) * TT * KP, KP, a.w, a.ld_w, row0, h * a.dim, a.dim, n, p.vec_k);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, begin);

    if (OUT && !CONST_DECAY) {
        for (int c = threadIdx.x; c < KP; c += blockDim.x) sd[c] = c < a.dim ? __bfloat162float(a.bonus[h * a.dim + c]) : 0.f;
    }
    if (!OUT) {
        for (int c = threadIdx.x; c < KP; c += blockDim.x) stot[c] = 1.f;
    }
    // S[i][j]: rows k_of(i), k_of(i) + 1, column j
    f32x2 S[8][4];
    const bool chunked = p.chunk_state != nullptr;
    float* state = (chunked ? p.chunk_state + static_cast<size_t>(blockIdx.z) * a.heads * KP * p.vp : a.state) +
                   static_cast<size_t>(h) * KP * p.vp + v0 + c_a;
    auto k_of = [&](int i) { return (i >> 1) * 4 * KG + kg * 4 + (i & 1) * 2; };
    const bool zero = !OUT || (!chunked && *a.kv_len + a.kv_off == 0);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f), y = x;
        if (!zero) {
            const float* q = state + static_cast<size_t>(k_of(i)) * p.vp;
            x = *reinterpret_cast<const float4*>(q);
            y = *reinterpret_cast<const float4*>(q + p.vp);
        }
        S[i][0] = pair(x.x, y.x); S[i][1] = pair(x.y, y.y); S[i][2] = pair(x.z, y.z); S[i][3] = pair(x.w, y.w);
    }
    const float lam = CONST_DECAY ? a.decay[h] : 0.f;
    const f32x2 lam2 = pair(lam, lam);
    const int col = c_a + fold_column<KG>(lane);   // what this lane stores of a token's output
    const bool ok = OUT && (KG <= 4 || (kg & ~3) == 0) && col < vcols, ok2 = KG == 2 && ok && col + 1 < vcols;
    float* out = OUT ? a.out + static_cast<size_t>(begin) * a.ld_out + h * a.vdim + v0 + col : nullptr;
    int batch = 0;
    for (int row0 = begin; row0 < end; row0 += TT, ++batch) {
        const int n = min(TT, end - row0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();   // this batch's raw rows are here, the last batch has been walked over
        if (row0 + TT < end) fetch(batch + 1, row0 + TT);
        const T* src = raw + (batch & 1) * raw_batch;
        if (OUT && !CONST_DECAY) {
            convert_keys<T, KP>(sr, sk, src, src + TT * KP, sd, own, a.dim);
        } else {
            if (OUT) convert_rows<T>(sr, src, KP, a.dim, n, a.silu);
            convert_rows<T>(sk, src + (OUT ? TT * KP : 0), KP, a.dim, n, a.silu);
        }
        convert_rows<T>(sv, src + (OUT ? 2 : 1) * TT * KP, VB, vcols, n, a.silu);
        __syncthreads();
        const float* swb = sw + (batch & 1) * TT * KP;
        if constexpr (!OUT) {
            // keys decayed to the batch's end, so that the state is scaled once per batch
            for (int c = threadIdx.x; c < KP; c += blockDim.x) {
                float d = 1.f;
                for (int t = n - 1; t >= 0; --t) {
                    sk[t * KP + c] *= d;
                    d *= CONST_DECAY ? lam : swb[t * KP + c];
                }
                sd[c] = d;
                stot[c] *= d;
            }
            __syncthreads();
#pragma unroll
            for (int i = 0; i < 8; i += 2) {
                const ulonglong2 d = *reinterpret_cast<const ulonglong2*>(sd + k_of(i));
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    S[i][j] = mul2(S[i][j], d.x);
                    S[i + 1][j] = mul2(S[i + 1][j], d.y);
                }
            }
        }
        for (int t = 0; t < n; ++t) {
            const float4 v = *reinterpret_cast<const float4*>(sv + t * VB + c_a);
            const f32x2 vv[4] = {pair(v.x, v.x), pair(v.y, v.y), pair(v.z, v.z), pair(v.w, v.w)};
            f32x2 o[4] = {0, 0, 0, 0};
#pragma unroll
            for (int i = 0; i < 8; i += 2) {
                const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(sk + t * KP + k_of(i));
                if constexpr (!OUT) {
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        S[i][j] = fma2(k.x, vv[j], S[i][j]);
                        S[i + 1][j] = fma2(k.y, vv[j], S[i + 1][j]);
                    }
                } else {
                    const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(sr + t * KP + k_of(i));
                    ulonglong2 w = make_ulonglong2(lam2, lam2);
                    if (!CONST_DECAY) w = *reinterpret_cast<const ulonglong2*>(swb + t * KP + k_of(i));
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (!CONST_DECAY) {
                            o[j] = fma2(r.x, S[i][j], o[j]);
                            o[j] = fma2(r.y, S[i + 1][j], o[j]);
                        }
                        S[i][j] = fma2(w.x, S[i][j], mul2(k.x, vv[j]));
                        S[i + 1][j] = fma2(w.y, S[i + 1][j], mul2(k.y, vv[j]));
                        if (CONST_DECAY) {
                            o[j] = fma2(r.x, S[i][j], o[j]);
                            o[j] = fma2(r.y, S[i + 1][j], o[j]);
                        }
                    }
                }
            }
            if constexpr (OUT) {
                float f[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float2 q = unpair(o[j]);
                    f[j] = q.x + q.y;
                }
                fold<KG>(f, lane);
                if (!CONST_DECAY) {
                    const float b = own[t];
                    f[0] = fmaf(b, sv[t * VB + col], f[0]);
                    if (KG == 2) f[1] = fmaf(b, sv[t * VB + col + 1], f[1]);
                }
                if (ok) out[0] = f[0];
                if (ok2) out[1] = f[1];
                out += a.ld_out;
            }
        }
    }
    if (!OUT || !chunked) {
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const float2 f[4] = {unpair(S[i][0]), unpair(S[i][1]), unpair(S[i][2]), unpair(S[i][3])};
            float* q = state + static_cast<size_t>(k_of(i)) * p.vp;
            *reinterpret_cast<float4*>(q) = make_float4(f[0].x, f[1].x, f[2].x, f[3].x);
            *reinterpret_cast<float4*>(q + p.vp) = make_float4(f[0].y, f[1].y, f[2].y, f[3].y);
        }
    }
    if (!OUT && blockIdx.y == 0) {   // every thread wrote the channels it reads here
        float* d = p.chunk_decay + (static_cast<size_t>(blockIdx.z) * a.heads + h) * KP;
        for (int c = threadIdx.x; c < KP; c += blockDim.x) d[c] = stot[c];
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

// ---------------------------------------------------------------- one token
constexpr int STEP_THREADS = 256;
constexpr int STEP_LOADS = 16;   // 16-byte pieces of the state per thread

struct StepParams {
    ScanStepArgs a;
    int kp, vp, cols;   // state rows and columns; columns per CTA
};

// blockIdx.x: head; blockIdx.y: block of value columns (one for a time mix, whose norm is per head)
template <typename T, bool TIME_MIX>
__global__ void __launch_bounds__(STEP_THREADS)
scan_step_kernel(const StepParams p) {
    const ScanArgs& a = p.a.scan;
    extern __shared__ __align__(16) float sm[];
    float* sr = sm;                       // [kp]
    float* sk = sr + p.kp;
    float* sw = sk + p.kp;
    float* sv = sw + p.kp;                // [cols]
    float* red = sv + p.cols;             // [row groups][cols]
    __shared__ float sh[64];
    __shared__ float s_own;
    __shared__ int s_last;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, v0 = blockIdx.y * p.cols, vcols = min(p.cols, a.vdim - v0);
    const int cg = p.cols / 4, groups = STEP_THREADS / cg;
    const int c4 = (tid % cg) * 4, g = tid / cg;
    grid_dep_trigger();
    // the state was last written by the step before, which the host has waited for: it is fetched before this kernel's turn
    float* state = a.state + static_cast<size_t>(h) * p.kp * p.vp + v0 + c4;
    float4 S[STEP_LOADS];
#pragma unroll
    for (int n = 0; n < STEP_LOADS; ++n) {
        const int i = g + n * groups;
        S[n] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (g < groups && i < p.kp) S[n] = *reinterpret_cast<const float4*>(state + static_cast<size_t>(i) * p.vp);
    }
    if (TIME_MIX) {
        const int per = (a.dim + 63) / 64;
        for (int i = tid; i < p.a.rank * per; i += STEP_THREADS) {
            prefetch_l2(p.a.w2 + static_cast<size_t>(i / per) * a.heads * a.dim + h * a.dim + i % per * 64);
        }
        if (tid * 64 < a.dim) {
            prefetch_l2(p.a.w0 + h * a.dim + tid * 64);
            prefetch_l2(a.bonus + h * a.dim + tid * 64);
            prefetch_l2(p.a.norm + h * a.vdim + tid * 64);
        }
    }
    grid_dep_wait();
    if (*a.kv_len + a.kv_off == 0) {
#pragma unroll
        for (int n = 0; n < STEP_LOADS; ++n) S[n] = make_float4(0.f, 0.f, 0.f, 0.f);
    }
    // what this thread puts into shared memory, loaded before anything is stored
    auto get = [&](const void* src, int col0, int c, int cols) {
        if (c >= cols) return 0.f;
        const float v = to_float<T>(static_cast<const T*>(src)[col0 + c]);
        return TIME_MIX ? v : silu_of<T>(v);
    };
    static_assert(STEP_THREADS >= 256, "one key channel per thread");
    const float r_t = get(a.r, h * a.dim, tid, a.dim), k_t = get(a.k, h * a.dim, tid, a.dim), v_t = get(a.v, h * a.vdim + v0, tid, vcols);
    const float x_t = TIME_MIX && tid < p.a.rank ? to_float<T>(static_cast<const T*>(p.a.inner)[tid]) : 0.f;
    const float z_t = TIME_MIX && tid < vcols ? to_float<T>(static_cast<const T*>(p.a.gate)[h * a.vdim + tid]) : 0.f;
    if (tid < p.kp) {
        sr[tid] = r_t;
        sk[tid] = k_t;
    }
    if (tid < p.cols) sv[tid] = v_t;
    for (int c = tid + STEP_THREADS; c < p.cols; c += STEP_THREADS) sv[c] = get(a.v, h * a.vdim + v0, c, vcols);
    if (TIME_MIX) {
        float* inner = red;               // [rank], before red is needed
        if (tid < p.a.rank) inner[tid] = tanhf(x_t);
        for (int k = tid + STEP_THREADS; k < p.a.rank; k += STEP_THREADS) inner[k] = tanhf(to_float<T>(static_cast<const T*>(p.a.inner)[k]));
        __syncthreads();
        // kp divides the threads: each channel's sum over the rank in parts
        float* part = red + p.a.rank;     // [STEP_THREADS]
        const int c = tid % p.kp, parts = STEP_THREADS / p.kp, channels = a.heads * a.dim;
        float z = 0.f;
        if (c < a.dim) {
            const bf16* w = p.a.w2 + h * a.dim + c;
#pragma unroll 16
            for (int k = tid / p.kp; k < p.a.rank; k += parts) z = fmaf(__bfloat162float(__ldg(w + static_cast<size_t>(k) * channels)), inner[k], z);
        }
        part[tid] = z;
        __syncthreads();
        if (tid < a.dim) {
            z = __bfloat162float(__ldg(p.a.w0 + h * a.dim + tid));
            for (int n = 0; n < parts; ++n) z += part[n * p.kp + tid];
            sw[tid] = expf(-expf(z));
        }
        if (tid >= a.dim && tid < p.kp) sw[tid] = 0.f;
        if (warp == 0) {
            float b = 0.f;
            for (int c = lane; c < a.dim; c += 32) b += sr[c] * __bfloat162float(a.bonus[h * a.dim + c]) * sk[c];
            b = warp_sum(b);
            if (lane == 0) s_own = b;
        }
    }
    __syncthreads();
    const float lam = TIME_MIX ? 0.f : a.decay[h];
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (g < groups) {
        const float4 v = *reinterpret_cast<const float4*>(sv + c4);
#pragma unroll
        for (int n = 0; n < STEP_LOADS; ++n) {
            const int i = g + n * groups;
            if (i < p.kp) {
                const float r = sr[i], k = sk[i], w = TIME_MIX ? sw[i] : lam;
                if (TIME_MIX) {
                    o.x = fmaf(r, S[n].x, o.x); o.y = fmaf(r, S[n].y, o.y); o.z = fmaf(r, S[n].z, o.z); o.w = fmaf(r, S[n].w, o.w);
                }
                S[n].x = fmaf(w, S[n].x, k * v.x); S[n].y = fmaf(w, S[n].y, k * v.y);
                S[n].z = fmaf(w, S[n].z, k * v.z); S[n].w = fmaf(w, S[n].w, k * v.w);
                if (!TIME_MIX) {
                    o.x = fmaf(r, S[n].x, o.x); o.y = fmaf(r, S[n].y, o.y); o.z = fmaf(r, S[n].z, o.z); o.w = fmaf(r, S[n].w, o.w);
                }
                *reinterpret_cast<float4*>(state + static_cast<size_t>(i) * p.vp) = S[n];
            }
        }
        *reinterpret_cast<float4*>(red + g * p.cols + c4) = o;
    }
    __syncthreads();
    const T* gate = static_cast<const T*>(p.a.gate);
    T* out = static_cast<T*>(p.a.out);
    auto gated = [&](float v, float z, float w, float rs) {
        const float s = 1.f / (1.f + expf(-z));
        return v * rs * w * (TIME_MIX ? z * s : s) * p.a.scale;
    };
    if (TIME_MIX) {
        float ss = 0.f;
        for (int c = tid; c < vcols; c += STEP_THREADS) {
            float v = s_own * sv[c];
            for (int n = 0; n < groups; ++n) v += red[n * p.cols + c];
            sv[c] = v;
            ss += v * v;
        }
        const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / a.vdim + p.a.eps);
        for (int c = tid; c < vcols; c += STEP_THREADS) {
            const int at = h * a.vdim + c;
            out[at] = from_float<T>(gated(sv[c], c == tid ? z_t : to_float<T>(gate[at]), __bfloat162float(__ldg(p.a.norm + at)), rs));
        }
    } else {
        for (int c = tid; c < vcols; c += STEP_THREADS) {
            float v = 0.f;
            for (int n = 0; n < groups; ++n) v += red[n * p.cols + c];
            a.out[h * a.vdim + v0 + c] = v;
        }
        // the CTA counted last has everything for the norm over all heads
        __threadfence();
        __syncthreads();
        if (tid == 0) {
            const int last = atomicAdd(p.a.ticket, 1) == static_cast<int>(gridDim.x * gridDim.y) - 1;
            if (last) *p.a.ticket = 0;
            s_last = last;
        }
        __syncthreads();
        if (s_last == 0) return;
        __threadfence();
        const int nv = a.heads * a.vdim;
        float ss = 0.f;
        if (nv % 8 == 0 && nv <= STEP_THREADS * 16 && reinterpret_cast<uintptr_t>(gate) % 16 == 0 && reinterpret_cast<uintptr_t>(out) % 16 == 0) {
            float f[2][8], z[2][8], w[2][8];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int c = (tid + n * STEP_THREADS) * 8;
                if (c >= nv) continue;
                const float4 x = __ldcg(reinterpret_cast<const float4*>(a.out + c)), y = __ldcg(reinterpret_cast<const float4*>(a.out + c + 4));
                f[n][0] = x.x; f[n][1] = x.y; f[n][2] = x.z; f[n][3] = x.w;
                f[n][4] = y.x; f[n][5] = y.y; f[n][6] = y.z; f[n][7] = y.w;
                load_vec<8>(gate + c, z[n]);
                load_vec<8>(p.a.norm + c, w[n]);
#pragma unroll
                for (int e = 0; e < 8; ++e) ss += f[n][e] * f[n][e];
            }
            const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / nv + p.a.eps);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int c = (tid + n * STEP_THREADS) * 8;
                if (c >= nv) continue;
#pragma unroll
                for (int e = 0; e < 8; ++e) f[n][e] = gated(f[n][e], z[n][e], w[n][e], rs);
                store_vec<8>(out + c, f[n]);
            }
            return;
        }
        for (int c = tid; c < nv; c += STEP_THREADS) {
            const float v = __ldcg(a.out + c);
            ss += v * v;
        }
        const float rs = rsqrtf(block_sum2(ss, 0.f, sh).x / nv + p.a.eps);
        for (int c = tid; c < nv; c += STEP_THREADS) {
            out[c] = from_float<T>(gated(__ldcg(a.out + c), to_float<T>(gate[c]), __bfloat162float(p.a.norm[c]), rs));
        }
    }
}

template <typename T, int KG, bool CONST_DECAY>
void run_scan(const ScanParams& base, const Geometry& g, cudaStream_t s) {
    using M = ScanSmem<T, KG, CONST_DECAY>;
    ScanParams p = base;
    const ScanArgs& a = p.a;
    const int vb = g.warps * Shape<KG>::CW;
    static bool configured = false;
    if (!configured) {
        CUDA_CHECK(cudaFuncSetAttribute(scan_kernel<T, KG, CONST_DECAY, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
        CUDA_CHECK(cudaFuncSetAttribute(scan_kernel<T, KG, CONST_DECAY, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
        configured = true;
    }
    const dim3 block(g.warps * 32);
    if (a.rows > kMinChunk) {
        // the shortest chunks whose CTAs all run at once (128 registers: 16 warps per SM)
        const long long slots = static_cast<long long>(runtime().num_sms) * (16 / g.warps);
        p.chunk = kMinChunk;
        while (p.chunk < 8 * kMinChunk && static_cast<long long>(a.heads) * g.vblocks * ceil_div(a.rows, p.chunk) > slots) p.chunk += TT;
        p.chunks = ceil_div(a.rows, p.chunk);
        launch_kernel(scan_kernel<T, KG, CONST_DECAY, false>, dim3(a.heads, g.vblocks, p.chunks), block, M::bytes(vb, false), s, p);
        const size_t n4 = static_cast<size_t>(a.heads) * g.kp * g.vp / 4;
        launch_kernel(scan_link_kernel, dim3(static_cast<unsigned>((n4 + 127) / 128)), dim3(128), 0, s, p, g.kp);
    } else {
        p.chunk = a.rows;
        p.chunks = 1;
        p.chunk_state = p.chunk_decay = nullptr;
    }
    launch_kernel(scan_kernel<T, KG, CONST_DECAY, true>, dim3(a.heads, g.vblocks, p.chunks), block, M::bytes(vb, true), s, p);
}

}  // namespace

bool scan_fits(int dim, int vdim) { return dim >= 1 && dim <= 256 && vdim >= 1 && vdim <= 512; }

size_t scan_state_floats(int heads, int dim, int vdim) {
    const Geometry g = geometry(dim, vdim);
    return static_cast<size_t>(heads) * g.kp * g.vp;
}

size_t scan_workspace_floats(int heads, int dim, int vdim, int rows) {
    const Geometry g = geometry(dim, vdim);
    return static_cast<size_t>(ceil_div(rows, kMinChunk)) * heads * g.kp * (g.vp + 1);
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
    auto aligned = [&](const void* q, int ld, int cols, int es) {
        return reinterpret_cast<uintptr_t>(q) % 16 == 0 && static_cast<size_t>(ld) * es % 16 == 0 && static_cast<size_t>(cols) * es % 16 == 0;
    };
    p.vec_k = aligned(a.r, a.ld_r, a.dim, sizeof(T)) && aligned(a.k, a.ld_k, a.dim, sizeof(T)) && (a.w == nullptr || aligned(a.w, a.ld_w, a.dim, 4));
    p.vec_v = aligned(a.v, a.ld_v, a.vdim, sizeof(T));
    p.chunk_state = a.ws;
    p.chunk_decay = a.ws + static_cast<size_t>(ceil_div(a.rows, kMinChunk)) * a.heads * g.kp * g.vp;
    auto run = [&](auto kg) {
        constexpr int KG = decltype(kg)::value;
        if (a.decay != nullptr) run_scan<T, KG, true>(p, g, s);
        else run_scan<T, KG, false>(p, g, s);
    };
    switch (g.kg) {
        case 2: run(std::integral_constant<int, 2>()); break;
        case 4: run(std::integral_constant<int, 4>()); break;
        case 8: run(std::integral_constant<int, 8>()); break;
        default: run(std::integral_constant<int, 16>()); break;
    }
}
void upload_transposed(const void* src, int rows, int cols, bf16* dst, cudaStream_t s) {
    const size_t n = static_cast<size_t>(rows) * cols;
    std::vector<bf16> a(n), b(n);
    CUDA_CHECK(cudaMemcpyAsync(a.data(), src, n * sizeof(bf16), cudaMemcpyDefault, s));
    CUDA_CHECK(cudaStreamSynchronize(s));
    for (int r = 0; r < rows; ++r) {
        for (int c = 0; c < cols; ++c) b[static_cast<size_t>(c) * rows + r] = a[static_cast<size_t>(r) * cols + c];
    }
    CUDA_CHECK(cudaMemcpyAsync(dst, b.data(), n * sizeof(bf16), cudaMemcpyHostToDevice, s));
    CUDA_CHECK(cudaStreamSynchronize(s));
}

bool scan_step_fits(int dim, int vdim, bool time_mix) {
    const Geometry g = geometry(dim, vdim);
    return !time_mix || static_cast<long long>(g.kp) * g.vp <= 4LL * STEP_LOADS * STEP_THREADS;
}

template <typename T>
void launch_scan_step(const ScanStepArgs& a, cudaStream_t s) {
    ProfileScope prof(KC_SCAN, s);
    const ScanArgs& sc = a.scan;
    const bool time_mix = sc.bonus != nullptr;
    CPM_REQUIRE(sc.rows == 1 && scan_fits(sc.dim, sc.vdim) && scan_step_fits(sc.dim, sc.vdim, time_mix), "recurrence step: unsupported sizes");
    const Geometry g = geometry(sc.dim, sc.vdim);
    StepParams p;
    p.a = a;
    p.kp = g.kp; p.vp = g.vp; p.cols = g.vp;
    int blocks = 1;
    if (!time_mix) {
        while (p.cols % 8 == 0 && (p.kp * p.cols > 4 * STEP_LOADS * STEP_THREADS || (p.cols >= 64 && sc.heads * blocks * 2 <= runtime().num_sms))) {
            p.cols /= 2;
            blocks *= 2;
        }
    }
    // columns beyond the real ones need no CTA: their state stays zero
    const dim3 grid(sc.heads, ceil_div(sc.vdim, p.cols));
    const int groups = STEP_THREADS / (p.cols / 4);
    CPM_REQUIRE(groups >= 1 && groups * STEP_LOADS >= p.kp, "recurrence step: unsupported sizes");
    const size_t smem = sizeof(float) * (3 * p.kp + p.cols + std::max(groups * p.cols, a.rank + STEP_THREADS));
    if (time_mix) launch_kernel(scan_step_kernel<T, true>, grid, dim3(STEP_THREADS), smem, s, p);
    else launch_kernel(scan_step_kernel<T, false>, grid, dim3(STEP_THREADS), smem, s, p);
}
template void launch_scan_step<bf16>(const ScanStepArgs&, cudaStream_t);
template void launch_scan_step<float>(const ScanStepArgs&, cudaStream_t);
template void launch_scan<bf16>(const ScanArgs&, cudaStream_t);
template void launch_scan<float>(const ScanArgs&, cudaStream_t);
