// Mixture of experts for layered models (layered.cuh): fp32 router with grouped choice and identity experts, the layout
// of the chosen rows, and the grouped expert products on the tensor cores.
//
//   route    fp32 logits (8 rows x 8 outputs per warp, rows staged in shared memory); the CTA counted last of a block of rows
//            picks its rows' experts; the CTA counted last of the launch cuts every expert's rows into groups
//   gather   each chosen row's input is copied to its place, expert after expert
//   gate/up  grouped tcgen05 product, SwiGLU in the epilogue
//   down     grouped tcgen05 product
// The weighted sum over a token's experts, the identity part and the output norm are one kernel (out_norm_kernel).
#include <algorithm>
#include <type_traits>

#include "gemm_common.cuh"
#include "layered.cuh"
#include "ptx.cuh"

namespace {

// ---------------------------------------------------------------- router
constexpr int RT_WARPS = 8;

struct RouteArgs {
    const float* x;
    const bf16* w;
    const float* correction;
    int rows, ld;
    int outputs, experts, top, groups, keep;
    float scale;
    int tile, direct;
    MoeBuffers b;
};

// Largest of n values in shared memory, lowest index first among equals: values as integers of the same order, so one
// warp-wide integer maximum and one minimum over the indices do.
__device__ __forceinline__ uint32_t ordered_bits(float v) {
    const uint32_t u = __float_as_uint(v + 0.f);   // -0 counts as +0
    return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}
__device__ __forceinline__ int argmax_of(const float* a, int n, int lane) {
    uint32_t v = 0u;
    int i = 0x7fffffff;
    for (int e = lane; e < n; e += 32) {
        const uint32_t u = ordered_bits(a[e]);
        if (u > v) { v = u; i = e; }
    }
    const uint32_t m = __reduce_max_sync(0xffffffffu, v);
    return __reduce_min_sync(0xffffffffu, v == m ? i : 0x7fffffff);
}

// The experts of one row, one warp.  sc: 2 * outputs + 2 * groups floats of scratch.  ALONE: the launch has one row, whose
// experts' row groups are written here as well.
template <bool ALONE>
__device__ void choose_experts(const RouteArgs& a, int row, float* sc, int lane) {
    const int n = a.outputs;
    float* score = sc;
    float* choice = sc + n;
    float* group = sc + 2 * n;
    float* kept = group + a.groups;
    const float* z = a.b.z + static_cast<size_t>(row) * n;
    float m = -INFINITY;
    for (int e = lane; e < n; e += 32) {
        score[e] = __ldcg(z + e);
        m = fmaxf(m, score[e]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    float sum = 0.f;
    for (int e = lane; e < n; e += 32) {
        score[e] = expf(score[e] - m);
        sum += score[e];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    for (int e = lane; e < n; e += 32) {
        score[e] = score[e] / sum;
        choice[e] = a.correction != nullptr ? score[e] + a.correction[e] : score[e];
    }
    __syncwarp();
    if (a.keep < a.groups) {
        const int per = n / a.groups;
        for (int g = lane; g < a.groups; g += 32) {
            float v = choice[g * per];
            for (int e = 1; e < per; ++e) v = fmaxf(v, choice[g * per + e]);
            group[g] = v;
            kept[g] = 0.f;
        }
        __syncwarp();
        for (int k = 0; k < a.keep; ++k) {
            const int g = argmax_of(group, a.groups, lane);
            __syncwarp();
            if (lane == 0) { kept[g] = 1.f; group[g] = -INFINITY; }
            __syncwarp();
        }
        for (int e = lane; e < n; e += 32) {
            if (kept[e / per] == 0.f) choice[e] = -INFINITY;
        }
        __syncwarp();
    }
    int mine = -1;       // lane k holds choice k
    float s_mine = 0.f;
    for (int k = 0; k < a.top; ++k) {
        const int e = argmax_of(choice, n, lane);
        if (lane == k) { mine = e; s_mine = score[e]; }
        __syncwarp();
        if (lane == 0) choice[e] = -INFINITY;
        __syncwarp();
    }
    float total = s_mine;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
    const float weight = s_mine / (total + 1e-20f) * a.scale;
    float idw = (mine >= a.experts) ? weight : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) idw += __shfl_xor_sync(0xffffffffu, idw, o);
    if (lane < a.top) {
        const size_t i = static_cast<size_t>(row) * a.top + lane;
        a.b.expert[i] = mine;
        a.b.weight[i] = weight;
        a.b.rank[i] = (!ALONE && mine < a.experts) ? atomicAdd(&a.b.counts[mine], 1) : 0;
    }
    if constexpr (ALONE) {
        const bool real = lane < a.top && mine < a.experts;
        const uint32_t reals = __ballot_sync(0xffffffffu, real);
        const int at = __popc(reals & ((1u << lane) - 1u));
        if (real) {
            a.b.offset[mine] = at;
            a.b.entries[at] = make_int4(mine, a.direct ? 0 : at, at, 1);
        }
        if (lane == 0) *a.b.n_entries = __popc(reals);
    }
    if (lane == 0) a.b.id_weight[row] = idw;
    __syncwarp();
}

// Rows of every expert one after the other, cut into groups of at most `tile` rows (as even as possible); one warp.
__device__ void lay_out_rows(const RouteArgs& a, int lane) {
    int row0 = 0, entry0 = 0;
    for (int e0 = 0; e0 < a.experts; e0 += 32) {
        const int e = e0 + lane;
        const int cnt = (e < a.experts) ? __ldcg(&a.b.counts[e]) : 0;
        const int ne = (cnt + a.tile - 1) / a.tile;
        int rows_to = cnt, entries_to = ne;   // inclusive prefix sums
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int r = __shfl_up_sync(0xffffffffu, rows_to, o), n = __shfl_up_sync(0xffffffffu, entries_to, o);
            if (lane >= o) { rows_to += r; entries_to += n; }
        }
        if (e < a.experts) {
            const int first = row0 + rows_to - cnt;
            a.b.offset[e] = first;
            a.b.counts[e] = 0;
            for (int k = 0; k < ne; ++k) {
                const int b = static_cast<int>(static_cast<long long>(cnt) * k / ne), c = static_cast<int>(static_cast<long long>(cnt) * (k + 1) / ne);
                const int at = entry0 + entries_to - ne + k;
                if (at < kMoeMaxEntries) a.b.entries[at] = make_int4(e, a.direct ? 0 : first + b, first + b, c - b);
            }
        }
        row0 += __shfl_sync(0xffffffffu, rows_to, 31);
        entry0 += __shfl_sync(0xffffffffu, entries_to, 31);
    }
    if (lane == 0) *a.b.n_entries = min(entry0, kMoeMaxEntries);
}

// Sums of N values over the lanes of a warp, N a multiple of 32: every exchange hands half of a lane's partial sums to its
// partner, so lane l ends up with values l * N / 32 .. of v[0 ..]; the additions are those of a plain butterfly.
template <int N>
__device__ __forceinline__ void warp_reduce_scatter(float* v, int lane) {
#pragma unroll
    for (int o = 16, half = N / 2; o > 0; o >>= 1, half >>= 1) {
        const bool upper = (lane & o) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
            const float give = upper ? v[j] : v[j + half], keep = upper ? v[j + half] : v[j];
            v[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
}

// A warp computes 8 rows x 8 outputs, lanes along the columns; WE of a CTA's warps are neighbours in the outputs, the rest in
// the rows.  Rows pass through two shared-memory stages, the next weights are in flight while the current ones are used.
// grid: (row blocks, blocks of 8 * WE outputs)
template <int WE>
struct RouteCfg {
    static constexpr int WR = RT_WARPS / WE;
    static constexpr int ROWS = 8 * WR;
    static constexpr int KC = WR >= 4 ? 128 : 512 / WR;   // columns per stage
    static constexpr int STAGE = ROWS * KC;               // floats
};
template <int WE>
__global__ void __launch_bounds__(RT_WARPS * 32, 2)
moe_route_kernel(const RouteArgs a) {
    using C = RouteCfg<WE>;
    grid_dep_trigger();
    extern __shared__ __align__(16) float sm[];
    __shared__ int s_last;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r0 = blockIdx.x * C::ROWS, nr = min(C::ROWS, a.rows - r0);
    const int e0 = (blockIdx.y * WE + warp % WE) * 8, wr = (warp / WE) * 8;
    const int steps = (a.ld + 127) / 128, stages = (a.ld + C::KC - 1) / C::KC;
    uint2 next[8];
    auto load_w = [&](int step) {
        const int c = step * 128 + lane * 4;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            next[i] = (e0 + i < a.outputs && c < a.ld) ? __ldg(reinterpret_cast<const uint2*>(a.w + static_cast<size_t>(e0 + i) * a.ld + c))
                                                       : make_uint2(0u, 0u);
        }
    };
    auto load_x = [&](int stage) {
        float* dst = sm + (stage & 1) * C::STAGE;
#pragma unroll
        for (int j = 0; j < C::STAGE / 4; j += RT_WARPS * 32) {
            const int i = (j + threadIdx.x) * 4, r = i / C::KC, c = stage * C::KC + i % C::KC;
            const bool in = r < nr && c < a.ld;   // elsewhere zeros are filled in
            ptx::cp_async16(dst + i, in ? a.x + static_cast<size_t>(r0 + r) * a.ld + c : a.x, in ? 16 : 0);
        }
        ptx::cp_async_commit();
    };
    load_w(0);   // the weights never depend on the previous kernel
    grid_dep_wait();
    float acc[64];
#pragma unroll
    for (int i = 0; i < 64; ++i) acc[i] = 0.f;
    load_x(0);
    for (int st = 0; st < stages; ++st) {
        if (st + 1 < stages) {
            load_x(st + 1);
            ptx::cp_async_wait<1>();
        } else {
            ptx::cp_async_wait<0>();
        }
        __syncthreads();
        const float* xs = sm + (st & 1) * C::STAGE + wr * C::KC + lane * 4;
#pragma unroll 1
        for (int k = 0; k < C::KC / 128; ++k) {
            const int step = st * (C::KC / 128) + k;
            if (step >= steps) break;
            float w[8][4];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const bf16* b = reinterpret_cast<const bf16*>(&next[i]);
#pragma unroll
                for (int e = 0; e < 4; ++e) w[i][e] = __bfloat162float(b[e]);
            }
            if (step + 1 < steps) load_w(step + 1);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                const float4 x = *reinterpret_cast<const float4*>(xs + r * C::KC + k * 128);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    float& s = acc[i * 8 + r];
                    s = fmaf(x.x, w[i][0], s);
                    s = fmaf(x.y, w[i][1], s);
                    s = fmaf(x.z, w[i][2], s);
                    s = fmaf(x.w, w[i][3], s);
                }
            }
        }
        __syncthreads();   // the stage is filled again two iterations on
    }
    warp_reduce_scatter<64>(acc, lane);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int k = lane * 2 + j, e = e0 + k / 8, r = wr + k % 8;
        if (r < nr && e < a.outputs) a.b.z[static_cast<size_t>(r0 + r) * a.outputs + e] = acc[j];
    }
    // the CTA counted last of this block of rows chooses its experts
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        int last = 1;
        if (gridDim.y > 1) {
            last = atomicAdd(&a.b.tickets[1 + blockIdx.x], 1) == static_cast<int>(gridDim.y) - 1;
            if (last) a.b.tickets[1 + blockIdx.x] = 0;
        }
        s_last = last;
    }
    __syncthreads();
    if (s_last == 0) return;
    __threadfence();
    const int per_warp = 2 * a.outputs + 2 * a.groups;
    for (int r = warp; r < nr; r += RT_WARPS) choose_experts<false>(a, r0 + r, sm + warp * per_warp, lane);
    // the CTA counted last of the launch lays out the rows
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        const int last = atomicAdd(&a.b.tickets[0], 1) == static_cast<int>(gridDim.x) - 1;
        if (last) a.b.tickets[0] = 0;
        s_last = last;
    }
    __syncthreads();
    if (s_last == 0) return;
    __threadfence();
    if (warp == 0) lay_out_rows(a, lane);
}

// A launch with a single row (decoding): one output per warp, whose weights are on their way before the row exists.  The
// additions are those of moe_route_kernel, in the same order.
constexpr int RT_PRE = 32;   // 128-column pieces of the weights held in registers
__global__ void __launch_bounds__(RT_WARPS * 32)
moe_route_one_kernel(const RouteArgs a) {
    grid_dep_trigger();
    extern __shared__ float sm[];
    __shared__ int s_last;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int e = blockIdx.x * RT_WARPS + warp;
    const bf16* w = a.w + static_cast<size_t>(e < a.outputs ? e : 0) * a.ld;
    uint2 wv[RT_PRE];
#pragma unroll
    for (int j = 0; j < RT_PRE; ++j) {
        const int c = j * 128 + lane * 4;
        wv[j] = c < a.ld ? __ldg(reinterpret_cast<const uint2*>(w + c)) : make_uint2(0u, 0u);
    }
    grid_dep_wait();
    float acc = 0.f;
    auto add = [&](const uint2& wp, const float4& x) {
        const bf16* b = reinterpret_cast<const bf16*>(&wp);
        acc = fmaf(x.x, __bfloat162float(b[0]), acc);
        acc = fmaf(x.y, __bfloat162float(b[1]), acc);
        acc = fmaf(x.z, __bfloat162float(b[2]), acc);
        acc = fmaf(x.w, __bfloat162float(b[3]), acc);
    };
#pragma unroll
    for (int j0 = 0; j0 < RT_PRE; j0 += 8) {
        float4 x[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = (j0 + j) * 128 + lane * 4;
            x[j] = c < a.ld ? *reinterpret_cast<const float4*>(a.x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) add(wv[j0 + j], x[j]);
    }
    for (int c = RT_PRE * 128 + lane * 4; c < a.ld; c += 128) {
        add(*reinterpret_cast<const uint2*>(w + c), *reinterpret_cast<const float4*>(a.x + c));
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane == 0 && e < a.outputs) a.b.z[e] = acc;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        const int last = atomicAdd(&a.b.tickets[0], 1) == static_cast<int>(gridDim.x) - 1;
        if (last) a.b.tickets[0] = 0;
        s_last = last;
    }
    __syncthreads();
    if (s_last == 0 || warp != 0) return;
    __threadfence();
    choose_experts<true>(a, 0, sm, lane);
}

// One CTA per token row: its input goes to every chosen expert's slot.
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ src, T* __restrict__ dst, const MoeBuffers b, int top, int experts, int ld) {
    grid_dependency_sync();
    __shared__ int slot[kMoeMaxTop];
    if (threadIdx.x < top) {
        const size_t i = static_cast<size_t>(blockIdx.x) * top + threadIdx.x;
        const int e = b.expert[i];
        slot[threadIdx.x] = e < experts ? b.offset[e] + b.rank[i] : -1;
    }
    __syncthreads();
    const int n16 = ld * static_cast<int>(sizeof(T)) / 16;
    const uint4* s = reinterpret_cast<const uint4*>(src + static_cast<size_t>(blockIdx.x) * ld);
    for (int c = threadIdx.x; c < n16; c += blockDim.x) {
        const uint4 v = s[c];
        for (int k = 0; k < top; ++k) {
            if (slot[k] >= 0) reinterpret_cast<uint4*>(dst + static_cast<size_t>(slot[k]) * ld)[c] = v;
        }
    }
}

// ---------------------------------------------------------------- grouped products
constexpr int BLOCK_K = 64;
constexpr int UMMA_K = 16;
constexpr int W_TILE_BYTES = gemm::BLOCK_N * BLOCK_K * 2;
constexpr int NUM_THREADS = 192;   // warp 0 TMA, warp 1 MMA + TMEM, warps 2-5 epilogue

template <int MT>
struct Cfg {
    static constexpr int STAGE_BYTES = W_TILE_BYTES + MT * BLOCK_K * 2;
    static constexpr int STAGES = (MT <= 16) ? 10 : (MT <= 32) ? 9 : (MT <= 64) ? 8 : (MT <= 128) ? 6 : 4;
    static constexpr int TMEM_COLS = (2 * MT < 32) ? 32 : 2 * MT;
    static constexpr int CTRL_BYTES = 256;
    static constexpr int ENTRY_BYTES = 16 * kMoeMaxEntries;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + CTRL_BYTES + gemm::SWIGLU_XCH_BYTES + ENTRY_BYTES + 1024;
    static_assert(SMEM_BYTES <= 232448, "shared memory budget");
};

struct GemmArgs {
    int n_tiles, kblocks, N;
    int n_tiles_s, kblocks_s, N_s;
    int groups_s;          // row groups of the shared expert (all tokens)
    int rows;              // tokens
    int tile;
    long long w_row_s;
    int xs_row0, ys_row0;
    bf16* y;
    int ldy;
    const int4* entries;
    const int32_t* n_entries;
    int uniform;           // > 0: the groups are not the router's, every one of this many matrices has all rows
    int* error;
};
// The row groups come from the router.  gate/up launches its successor only after its own wait, i.e. when the router has
// finished; down may therefore read the groups, and ask for their weights, before it waits for gate/up.

// Output tile t: the shared expert's tiles come first, then the experts' row groups; the feature tile runs fastest, so
// CTAs of a wave share a group's rows and its expert's matrix passes through L2 once for all of the expert's groups.
struct TileJob {
    bool shared;
    int n_tile, kblocks, N;
    int w_row;             // first row of the weight tile in the weight map (without the k-block)
    int x_row, y_row, rows;
};

template <bool SWIGLU>
__device__ __forceinline__ TileJob tile_job(const GemmArgs& a, const int4* entries, int t) {
    TileJob j;
    const int ts = a.groups_s * a.n_tiles_s;
    if (t < ts) {
        const int g = t / a.n_tiles_s;
        j.shared = true;
        j.n_tile = t - g * a.n_tiles_s;
        j.kblocks = a.kblocks_s;
        j.N = a.N_s;
        j.w_row = static_cast<int>(a.w_row_s) + j.n_tile * a.kblocks_s * gemm::BLOCK_N;
        j.x_row = a.xs_row0 + g * a.tile;
        j.y_row = a.ys_row0 + g * a.tile;
        j.rows = min(a.tile, a.rows - g * a.tile);
    } else {
        const int g = (t - ts) / a.n_tiles;
        const int4 e = entries[g];
        j.shared = false;
        j.n_tile = (t - ts) - g * a.n_tiles;
        j.kblocks = a.kblocks;
        j.N = a.N;
        j.w_row = (e.x * a.n_tiles + j.n_tile) * a.kblocks * gemm::BLOCK_N;
        j.x_row = SWIGLU ? e.y : e.z;   // the down product reads the rows gate/up wrote
        j.y_row = e.z;
        j.rows = e.w;
    }
    return j;
}

template <int MT, bool SWIGLU>
__global__ void __launch_bounds__(NUM_THREADS, 1)
moe_gemm_umma_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x,
                     const __grid_constant__ CUtensorMap tm_xs, const GemmArgs a) {
    using C = Cfg<MT>;
    constexpr int XBOX = MT < 64 ? MT : 64;   // rows per copy of the row operand (x_box of the maps)
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
    uint8_t* tiles = smem;
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::STAGES * C::STAGE_BYTES);
    uint64_t* empty = full + C::STAGES;
    uint64_t* acc_full = empty + C::STAGES;
    uint64_t* acc_empty = acc_full + 2;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* xch = reinterpret_cast<float*>(smem + C::STAGES * C::STAGE_BYTES + C::CTRL_BYTES);
    int4* entries = reinterpret_cast<int4*>(smem + C::STAGES * C::STAGE_BYTES + C::CTRL_BYTES + gemm::SWIGLU_XCH_BYTES);

    const int warp = threadIdx.x >> 5;
    const int lane = threadIdx.x & 31;
    constexpr bool kGroupsEarly = !SWIGLU;
    if (kGroupsEarly) grid_dep_trigger();
    if (threadIdx.x == 0) {
        for (int s = 0; s < C::STAGES; ++s) {
            ptx::mbar_init(&full[s], 1);
            ptx::mbar_init(&empty[s], 1);
        }
        for (int s = 0; s < 2; ++s) {
            ptx::mbar_init(&acc_full[s], 1);
            ptx::mbar_init(&acc_empty[s], 128);
        }
        *abort_flag = 0;
        ptx::mbar_fence_init();
        ptx::prefetch_tensormap(&tm_w);
        ptx::prefetch_tensormap(&tm_x);
        ptx::prefetch_tensormap(&tm_xs);
    }
    if (warp == 1) {
        ptx::tmem_alloc(tmem_slot, C::TMEM_COLS);
        ptx::tmem_relinquish();
    }
    auto read_groups = [&]() -> int {
        if (a.uniform > 0) {
            const int per = (a.rows + a.tile - 1) / a.tile, n = a.uniform * per;
            for (int i = threadIdx.x; i < n; i += NUM_THREADS) {
                const int m = i / per, r = (i - m * per) * a.tile;
                entries[i] = make_int4(m, m * a.rows + r, m * a.rows + r, min(a.tile, a.rows - r));
            }
            return n;
        }
        const int n = min(__ldcg(a.n_entries), kMoeMaxEntries);
        for (int i = threadIdx.x; i < n; i += NUM_THREADS) entries[i] = __ldcg(a.entries + i);
        return n;
    };
    int n_entries = kGroupsEarly ? read_groups() : 0;
    ptx::tc_fence_before();
    __syncthreads();
    ptx::tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    // weights of the first k-blocks, as far as the tiles are known, before the wait for the predecessor
    const int shared_tiles = a.groups_s * a.n_tiles_s;
    int pre = 0;
    if (threadIdx.x == 0) {
        const int known = shared_tiles + n_entries * a.n_tiles;
        for (int t = blockIdx.x; t < known && pre < C::STAGES; t += gridDim.x) {
            const TileJob j = tile_job<SWIGLU>(a, entries, t);
            const uint32_t bytes = W_TILE_BYTES + (j.rows + XBOX - 1) / XBOX * (XBOX * BLOCK_K * 2);
            for (int kb = 0; kb < j.kblocks && pre < C::STAGES; ++kb, ++pre) {
                ptx::mbar_arrive_expect_tx(&full[pre], bytes);
                ptx::tma_load_2d(tiles + pre * C::STAGE_BYTES, &tm_w, &full[pre], 0, j.w_row + kb * gemm::BLOCK_N);
            }
        }
    }
    grid_dep_wait();
    if (!kGroupsEarly) {
        grid_dep_trigger();
        n_entries = read_groups();
        __syncthreads();
    }
    const int total = shared_tiles + n_entries * a.n_tiles;

    if (warp == 0) {
        // ------------------------------------------------ TMA producer
        if (lane == 0) {
            int stage = 0;
            uint32_t phase = 0;
            int issued = 0;
            bool ok = true;
            for (int t = blockIdx.x; ok && t < total; t += gridDim.x) {
                const TileJob j = tile_job<SWIGLU>(a, entries, t);
                const int boxes = (j.rows + XBOX - 1) / XBOX;   // rows nobody asked for are not fetched
                const uint32_t bytes = W_TILE_BYTES + boxes * (XBOX * BLOCK_K * 2);
                for (int kb = 0; kb < j.kblocks; ++kb, ++issued) {
                    uint8_t* dst = tiles + stage * C::STAGE_BYTES;
                    if (issued >= pre) {
                        if (!ptx::mbar_wait(&empty[stage], phase ^ 1, abort_flag)) { ok = false; break; }
                        ptx::mbar_arrive_expect_tx(&full[stage], bytes);
                        ptx::tma_load_2d(dst, &tm_w, &full[stage], 0, j.w_row + kb * gemm::BLOCK_N);
                    }
                    for (int b = 0; b < boxes; ++b) {
                        ptx::tma_load_2d(dst + W_TILE_BYTES + b * (XBOX * BLOCK_K * 2), j.shared ? &tm_xs : &tm_x, &full[stage], kb * BLOCK_K,
                                         j.x_row + b * XBOX);
                    }
                    if (++stage == C::STAGES) { stage = 0; phase ^= 1; }
                }
            }
            if (!ok) {
                // give copies already in flight time to land before the CTA retires
                const long long t0 = clock64();
                while (clock64() - t0 < 2000000LL) {}
            }
        }
    } else if (warp == 1) {
        // ------------------------------------------------ MMA issuer
        if (lane == 0) {
            int stage = 0;
            uint32_t phase = 0;
            int acc = 0;
            uint32_t acc_phase = 0;
            bool ok = true;
            for (int t = blockIdx.x; ok && t < total; t += gridDim.x) {
                const TileJob j = tile_job<SWIGLU>(a, entries, t);
                // a group that is not full costs only its rows (rounded up to 16)
                const int n_mma = min(MT, (j.rows + 15) & ~15);
                const uint32_t idesc = ptx::umma_idesc_bf16(gemm::BLOCK_N, n_mma, 0, 0);
                if (!ptx::mbar_wait(&acc_empty[acc], acc_phase ^ 1, abort_flag)) break;
                ptx::tc_fence_after();
                const uint32_t d_tmem = tmem_base + acc * MT;
                for (int kb = 0; kb < j.kblocks; ++kb) {
                    if (!ptx::mbar_wait(&full[stage], phase, abort_flag)) { ok = false; break; }
                    ptx::tc_fence_after();
                    const uint32_t wa = ptx::smem_u32(tiles + stage * C::STAGE_BYTES);
                    const uint32_t xa = wa + W_TILE_BYTES;
#pragma unroll
                    for (int k = 0; k < BLOCK_K / UMMA_K; ++k) {
                        const uint64_t da = ptx::umma_desc_sw128(wa + k * UMMA_K * 2, 16, 1024);
                        const uint64_t db = ptx::umma_desc_sw128(xa + k * UMMA_K * 2, 16, 1024);
                        ptx::umma_ss(d_tmem, da, db, idesc, (kb > 0 || k > 0) ? 1u : 0u);
                    }
                    ptx::umma_commit(&empty[stage]);
                    if (++stage == C::STAGES) { stage = 0; phase ^= 1; }
                }
                if (!ok) break;
                ptx::umma_commit(&acc_full[acc]);
                acc ^= 1;
                if (acc == 0) acc_phase ^= 1;
            }
        }
    } else {
        // ------------------------------------------------ epilogue (128 threads; lane = feature, column = row of the group)
        const int q = warp & 3;
        const int row = q * 32 + lane;
        int acc = 0, xi = 0;
        uint32_t acc_phase = 0;
        for (int t = blockIdx.x; t < total; t += gridDim.x) {
            const TileJob j = tile_job<SWIGLU>(a, entries, t);
            const int n = SWIGLU ? j.n_tile * 64 + (row & 63) : j.n_tile * gemm::BLOCK_N + row;
            if (!ptx::mbar_wait_warp(&acc_full[acc], acc_phase, abort_flag)) break;
            ptx::tc_fence_after();
            const uint32_t t_addr = tmem_base + (static_cast<uint32_t>(q * 32) << 16) + acc * MT;
#pragma unroll 1
            for (int c0 = 0; c0 < MT; c0 += 16) {
                if (c0 >= j.rows) break;   // uniform across the CTA
                uint32_t r[16];
                ptx::tmem_ld16(t_addr + c0, r);
                ptx::tmem_wait_ld();
                bf16* y = a.y + static_cast<size_t>(j.y_row + c0) * a.ldy + n;
                if constexpr (SWIGLU) {
                    // lanes 0-63 hold the gate projection, lanes 64-127 the up projection of the same 64 features; the gate
                    // values pass through one of two shared-memory buffers to the warps of the up half, which store
                    float* xb = xch + (xi & 1) * (2 * 16 * 32);
                    ++xi;
                    if (q < 2) {
#pragma unroll
                        for (int c = 0; c < 16; ++c) xb[(q * 16 + c) * 32 + lane] = __bfloat162float(__float2bfloat16(__uint_as_float(r[c])));
                    }
                    // a buffer is written again two batches later, past the next batch's barrier
                    ptx::named_bar_sync(1, 128);
                    if (q >= 2 && n < j.N) {
#pragma unroll
                        for (int c = 0; c < 16; ++c) {
                            if (c0 + c < j.rows) {
                                const float uv = __bfloat162float(__float2bfloat16(__uint_as_float(r[c])));
                                y[static_cast<size_t>(c) * a.ldy] = __float2bfloat16(silu_mul(xb[((q - 2) * 16 + c) * 32 + lane], uv));
                            }
                        }
                    }
                } else if (n < j.N) {
#pragma unroll
                    for (int c = 0; c < 16; ++c) {
                        if (c0 + c < j.rows) y[static_cast<size_t>(c) * a.ldy] = __float2bfloat16(__uint_as_float(r[c]));
                    }
                }
            }
            ptx::tc_fence_before();
            ptx::mbar_arrive(&acc_empty[acc]);
            if (++acc == 2) { acc = 0; acc_phase ^= 1; }
        }
    }

    ptx::tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        ptx::tc_fence_after();
        ptx::tmem_dealloc(tmem_base, C::TMEM_COLS);
    }
    if (threadIdx.x == 0 && *abort_flag) atomicOr(a.error, ERR_GEMM_TIMEOUT);
}

template <int MT, bool SWIGLU>
void launch_gemm(const MoeGemmPlan& p, const GemmArgs& a, int grid, cudaStream_t s) {
    static bool configured = false;
    if (!configured) {
        CUDA_CHECK(cudaFuncSetAttribute(moe_gemm_umma_kernel<MT, SWIGLU>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg<MT>::SMEM_BYTES));
        configured = true;
    }
    launch_kernel(moe_gemm_umma_kernel<MT, SWIGLU>, dim3(grid), dim3(NUM_THREADS), Cfg<MT>::SMEM_BYTES, s, p.tm_w, p.tm_x, p.tm_xs, a);
}

CUtensorMap weight_map(const bf16* w, size_t elems) { return make_tmap_2d(w, BLOCK_K, elems / BLOCK_K, BLOCK_K * 2, BLOCK_K, gemm::BLOCK_N); }

}  // namespace

size_t moe_ticket_ints(int max_rows) { return 1 + static_cast<size_t>(max_rows); }

int moe_pick_tile(const LayerSpec& sp, int rows) {
    // tokens of one expert: the average with some room for uneven choices, never more than all
    const long long avg = (static_cast<long long>(rows) * sp.top * 5 / 4 + sp.experts + sp.identity - 1) / (sp.experts + sp.identity);
    int tile = 16;
    while (tile < 256 && tile < std::min<long long>(avg, rows)) tile *= 2;
    while (tile < 256 && moe_max_entries(sp, rows, tile) > kMoeMaxEntries) tile *= 2;
    return tile;
}

int moe_max_entries(const LayerSpec& sp, int rows, int tile) {
    const long long slots = static_cast<long long>(rows) * std::min(sp.top, sp.experts);
    return static_cast<int>(std::min<long long>(slots, slots / tile + sp.experts));
}

void launch_moe_route(const LayerSpec& sp, const float* x32, const bf16* w, const float* correction, const MoeBuffers& b, int rows,
                      int ld, int tile, bool direct, cudaStream_t s) {
    ProfileScope prof(KC_ROUTE, s);
    RouteArgs a;
    a.x = x32; a.w = w; a.correction = correction;
    a.rows = rows; a.ld = ld;
    a.outputs = sp.experts + sp.identity; a.experts = sp.experts; a.top = sp.top;
    a.groups = sp.groups; a.keep = sp.keep_groups;
    a.scale = sp.router_scale;
    a.tile = tile; a.direct = direct ? 1 : 0;
    a.b = b;
    CPM_REQUIRE(moe_max_entries(sp, rows, tile) <= kMoeMaxEntries, "mixture of experts: too many row groups");
    const size_t choose = static_cast<size_t>(RT_WARPS) * (2 * a.outputs + 2 * a.groups) * sizeof(float);
    if (rows == 1) {
        const size_t smem = (2 * a.outputs + 2 * a.groups) * sizeof(float);   // at most 16 KB
        launch_kernel(moe_route_one_kernel, dim3(ceil_div(a.outputs, RT_WARPS)), dim3(RT_WARPS * 32), smem, s, a);
        return;
    }
    auto run = [&](auto we) {
        constexpr int WE = decltype(we)::value;
        using C = RouteCfg<WE>;
        static bool configured = false;
        if (!configured) {
            CUDA_CHECK(cudaFuncSetAttribute(moe_route_kernel<WE>, cudaFuncAttributeMaxDynamicSharedMemorySize, RT_WARPS * 4 * kMoeMaxOutputs * 4));
            configured = true;
        }
        launch_kernel(moe_route_kernel<WE>, dim3(ceil_div(rows, C::ROWS), ceil_div(a.outputs, 8 * WE)), dim3(RT_WARPS * 32),
                      std::max<size_t>(choose, 2 * C::STAGE * sizeof(float)), s, a);
    };
    // few rows: all warps side by side in the outputs, so that the rows spread over more CTAs
    if (a.outputs > 32 || rows <= 64) run(std::integral_constant<int, 8>());
    else if (a.outputs > 16) run(std::integral_constant<int, 4>());
    else if (a.outputs > 8) run(std::integral_constant<int, 2>());
    else run(std::integral_constant<int, 1>());
}

template <typename T>
void launch_moe_gather(const LayerSpec& sp, const T* src, T* dst, const MoeBuffers& b, int rows, int ld, cudaStream_t s) {
    ProfileScope prof(KC_ROUTE, s);
    launch_kernel(moe_gather_kernel<T>, dim3(rows), dim3(256), 0, s, src, dst, b, sp.top, sp.experts, ld);
}
template void launch_moe_gather<bf16>(const LayerSpec&, const bf16*, bf16*, const MoeBuffers&, int, int, cudaStream_t);
template void launch_moe_gather<float>(const LayerSpec&, const float*, float*, const MoeBuffers&, int, int, cudaStream_t);

size_t moe_gate_up_offset(const LayerSpec& sp, int K, int expert) { return static_cast<size_t>(expert) * 2 * pad64(sp.expert_ff) * K; }
size_t moe_gate_up_elems(const LayerSpec& sp, int K) { return moe_gate_up_offset(sp, K, sp.experts) + static_cast<size_t>(2) * pad64(sp.shared_ff) * K; }
size_t moe_down_offset(const LayerSpec& sp, int width, int expert) { return static_cast<size_t>(expert) * linear_weight_elems(width, pad64(sp.expert_ff)); }
size_t moe_down_elems(const LayerSpec& sp, int width) { return moe_down_offset(sp, width, sp.experts) + linear_weight_elems(width, pad64(sp.shared_ff)); }

MoeGemmPlan make_grouped_plan(const bf16* w, int n, int N, int N_s, int K, const bf16* x, bf16* y, int ldy, int rows) {
    CPM_REQUIRE(K % BLOCK_K == 0 && n >= 1 && N >= 1 && rows >= 1, "grouped product: bad sizes");
    MoeGemmPlan p;
    p.tile = 16;
    while (p.tile < 256 && p.tile < rows) p.tile *= 2;
    const size_t one = linear_weight_elems(N, K);
    p.tm_w = weight_map(w, n * one + (N_s > 0 ? linear_weight_elems(N_s, K) : 0));
    p.tm_x = make_tmap_2d(x, K, static_cast<uint64_t>(n + (N_s > 0 ? 1 : 0)) * rows, static_cast<uint64_t>(K) * 2, BLOCK_K, std::min(p.tile, 64));
    p.tm_xs = p.tm_x;
    p.rows = rows;
    p.uniform = n;
    p.max_entries = n * ceil_div(rows, p.tile);
    CPM_REQUIRE(p.max_entries <= kMoeMaxEntries, "grouped product: too many row groups");
    p.n_tiles = ceil_div(N, gemm::BLOCK_N); p.kblocks = K / BLOCK_K; p.N = N;
    p.n_tiles_s = N_s > 0 ? ceil_div(N_s, gemm::BLOCK_N) : 0; p.kblocks_s = p.kblocks; p.N_s = N_s;
    p.w_row_s = static_cast<long long>(n * one / BLOCK_K);
    p.xs_row0 = p.ys_row0 = n * rows;
    p.y = y; p.ldy = ldy;
    return p;
}

MoeGemmPlan make_moe_gate_up_plan(const LayerSpec& sp, const bf16* w, const bf16* x, int x_rows, const bf16* xs, int K, bf16* act,
                                  int ld_act, int rows, int tile, const MoeBuffers& b) {
    CPM_REQUIRE(K % BLOCK_K == 0 && ld_act % BLOCK_K == 0, "mixture of experts: padded widths must be multiples of 64");
    MoeGemmPlan p;
    const int ff = pad64(sp.expert_ff), ffs = pad64(sp.shared_ff);
    p.tm_w = weight_map(w, moe_gate_up_elems(sp, K));
    p.tm_x = make_tmap_2d(x, K, x_rows, static_cast<uint64_t>(K) * 2, BLOCK_K, std::min(tile, 64));
    p.tm_xs = make_tmap_2d(xs, K, rows, static_cast<uint64_t>(K) * 2, BLOCK_K, std::min(tile, 64));
    p.tile = tile; p.rows = rows; p.max_entries = moe_max_entries(sp, rows, tile);
    p.swiglu = 1;
    p.n_tiles = ff / 64; p.kblocks = K / BLOCK_K; p.N = ff;
    p.n_tiles_s = ffs / 64; p.kblocks_s = p.kblocks; p.N_s = ffs;
    p.w_row_s = static_cast<long long>(moe_gate_up_offset(sp, K, sp.experts) / BLOCK_K);
    p.xs_row0 = 0; p.ys_row0 = rows * sp.top;
    p.y = act; p.ldy = ld_act;
    p.entries = b.entries; p.n_entries = b.n_entries;
    return p;
}

MoeGemmPlan make_moe_down_plan(const LayerSpec& sp, const bf16* w, const bf16* act, int act_rows, int ld_act, int width, bf16* y,
                               int ld_y, int rows, int tile, const MoeBuffers& b) {
    CPM_REQUIRE(ld_act % BLOCK_K == 0, "mixture of experts: padded widths must be multiples of 64");
    MoeGemmPlan p;
    const int ff = pad64(sp.expert_ff), ffs = pad64(sp.shared_ff);
    p.tm_w = weight_map(w, moe_down_elems(sp, width));
    p.tm_x = make_tmap_2d(act, ld_act, act_rows, static_cast<uint64_t>(ld_act) * 2, BLOCK_K, std::min(tile, 64));
    p.tm_xs = p.tm_x;
    p.tile = tile; p.rows = rows; p.max_entries = moe_max_entries(sp, rows, tile);
    p.n_tiles = ceil_div(width, gemm::BLOCK_N); p.kblocks = ff / BLOCK_K; p.N = width;
    p.n_tiles_s = ffs > 0 ? p.n_tiles : 0; p.kblocks_s = ffs / BLOCK_K; p.N_s = width;
    p.w_row_s = static_cast<long long>(moe_down_offset(sp, width, sp.experts) / BLOCK_K);
    p.xs_row0 = p.ys_row0 = rows * sp.top;
    p.y = y; p.ldy = ld_y;
    p.entries = b.entries; p.n_entries = b.n_entries;
    return p;
}

void launch_moe_gemm(const MoeGemmPlan& p, cudaStream_t s) {
    ProfileScope prof(p.uniform > 0 ? KC_LINEAR : KC_MOE, s);
    GemmArgs a;
    a.n_tiles = p.n_tiles; a.kblocks = p.kblocks; a.N = p.N;
    a.n_tiles_s = p.n_tiles_s; a.kblocks_s = p.kblocks_s; a.N_s = p.N_s;
    a.groups_s = p.n_tiles_s > 0 ? ceil_div(p.rows, p.tile) : 0;
    if (a.n_tiles_s == 0) a.n_tiles_s = 1;   // a divisor only
    a.rows = p.rows; a.tile = p.tile;
    a.w_row_s = p.w_row_s; a.xs_row0 = p.xs_row0; a.ys_row0 = p.ys_row0;
    a.y = p.y; a.ldy = p.ldy;
    a.entries = p.entries; a.n_entries = p.n_entries;
    a.uniform = p.uniform;
    a.error = runtime().d_error;
    const long long most = static_cast<long long>(a.groups_s) * a.n_tiles_s + static_cast<long long>(p.max_entries) * p.n_tiles;
    const int grid = static_cast<int>(std::max<long long>(1, std::min<long long>(most, runtime().num_sms)));
    switch (p.tile * 2 + p.swiglu) {
        case 16 * 2: launch_gemm<16, false>(p, a, grid, s); break;
        case 16 * 2 + 1: launch_gemm<16, true>(p, a, grid, s); break;
        case 32 * 2: launch_gemm<32, false>(p, a, grid, s); break;
        case 32 * 2 + 1: launch_gemm<32, true>(p, a, grid, s); break;
        case 64 * 2: launch_gemm<64, false>(p, a, grid, s); break;
        case 64 * 2 + 1: launch_gemm<64, true>(p, a, grid, s); break;
        case 128 * 2: launch_gemm<128, false>(p, a, grid, s); break;
        case 128 * 2 + 1: launch_gemm<128, true>(p, a, grid, s); break;
        case 256 * 2: launch_gemm<256, false>(p, a, grid, s); break;
        case 256 * 2 + 1: launch_gemm<256, true>(p, a, grid, s); break;
        default: throw std::invalid_argument("cpmcu_b200: bad row group size");
    }
}
