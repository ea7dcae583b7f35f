// Linear attention with a constant decay per head ("lightning attention"), from per-request state, and the norm and
// gate behind it.  With q = silu(q'), k = silu(k'), v = silu(v') read out of a float32 projection, per head
//
//     S_t = a S_(t-1) + k_t v_t^T   (d x dv, float32) ;   o_t = S_t^T q_t
//
// Two forms of the same sums:
//
//   sharpi_lightning_walk     short portions and decoded tokens: a block holds [d, 32 VEC columns] of a head's state in
//                             registers (warp w owns d / 8 of its rows, a lane VEC neighbouring columns, so a state row
//                             is read and written in whole lines), walks the portion's rows, and adds the eight
//                             warps' parts of an output in a fixed order.
//   sharpi_lightning_chunks   longer portions, in chunks of LIN_CHUNK rows so that every chunk of every head works at
//                             once: (1) a chunk's own contribution to the state, sum_i a^(last - i) k_i v_i^T, for all
//                             chunks; (2) a walk over the chunks that leaves the state before every chunk and the
//                             portion's last state; (3) per chunk o_i = sum_(j <= i) a^(i - j) (q_i . k_j) v_j
//                             + a^(i + 1) S^T q_i.  All products are float32 FMAs on tiles of 64 x 64.
//   sharpi_norm_sigmoid_gate  out = y / sqrt(mean(y^2) + eps) * w * sigmoid(g) * scale over a whole row (all heads side
//                             by side), written into a column range of a wider matrix.
//
// The powers of a come from a table made on the host (a^0 .. a^LIN_CHUNK, formed in float64).  Which of the two forms
// serves a request depends on the number of its rows in the step alone, and inside a form a row's sums do not depend
// on what else is in the step.  The state is read at the start of a portion and stored behind its last row.
#include "common.cuh"

constexpr int LIN_THREADS = 256;
constexpr int LIN_WARPS = LIN_THREADS / 32;
constexpr int LIN_STAGE = 8;             // rows of a walk staged together
constexpr int LIN_CHUNK = 64;            // rows of a chunk
constexpr int LIN_LD = 68;               // floats between two rows of a tile in shared memory
constexpr int LIN_MAX_KEY = 512;

// silu with the exact exponential and division, or (FAST, where the activations only have to hold up to bfloat16) with the
// hardware's: a relative error of about 2^-21
template <bool FAST> __device__ __forceinline__ float silu_f32(float z) {
    return FAST ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));
}

struct LinArgs {
    const float* proj;          // [T, ld]: q at col_q (heads * d), k at col_k (heads * d), v at col_v (heads * dv)
    int ld, col_q, col_k, col_v;
    const float* pow;           // [heads][LIN_CHUNK + 1]: powers of the head's decay
    const int* row_offsets;     // [B + 1]
    const int* state_slots;     // [B]
    float* state;               // [slots][heads][d][dv]
    long long state_stride;
    float* y;                   // [T, heads * dv]
    int heads, d, dv;
    int fast;                   // activations with the hardware's exponential
    const int* requests;        // walk: the requests to serve (null: all)
    const int* chunks;          // chunks: [n, 4] first row, rows, request, -
    const int* spans;           // chunks: [m, 4] request, first chunk, number of chunks, -
    float* sums;                // chunks: [n][heads][d][dv] scratch
};

// -------------------------------------------------------------------------------------------------------------
// the walk
// -------------------------------------------------------------------------------------------------------------
template <int VEC> struct Pack { float v[VEC]; };

template <int VEC> __device__ __forceinline__ Pack<VEC> load_pack(const float* p) {
    Pack<VEC> r;
    if (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[1 % VEC] = x.y; r.v[2 % VEC] = x.z; r.v[3 % VEC] = x.w;
    } else if (VEC == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        r.v[0] = x.x; r.v[1 % VEC] = x.y;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VEC> __device__ __forceinline__ void store_pack(float* p, const Pack<VEC>& r) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % VEC], r.v[2 % VEC], r.v[3 % VEC]);
    else if (VEC == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[1 % VEC]);
    else *p = r.v[0];
}

template <bool FAST, int ROWS, int VEC>  // state rows a warp (8 ROWS >= d), columns a lane
__global__ void __launch_bounds__(LIN_THREADS) lightning_walk_kernel(LinArgs a) {
    constexpr int COLS = 32 * VEC;
    __shared__ __align__(16) float q_s[LIN_STAGE][LIN_WARPS * ROWS];
    __shared__ __align__(16) float k_s[LIN_STAGE][LIN_WARPS * ROWS];
    __shared__ __align__(16) float v_s[LIN_STAGE][COLS];
    __shared__ __align__(16) float part_s[LIN_STAGE][LIN_WARPS][COLS];
    pdl_wait();
    const int req = a.requests ? a.requests[blockIdx.z] : blockIdx.z;
    const int h = blockIdx.y;
    const int first = a.row_offsets[req], rows = a.row_offsets[req + 1] - first;
    if (rows <= 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int d = a.d, dv = a.dv;
    const int c0 = blockIdx.x * COLS;
    const int c = c0 + lane * VEC;
    const bool live = c < dv;                                  // dv is a multiple of VEC
    float* st = a.state + (size_t)a.state_slots[req] * a.state_stride + (size_t)h * d * dv;
    const float decay = a.pow[h * (LIN_CHUNK + 1) + 1];
    Pack<VEC> S[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = warp * ROWS + j;
        if (live && n < d) {
            S[j] = load_pack<VEC>(st + (size_t)n * dv + c);
        } else {
#pragma unroll
            for (int u = 0; u < VEC; ++u) S[j].v[u] = 0.0f;
        }
    }
    for (int r0 = 0; r0 < rows; r0 += LIN_STAGE) {
        const int nr = min(LIN_STAGE, rows - r0);
        if (r0) __syncthreads();                               // the rows before are no longer read
        const float* src = a.proj + (size_t)(first + r0) * a.ld;
        for (int i = threadIdx.x; i < nr * LIN_WARPS * ROWS; i += LIN_THREADS) {
            const int r = i / (LIN_WARPS * ROWS), n = i % (LIN_WARPS * ROWS);
            const float* row = src + (size_t)r * a.ld + (size_t)h * d + n;
            q_s[r][n] = n < d ? silu_f32<FAST>(row[a.col_q]) : 0.0f;
            k_s[r][n] = n < d ? silu_f32<FAST>(row[a.col_k]) : 0.0f;
        }
        for (int i = threadIdx.x; i < nr * COLS; i += LIN_THREADS) {
            const int r = i / COLS, cc = c0 + i % COLS;
            v_s[r][i % COLS] = cc < dv ? silu_f32<FAST>(src[(size_t)r * a.ld + a.col_v + (size_t)h * dv + cc]) : 0.0f;
        }
        __syncthreads();
        for (int r = 0; r < nr; ++r) {
            const Pack<VEC> v = load_pack<VEC>(&v_s[r][lane * VEC]);
            Pack<VEC> acc;
#pragma unroll
            for (int u = 0; u < VEC; ++u) acc.v[u] = 0.0f;
#pragma unroll
            for (int j = 0; j < ROWS; ++j) {
                const float k = k_s[r][warp * ROWS + j], q = q_s[r][warp * ROWS + j];
#pragma unroll
                for (int u = 0; u < VEC; ++u) {
                    S[j].v[u] = fmaf(decay, S[j].v[u], k * v.v[u]);
                    acc.v[u] = fmaf(q, S[j].v[u], acc.v[u]);
                }
            }
            store_pack<VEC>(&part_s[r][warp][lane * VEC], acc);
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nr * COLS; i += LIN_THREADS) {
            const int r = i / COLS, cc = i % COLS;
            if (c0 + cc >= dv) continue;
            float sum = 0.0f;
#pragma unroll
            for (int w = 0; w < LIN_WARPS; ++w) sum += part_s[r][w][cc];
            a.y[(size_t)(first + r0 + r) * a.heads * dv + (size_t)h * dv + c0 + cc] = sum;
        }
    }
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
        const int n = warp * ROWS + j;
        if (live && n < d) store_pack<VEC>(st + (size_t)n * dv + c, S[j]);
    }
}

template <int ROWS, int VEC>
static int launch_walk(const LinArgs& a, int n, cudaStream_t stream) {
    const dim3 grid((a.dv + 32 * VEC - 1) / (32 * VEC), a.heads, n);
    if (a.fast) SHARPI_LAUNCH_PDL((lightning_walk_kernel<true, ROWS, VEC>), grid, LIN_THREADS, 0, stream, a);
    else SHARPI_LAUNCH_PDL((lightning_walk_kernel<false, ROWS, VEC>), grid, LIN_THREADS, 0, stream, a);
    return SHARPI_OK;
}

static bool fill_args(LinArgs& a, const float* proj, int ld, int col_q, int col_k, int col_v, const float* pow,
                      const int* row_offsets, const int* state_slots, float* state, long long state_stride, float* y,
                      int heads, int d, int dv) {
    if (heads <= 0 || heads > 65535 || d <= 0 || d > LIN_MAX_KEY || dv <= 0 || col_q < 0 || col_k < 0 || col_v < 0 ||
        col_q + heads * d > ld || col_k + heads * d > ld || col_v + heads * dv > ld)
        return false;
    a.proj = proj; a.ld = ld; a.col_q = col_q; a.col_k = col_k; a.col_v = col_v; a.pow = pow;
    a.row_offsets = row_offsets; a.state_slots = state_slots; a.state = state; a.state_stride = state_stride; a.y = y;
    a.heads = heads; a.d = d; a.dv = dv; a.requests = nullptr; a.chunks = nullptr; a.spans = nullptr; a.sums = nullptr;
    return true;
}

// `requests` (nullable): the `n` requests of the step to serve; null: requests 0 .. n - 1.
SHARPI_API int sharpi_lightning_walk(const float* proj, int ld, int col_q, int col_k, int col_v, const float* pow,
                                     const int* row_offsets, const int* state_slots, const int* requests, int n,
                                     float* state, long long state_stride, float* y, int heads, int d, int dv,
                                     int fast, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    LinArgs a;
    if (n > 65535 || !fill_args(a, proj, ld, col_q, col_k, col_v, pow, row_offsets, state_slots, state, state_stride, y,
                                heads, d, dv))
        return SHARPI_BAD_ARGUMENT;
    a.requests = requests; a.fast = fast;
    const bool al4 = dv % 4 == 0 && state_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
    const bool al2 = dv % 2 == 0 && state_stride % 2 == 0 && (reinterpret_cast<uintptr_t>(state) & 7) == 0;
    const int vec = (al4 && dv > 64) ? 4 : (al2 && dv > 32) ? 2 : 1;
    if (d <= 32) return vec == 4 ? launch_walk<4, 4>(a, n, stream) : vec == 2 ? launch_walk<4, 2>(a, n, stream) : launch_walk<4, 1>(a, n, stream);
    if (d <= 64) return vec == 4 ? launch_walk<8, 4>(a, n, stream) : vec == 2 ? launch_walk<8, 2>(a, n, stream) : launch_walk<8, 1>(a, n, stream);
    if (d <= 128) return vec == 4 ? launch_walk<16, 4>(a, n, stream) : vec == 2 ? launch_walk<16, 2>(a, n, stream) : launch_walk<16, 1>(a, n, stream);
    if (d <= 256) return vec >= 2 && al2 ? launch_walk<32, 2>(a, n, stream) : launch_walk<32, 1>(a, n, stream);
    return launch_walk<64, 1>(a, n, stream);
}

// -------------------------------------------------------------------------------------------------------------
// chunks
// -------------------------------------------------------------------------------------------------------------
// A 64 x 64 tile of columns c .. c + 63 (those below `cols`; zeros behind) of rows row0 .. row0 + rows - 1 (zeros behind):
// as it is (ACT 0), through silu (1: exact, 2: fast), and times pw[rows - 1 - row] where `pw` is given.
template <int ACT>
__device__ __forceinline__ float tile_value(float x, float f) {
    return ACT == 0 ? x : f * silu_f32<ACT == 2>(x);
}

template <int ACT>
__device__ __forceinline__ void load_tile(float* dst, const float* src, size_t ld, int c, int cols, int rows, bool vec,
                                          const float* pw = nullptr) {
    if (vec) {
        float4 x[4];                                           // all four pieces of a thread are asked for at once
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const int i = threadIdx.x + p * LIN_THREADS, r = i >> 4, e = (i & 15) * 4;
            x[p] = r < rows && c + e < cols ? *reinterpret_cast<const float4*>(src + (size_t)r * ld + c + e)
                                            : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
#pragma unroll
        for (int p = 0; p < 4; ++p) {
            const int i = threadIdx.x + p * LIN_THREADS, r = i >> 4, e = (i & 15) * 4;
            const float f = pw && r < rows ? pw[rows - 1 - r] : 1.0f;
            *reinterpret_cast<float4*>(dst + r * LIN_LD + e) = make_float4(
                tile_value<ACT>(x[p].x, f), tile_value<ACT>(x[p].y, f), tile_value<ACT>(x[p].z, f), tile_value<ACT>(x[p].w, f));
        }
    } else {
        for (int i = threadIdx.x; i < LIN_CHUNK * 64; i += LIN_THREADS) {
            const int r = i >> 6, e = i & 63;
            float x = 0.0f;
            if (r < rows && c + e < cols) x = tile_value<ACT>(src[(size_t)r * ld + c + e], pw ? pw[rows - 1 - r] : 1.0f);
            dst[r * LIN_LD + e] = x;
        }
    }
}

// acc[a][b] += sum_k A[ty + 16 a][k] B[k][4 tx + b] over the 64 columns of a tile
__device__ __forceinline__ void tile_mul(const float* A, const float* B, int ty, int tx, float acc[4][4]) {
#pragma unroll 4
    for (int k = 0; k < 64; k += 4) {
        float4 x[4], y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) x[i] = *reinterpret_cast<const float4*>(A + (ty + 16 * i) * LIN_LD + k);
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = *reinterpret_cast<const float4*>(B + (k + i) * LIN_LD + 4 * tx);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float xs[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                acc[i][0] = fmaf(xs[kk], y[kk].x, acc[i][0]);
                acc[i][1] = fmaf(xs[kk], y[kk].y, acc[i][1]);
                acc[i][2] = fmaf(xs[kk], y[kk].z, acc[i][2]);
                acc[i][3] = fmaf(xs[kk], y[kk].w, acc[i][3]);
            }
        }
    }
}

// acc[a][b] += sum_k A[ty + 16 a][k] B[tx + 16 b][k]
__device__ __forceinline__ void tile_mul_t(const float* A, const float* B, int ty, int tx, float acc[4][4]) {
#pragma unroll 4
    for (int k = 0; k < 64; k += 4) {
        float4 x[4], y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) x[i] = *reinterpret_cast<const float4*>(A + (ty + 16 * i) * LIN_LD + k);
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = *reinterpret_cast<const float4*>(B + (tx + 16 * i) * LIN_LD + k);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                acc[i][j] = fmaf(x[i].x, y[j].x, acc[i][j]);
                acc[i][j] = fmaf(x[i].y, y[j].y, acc[i][j]);
                acc[i][j] = fmaf(x[i].z, y[j].z, acc[i][j]);
                acc[i][j] = fmaf(x[i].w, y[j].w, acc[i][j]);
            }
    }
}

// (1) sums[chunk][h][n][v] = sum_i a^(rows - 1 - i) k_i[n] v_i[v]; a block makes 64 x 64 of them
template <bool FAST>
__global__ void __launch_bounds__(LIN_THREADS) lightning_sums_kernel(LinArgs a, int tiles_v, int vec) {
    __shared__ __align__(16) float k_s[LIN_CHUNK * LIN_LD];
    __shared__ __align__(16) float v_s[LIN_CHUNK * LIN_LD];
    pdl_wait();
    const int chunk = blockIdx.z, h = blockIdx.y;
    const int n0 = (blockIdx.x / tiles_v) * 64, c0 = (blockIdx.x % tiles_v) * 64;
    const int row0 = a.chunks[4 * chunk], rows = a.chunks[4 * chunk + 1];
    const float* src = a.proj + (size_t)row0 * a.ld;
    load_tile<FAST ? 2 : 1>(k_s, src + a.col_k + (size_t)h * a.d, a.ld, n0, a.d, rows, vec, a.pow + h * (LIN_CHUNK + 1));
    load_tile<FAST ? 2 : 1>(v_s, src + a.col_v + (size_t)h * a.dv, a.ld, c0, a.dv, rows, vec);
    __syncthreads();
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4] = {};
#pragma unroll 4
    for (int i = 0; i < LIN_CHUNK; ++i) {                      // rows behind the chunk's last are zeros
        const float4 k = *reinterpret_cast<const float4*>(k_s + i * LIN_LD + 4 * ty);
        const float4 v = *reinterpret_cast<const float4*>(v_s + i * LIN_LD + 4 * tx);
        const float ks[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            acc[e][0] = fmaf(ks[e], v.x, acc[e][0]);
            acc[e][1] = fmaf(ks[e], v.y, acc[e][1]);
            acc[e][2] = fmaf(ks[e], v.z, acc[e][2]);
            acc[e][3] = fmaf(ks[e], v.w, acc[e][3]);
        }
    }
    float* out = a.sums + ((size_t)chunk * a.heads + h) * a.d * a.dv;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const int n = n0 + 4 * ty + e;
        if (n >= a.d) break;
        float* o = out + (size_t)n * a.dv + c0 + 4 * tx;
        if (vec) {
            if (c0 + 4 * tx < a.dv) *reinterpret_cast<float4*>(o) = make_float4(acc[e][0], acc[e][1], acc[e][2], acc[e][3]);
        } else {
            for (int u = 0; u < 4; ++u)
                if (c0 + 4 * tx + u < a.dv) o[u] = acc[e][u];
        }
    }
}

// (2) over the chunks of a portion: sums[chunk] <- the state before the chunk; state <- a^rows state + the chunk's sum
template <int VEC>
__global__ void __launch_bounds__(LIN_THREADS) lightning_carry_kernel(LinArgs a) {
    pdl_wait();
    const int* span = a.spans + 4 * blockIdx.z;
    const int req = span[0], chunk0 = span[1], n = span[2];
    const int h = blockIdx.y;
    const int size = a.d * a.dv;
    const int i = (blockIdx.x * LIN_THREADS + threadIdx.x) * VEC;
    if (i >= size) return;
    float* st = a.state + (size_t)a.state_slots[req] * a.state_stride + (size_t)h * size + i;
    const float* pw = a.pow + h * (LIN_CHUNK + 1);
    const size_t step = (size_t)a.heads * size;
    float* u = a.sums + (size_t)chunk0 * step + (size_t)h * size + i;
    Pack<VEC> S = load_pack<VEC>(st);
    constexpr int AHEAD = 8;                                   // chunk sums asked for ahead of the walk
    Pack<VEC> next[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
        if (k < n) next[k] = load_pack<VEC>(u + k * step);
    for (int c = 0; c < n; c += AHEAD) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            if (c + k >= n) break;
            const Pack<VEC> own = next[k];
            if (c + k + AHEAD < n) next[k] = load_pack<VEC>(u + (size_t)(c + k + AHEAD) * step);
            store_pack<VEC>(u + (size_t)(c + k) * step, S);
            const float p = pw[a.chunks[4 * (chunk0 + c + k) + 1]];
#pragma unroll
            for (int e = 0; e < VEC; ++e) S.v[e] = fmaf(p, S.v[e], own.v[e]);
        }
    }
    store_pack<VEC>(st, S);
}

// (3) the outputs of one chunk's rows, 64 value columns of one head
template <bool FAST>
__global__ void __launch_bounds__(LIN_THREADS, 3) lightning_out_kernel(LinArgs a, int vec) {
    extern __shared__ __align__(16) float lin_smem[];
    float* q_s = lin_smem;
    float* k_s = q_s + LIN_CHUNK * LIN_LD;
    float* s_s = k_s + LIN_CHUNK * LIN_LD;
    float* pw = s_s + LIN_CHUNK * LIN_LD;
    pdl_wait();
    const int chunk = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * 64;
    const int row0 = a.chunks[4 * chunk], rows = a.chunks[4 * chunk + 1];
    const float* src = a.proj + (size_t)row0 * a.ld;
    const float* before = a.sums + ((size_t)chunk * a.heads + h) * a.d * a.dv;
    if (threadIdx.x <= LIN_CHUNK) pw[threadIdx.x] = a.pow[h * (LIN_CHUNK + 1) + threadIdx.x];
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    constexpr int ACT = FAST ? 2 : 1;
    float score[4][4] = {}, past[4][4] = {};
    for (int n0 = 0; n0 < a.d; n0 += 64) {
        if (n0) __syncthreads();
        load_tile<ACT>(q_s, src + a.col_q + (size_t)h * a.d, a.ld, n0, a.d, rows, vec);
        load_tile<ACT>(k_s, src + a.col_k + (size_t)h * a.d, a.ld, n0, a.d, rows, vec);
        load_tile<0>(s_s, before + (size_t)n0 * a.dv, a.dv, c0, a.dv, min(64, a.d - n0), vec);
        __syncthreads();
        tile_mul_t(q_s, k_s, ty, tx, score);
        tile_mul(q_s, s_s, ty, tx, past);
    }
    __syncthreads();
    load_tile<ACT>(k_s, src + a.col_v + (size_t)h * a.dv, a.ld, c0, a.dv, rows, vec);         // the values
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int r = ty + 16 * i, s = tx + 16 * j;
            q_s[r * LIN_LD + s] = s <= r ? score[i][j] * pw[r - s] : 0.0f;                    // the decayed scores
        }
    __syncthreads();
    float own[4][4] = {};
    tile_mul(q_s, k_s, ty, tx, own);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = ty + 16 * i;
        if (r >= rows) continue;
        const float p = pw[r + 1];
        float* o = a.y + (size_t)(row0 + r) * a.heads * a.dv + (size_t)h * a.dv + c0 + 4 * tx;
        if (vec) {
            if (c0 + 4 * tx < a.dv)
                *reinterpret_cast<float4*>(o) = make_float4(fmaf(p, past[i][0], own[i][0]), fmaf(p, past[i][1], own[i][1]),
                                                            fmaf(p, past[i][2], own[i][2]), fmaf(p, past[i][3], own[i][3]));
        } else {
            for (int u = 0; u < 4; ++u)
                if (c0 + 4 * tx + u < a.dv) o[u] = fmaf(p, past[i][u], own[i][u]);
        }
    }
}

// `chunks` int32 [n_chunks, 4] (first row, rows <= LIN_CHUNK, request, unused), the chunks of a request one after the
// other; `spans` int32 [n_spans, 4] (request, first chunk, number of chunks, unused); `sums` float32
// [n_chunks * heads * d * dv] of scratch.
SHARPI_API int sharpi_lightning_chunks(const float* proj, int ld, int col_q, int col_k, int col_v, const float* pow,
                                       const int* row_offsets, const int* state_slots, const int* chunks, int n_chunks,
                                       const int* spans, int n_spans, float* sums, float* state, long long state_stride,
                                       float* y, int heads, int d, int dv, int fast, cudaStream_t stream) {
    if (n_chunks <= 0) return SHARPI_OK;
    LinArgs a;
    if (n_chunks > 65535 || n_spans <= 0 || n_spans > 65535 ||
        !fill_args(a, proj, ld, col_q, col_k, col_v, pow, row_offsets, state_slots, state, state_stride, y, heads, d, dv))
        return SHARPI_BAD_ARGUMENT;
    a.chunks = chunks; a.spans = spans; a.sums = sums; a.fast = fast;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(sums) |
                           reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(y);
    const int vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && col_q % 4 == 0 && col_k % 4 == 0 && col_v % 4 == 0 &&
                    state_stride % 4 == 0 && (ptrs & 15) == 0;
    const int tiles_n = (d + 63) / 64, tiles_v = (dv + 63) / 64;
    const dim3 sum_grid(tiles_n * tiles_v, heads, n_chunks);
    if (fast) SHARPI_LAUNCH_PDL(lightning_sums_kernel<true>, sum_grid, LIN_THREADS, 0, stream, a, tiles_v, vec);
    else SHARPI_LAUNCH_PDL(lightning_sums_kernel<false>, sum_grid, LIN_THREADS, 0, stream, a, tiles_v, vec);
    const int size = d * dv;
    if (vec)
        SHARPI_LAUNCH_PDL(lightning_carry_kernel<2>, dim3((size / 2 + LIN_THREADS - 1) / LIN_THREADS, heads, n_spans),
                          LIN_THREADS, 0, stream, a);
    else
        SHARPI_LAUNCH_PDL(lightning_carry_kernel<1>, dim3((size + LIN_THREADS - 1) / LIN_THREADS, heads, n_spans),
                          LIN_THREADS, 0, stream, a);
    constexpr size_t smem = (3 * LIN_CHUNK * LIN_LD + LIN_CHUNK + 4) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(lightning_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||
            cudaFuncSetAttribute(lightning_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return SHARPI_LAUNCH_FAILED;
        configured = true;
    }
    if (fast) SHARPI_LAUNCH_PDL(lightning_out_kernel<true>, dim3(tiles_v, heads, n_chunks), LIN_THREADS, smem, stream, a, vec);
    else SHARPI_LAUNCH_PDL(lightning_out_kernel<false>, dim3(tiles_v, heads, n_chunks), LIN_THREADS, smem, stream, a, vec);
    return SHARPI_OK;
}

// -------------------------------------------------------------------------------------------------------------
// norm over a whole row, weight, sigmoid gate, factor
// -------------------------------------------------------------------------------------------------------------
constexpr int GATE_PER = 8;              // elements a thread keeps; wider rows are read twice

template <typename TO, int THREADS>
__global__ void __launch_bounds__(THREADS)
norm_sigmoid_gate_kernel(const float* y, const float* g, int ld_g, const float* __restrict__ w, float eps, float scale,
                         int width, TO* out, int ld_out) {
    __shared__ float scratch[32];
    pdl_wait();
    const size_t t = blockIdx.x;
    const float* yr = y + t * width;
    const float* gr = g + t * ld_g;
    float v[GATE_PER], gg[GATE_PER];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < GATE_PER; ++k) {
        const int i = threadIdx.x + k * THREADS;
        v[k] = i < width ? yr[i] : 0.0f;
        gg[k] = i < width ? gr[i] : 0.0f;
    }
#pragma unroll
    for (int k = 0; k < GATE_PER; ++k) ss += v[k] * v[k];
    for (int i = threadIdx.x + GATE_PER * THREADS; i < width; i += THREADS) ss += yr[i] * yr[i];
    ss = block_sum(ss, scratch);
    const float f = scale / sqrtf(ss / (float)width + eps);
    TO* o = out + t * ld_out;
#pragma unroll
    for (int k = 0; k < GATE_PER; ++k) {
        const int i = threadIdx.x + k * THREADS;
        if (i < width) o[i] = from_float<TO>(v[k] * f * w[i] / (1.0f + expf(-gg[k])));
    }
    for (int i = threadIdx.x + GATE_PER * THREADS; i < width; i += THREADS)
        o[i] = from_float<TO>(yr[i] * f * w[i] / (1.0f + expf(-gr[i])));
}

// `out`: a column range of a matrix whose rows are `ld_out` elements apart
SHARPI_API int sharpi_norm_sigmoid_gate(const float* y, const float* g, int ld_g, const float* w, float eps, float scale,
                                        int T, int width, void* out, int ld_out, int out_dtype, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (width <= 0 || ld_g < width || ld_out < width) return SHARPI_BAD_ARGUMENT;
#define GATE_CASE(TO, N) \
    SHARPI_LAUNCH_PDL((norm_sigmoid_gate_kernel<TO, N>), T, N, 0, stream, y, g, ld_g, w, eps, scale, width, (TO*)out, ld_out)
    if (out_dtype == SHARPI_F32) {
        if (width <= 256 * GATE_PER) GATE_CASE(float, 256); else GATE_CASE(float, 1024);
    } else if (out_dtype == SHARPI_BF16) {
        if (width <= 256 * GATE_PER) GATE_CASE(bf16, 256); else GATE_CASE(bf16, 1024);
    } else {
        return SHARPI_BAD_ARGUMENT;
    }
#undef GATE_CASE
    return SHARPI_OK;
}
