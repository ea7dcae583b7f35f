// The gated delta rule with a decay per key channel, from per-request state.  Per head (key size d, value size dv), for the
// rows of a request in order:
//
//     S <- g_t * S  (row c of S by g_t[c]);  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t
//
// with q and k unit vectors (q also times d^(-1/2)), beta = sigmoid(.), g = exp(-exp(A) softplus(z + bias)).
//
//   sharpi_delta_prep    behind the fused projection [q | k | v | low | b]: the short causal convolution and silu of every
//                        channel of q, k, v (inputs before a portion come from the request's state, which moves on), the
//                        unit norms, beta, and the low-rank columns rounded for the product that reads them.
//   sharpi_delta_walk    decoded tokens and short portions, row by row: eight lanes hold one column of S in registers
//                        (columns are stored one after the other, so a column's elements are contiguous), a row costs one
//                        exchange among the eight for S^T k and S^T q together: with the decayed S,
//                        o = S^T q + (k . q) u.
//   sharpi_delta_chunks  longer portions in chunks of DC_ROWS rows.  With S_0 the state before a chunk, D_t the product of
//                        the decays up to row t and P_ts that of the rows s + 1 .. t (products of numbers in (0, 1): no
//                        logarithm is summed and no exponent can overflow),
//                            u_t = beta_t (v_t - (D_t k_t)^T S_0 - sum_(s < t) A_ts u_s),   A_ts = sum_c k_t P_ts k_s
//                            o_t = (D_t q_t)^T S_0 + sum_(s <= t) B_ts u_s,                 B_ts = sum_c q_t P_ts k_s
//                            S   = D_last S_0 + sum_s (P_(s,last) k_s) u_s^T
//                        Solving the triangular system once for the columns of v and once for those of D k gives
//                        U = U_0 - W S_0, and with it o = B U_0 + (D q - B W) S_0.  (1) one kernel forms W, D q - B W,
//                        the decayed keys, U_0 and B U_0 for every chunk and head at once; (2) one walks a portion's
//                        chunks: one product with S_0 for all of a chunk's rows and one back into the state.
//   sharpi_head_norm_gate  out = y / sqrt(mean over the head (y^2) + eps) * w * sigmoid(gate)
//
// Everything is float32.  The chunks' walk is float32 FMAs, or (`split`, key sizes that are multiples of 64) tensor-core
// products of operands cut into three bfloat16 pieces each, 24 bits in all, of which the six products above 2^-24 are
// formed and added in float32; the state itself stays float32 in registers.  A request's form (walk or chunks) and its chunks depend on its own rows alone, and no sum
// depends on what else is in the step.  State per request and head: dv columns of dp = d rounded up to 4 floats.
#include "common.cuh"
#include "mma_sync.cuh"

constexpr int DELTA_MAX_KEY = 512;        // walk
constexpr int DELTA_MAX_CHUNK_KEY = 256;  // chunks

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float delta_decay(float z, float rate) {           // rate = exp(A)
    const float sp = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
    return expf(-rate * sp);
}

// -------------------------------------------------------------------------------------------------------------
// convolution, silu, unit norms, beta, low-rank columns
// -------------------------------------------------------------------------------------------------------------
struct PrepArgs {
    const float* proj;          // [T, ld]: q (kvh * d) | k (kvh * d) | v (heads * dv) | low (R) | b (heads)
    int ld;
    const float* conv;          // [taps][C]
    float* conv_state;          // [slots][taps - 1][C], oldest first
    long long conv_stride;
    const int* row_offsets;     // [B + 1]
    const int* state_slots;     // [B]
    const int* tiles;           // [n, 4] first row, rows, request, -; null: tile i is request i's rows
    float* qkv;                 // [T, C]
    float* beta;                // [T, heads]
    void* low;                  // [T, R]
    int kvh, heads, d, dv, taps, C, R;
    float q_scale;
};

constexpr int PREP_WARPS = 4;

// A warp serves one unit of a tile's rows: a head of q or of k (its norm is a sum over the unit), 32 NPL channels of v, or
// 32 NPL of the columns behind.  TAPS > 0: the window of inputs is kept in registers while the rows are walked.
template <typename TO, int NPL, int TAPS>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_prep_kernel(PrepArgs a) {
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int unit = blockIdx.y * PREP_WARPS + warp;
    int first, rows, req;
    if (a.tiles) {
        first = a.tiles[4 * blockIdx.x]; rows = a.tiles[4 * blockIdx.x + 1]; req = a.tiles[4 * blockIdx.x + 2];
    } else {
        req = blockIdx.x; first = a.row_offsets[req]; rows = a.row_offsets[req + 1] - first;
    }
    if (rows <= 0) return;
    constexpr int SPAN = 32 * NPL;
    const int v_width = a.heads * a.dv, v_units = (v_width + SPAN - 1) / SPAN;
    const int tail_width = a.R + a.heads, tail_units = (tail_width + SPAN - 1) / SPAN;
    if (unit >= 2 * a.kvh + v_units + tail_units) return;
    if (unit >= 2 * a.kvh + v_units) {                         // low-rank columns and beta
        const int c0 = (unit - 2 * a.kvh - v_units) * SPAN;
        for (int r = 0; r < rows; ++r) {
            const size_t t = first + r;
            const float* src = a.proj + t * a.ld + a.C;
#pragma unroll
            for (int j = 0; j < NPL; ++j) {
                const int c = c0 + lane + 32 * j;
                if (c < a.R) reinterpret_cast<TO*>(a.low)[t * a.R + c] = from_float<TO>(src[c]);
                else if (c < tail_width) a.beta[t * a.heads + c - a.R] = sigmoid_f(src[c]);
            }
        }
        return;
    }
    int c0, n;
    float scale = 0.0f;                                        // of the unit norm; 0: none
    if (unit < 2 * a.kvh) {
        c0 = unit * a.d; n = a.d; scale = unit < a.kvh ? a.q_scale : 1.0f;
    } else {
        const int v0 = (unit - 2 * a.kvh) * SPAN;
        c0 = 2 * a.kvh * a.d + v0; n = min(SPAN, v_width - v0);
    }
    const int portion = a.row_offsets[req], i0 = first - portion, K = a.taps - 1;
    float* st = a.conv_state + (size_t)a.state_slots[req] * a.conv_stride;
    const float* src = a.proj + c0;
    auto input = [&](int i, int e) -> float {                  // the unit's element e at place i of the portion (i >= -K)
        return i >= 0 ? src[(size_t)(portion + i) * a.ld + e] : st[(size_t)(K + i) * a.C + c0 + e];
    };
    constexpr int WIN = TAPS > 1 ? TAPS - 1 : 1;
    float win[WIN][NPL], w[TAPS > 0 ? TAPS : 1][NPL], next[NPL];
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < NPL; ++j) {
            const int e = lane + 32 * j;
#pragma unroll
            for (int k = 0; k < TAPS; ++k) w[k][j] = e < n ? a.conv[(size_t)k * a.C + c0 + e] : 0.0f;
            if (TAPS > 1) {
#pragma unroll
                for (int k = 0; k < WIN; ++k) win[k][j] = e < n ? input(i0 - WIN + k, e) : 0.0f;
            }
            next[j] = e < n ? input(i0, e) : 0.0f;
        }
    }
    for (int r = 0; r < rows; ++r) {
        float y[NPL];
        float ss = 0.0f;
#pragma unroll
        for (int j = 0; j < NPL; ++j) {
            const int e = lane + 32 * j;
            float acc = 0.0f;
            if (TAPS > 0) {
                const float cur = next[j];
                next[j] = e < n && r + 1 < rows ? input(i0 + r + 1, e) : 0.0f;
#pragma unroll
                for (int k = 0; k + 1 < TAPS; ++k) acc = fmaf(w[k][j], win[k % WIN][j], acc);
                acc = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][j], cur, acc);
#pragma unroll
                for (int k = 0; k + 1 < WIN; ++k) win[k][j] = win[(k + 1) % WIN][j];
                win[WIN - 1][j] = cur;
            } else if (e < n) {
                for (int k = 0; k < a.taps; ++k) acc = fmaf(a.conv[(size_t)k * a.C + c0 + e], input(i0 + r - K + k, e), acc);
            }
            y[j] = acc / (1.0f + expf(-acc));
            ss = fmaf(y[j], y[j], ss);
        }
        float f = 1.0f;
        if (scale != 0.0f) f = scale / sqrtf(warp_sum(ss) + 1e-6f);
        float* out = a.qkv + (size_t)(first + r) * a.C + c0;
#pragma unroll
        for (int j = 0; j < NPL; ++j)
            if (lane + 32 * j < n) out[lane + 32 * j] = y[j] * f;
    }
    // A portion's first tile has at least taps - 1 rows (or is the whole portion), so no other tile reads the state: it may
    // move on now.  Every lane rewrites the channels it read.
    if (i0 == 0 && K > 0) {
        const int total = a.row_offsets[req + 1] - portion;
        for (int j = 0; j < K; ++j)
            for (int e = lane; e < n; e += 32) {
                const int i = total - K + j;                   // ascending j: place j + total is read before it is written
                st[(size_t)j * a.C + c0 + e] = i >= 0 ? src[(size_t)(portion + i) * a.ld + e] : st[(size_t)(j + total) * a.C + c0 + e];
            }
    }
}

template <typename TO, int NPL>
static int launch_prep(const PrepArgs& a, dim3 grid, cudaStream_t stream) {
    switch (a.taps) {
        case 1: SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, NPL, 1>), grid, PREP_WARPS * 32, 0, stream, a); break;
        case 2: SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, NPL, 2>), grid, PREP_WARPS * 32, 0, stream, a); break;
        case 3: SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, NPL, 3>), grid, PREP_WARPS * 32, 0, stream, a); break;
        case 4: SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, NPL, 4>), grid, PREP_WARPS * 32, 0, stream, a); break;
        default: SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, NPL, 0>), grid, PREP_WARPS * 32, 0, stream, a); break;
    }
    return SHARPI_OK;
}

template <typename TO>
static int launch_prep_size(const PrepArgs& a, int n_tiles, cudaStream_t stream) {
    const int npl = a.d <= 32 ? 1 : a.d <= 64 ? 2 : a.d <= 128 ? 4 : a.d <= 256 ? 8 : 16;
    const int span = 32 * npl;
    const int units = 2 * a.kvh + (a.heads * a.dv + span - 1) / span + (a.R + a.heads + span - 1) / span;
    const dim3 grid(n_tiles, (units + PREP_WARPS - 1) / PREP_WARPS);
    if (npl == 1) return launch_prep<TO, 1>(a, grid, stream);
    if (npl == 2) return launch_prep<TO, 2>(a, grid, stream);
    if (npl == 4) return launch_prep<TO, 4>(a, grid, stream);
    SHARPI_LAUNCH_PDL((delta_prep_kernel<TO, 16, 0>), grid, PREP_WARPS * 32, 0, stream, a);
    return SHARPI_OK;
}

// `tiles` (nullable) int32 [n_tiles, 4]: the rows of the step in pieces (first row, rows, request, unused) that cross no
// request; a request's first piece holds at least taps - 1 rows or all it has.  Null: n_tiles requests, a piece each.
SHARPI_API int sharpi_delta_prep(const float* proj, int ld, const float* conv, float* conv_state, long long conv_stride,
                                 const int* row_offsets, const int* state_slots, const int* tiles, int n_tiles, float* qkv,
                                 float* beta, void* low, int low_dtype, int kvh, int heads, int d, int dv, int taps, int R,
                                 float q_scale, cudaStream_t stream) {
    if (n_tiles <= 0) return SHARPI_OK;
    PrepArgs a;
    if (kvh <= 0 || heads <= 0 || heads % kvh != 0 || d <= 0 || d > DELTA_MAX_KEY || dv <= 0 || taps <= 0 || R < 0 ||
        (taps > 1 && !conv_state))
        return SHARPI_BAD_ARGUMENT;
    a.proj = proj; a.ld = ld; a.conv = conv; a.conv_state = conv_state; a.conv_stride = conv_stride;
    a.row_offsets = row_offsets; a.state_slots = state_slots; a.tiles = tiles; a.qkv = qkv; a.beta = beta; a.low = low;
    a.kvh = kvh; a.heads = heads; a.d = d; a.dv = dv; a.taps = taps; a.R = R; a.q_scale = q_scale;
    a.C = 2 * kvh * d + heads * dv;
    if (a.C + R + heads > ld) return SHARPI_BAD_ARGUMENT;
    if (low_dtype == SHARPI_F32) return launch_prep_size<float>(a, n_tiles, stream);
    if (low_dtype == SHARPI_BF16) return launch_prep_size<bf16>(a, n_tiles, stream);
    return SHARPI_BAD_ARGUMENT;
}

// -------------------------------------------------------------------------------------------------------------
// the recurrence
// -------------------------------------------------------------------------------------------------------------
struct DeltaArgs {
    const float* qkv;           // [T, C]: q (kvh * d) | k (kvh * d) | v (heads * dv), as sharpi_delta_prep leaves them
    const float* beta;          // [T, heads]
    const float* z;             // [T, ldz]: the decay's projection, heads * d
    int ldz;
    const float* dt_bias;       // [heads * d]
    const float* a_log;         // [heads]
    const int* row_offsets;     // [B + 1]
    const int* state_slots;     // [B]
    const int* requests;        // walk: the requests to serve (null: all)
    const int* chunks;          // chunks: [n, 4] first row, rows, request, -
    const int* spans;           // chunks: [m, 4] request, first chunk, number of chunks, -
    float* state;               // [slots][heads][dv][dp]
    long long state_stride;
    float* y;                   // [T, heads * dv]
    float* mats;                // chunks: [n][heads][dp][48]: -W | D q - B W | decayed keys, a key channel's rows together;
                                // split: [n][heads][73 dp] words, the operands of the tensor-core walk (delta_carry_mma)
    float* last;                // chunks: [n][heads][dp]: the product of all decays of the chunk
    float* u0;                  // chunks: [n][heads][DC_ROWS][dv]
    int kvh, heads, d, dp, dv, C;
};

constexpr int WALK_THREADS = 256;
constexpr int WALK_LANES = 8;                                  // lanes of a column
constexpr int WALK_COLS = WALK_THREADS / WALK_LANES;
constexpr int WALK_STAGE = 8;                                  // rows staged together (one warp each forms k . q)

// A walk over many rows (LONG) starts on an empty GPU and lets nothing onto its SMs: its few blocks would otherwise land
// several to an SM.
template <int R4, bool LONG>                                   // float4 of a column a lane: 32 R4 >= d
__global__ void __launch_bounds__(WALK_THREADS) delta_walk_kernel(DeltaArgs a) {
    constexpr int DP = 32 * R4;
    extern __shared__ __align__(16) float walk_smem[];
    float* q_s = walk_smem;                                    // [STAGE][DP] each, zeros behind d
    float* k_s = q_s + WALK_STAGE * DP;
    float* g_s = k_s + WALK_STAGE * DP;
    float* v_s = g_s + WALK_STAGE * DP;                        // [STAGE][COLS]
    float* o_s = v_s + WALK_STAGE * WALK_COLS;
    float* b_s = o_s + WALK_STAGE * WALK_COLS;                 // [STAGE] beta, [STAGE] k . q
    const int h = blockIdx.y, hk = h / (a.heads / a.kvh);
    const float rate = expf(a.a_log[h]);
    if (LONG) pdl_wait_only();
    else pdl_wait();
    const int req = a.requests ? a.requests[blockIdx.z] : blockIdx.z;
    const int first = a.row_offsets[req], rows = a.row_offsets[req + 1] - first;
    if (rows <= 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int sub = threadIdx.x & (WALK_LANES - 1), col = threadIdx.x / WALK_LANES;
    const int c0 = blockIdx.x * WALK_COLS, c = c0 + col;
    float* st = a.state + (size_t)a.state_slots[req] * a.state_stride + ((size_t)h * a.dv + c) * a.dp;
    float4 S[R4];
#pragma unroll
    for (int j = 0; j < R4; ++j) {
        const int e = 4 * (sub + WALK_LANES * j);
        S[j] = c < a.dv && e < a.dp ? *reinterpret_cast<const float4*>(st + e) : make_float4(0, 0, 0, 0);
    }
    for (int r0 = 0; r0 < rows; r0 += WALK_STAGE) {
        const int nr = min(WALK_STAGE, rows - r0);
        if (r0) __syncthreads();                               // the rows before are no longer read
        for (int i = threadIdx.x; i < nr * DP; i += WALK_THREADS) {
            const int r = i / DP, e = i % DP;
            const size_t t = first + r0 + r;
            const float* row = a.qkv + t * a.C;
            float q = 0.0f, k = 0.0f, g = 0.0f;
            if (e < a.d) {
                q = row[hk * a.d + e];
                k = row[(a.kvh + hk) * a.d + e];
                g = delta_decay(a.z[t * a.ldz + h * a.d + e] + a.dt_bias[h * a.d + e], rate);
            }
            q_s[i] = q; k_s[i] = k; g_s[i] = g;
        }
        for (int i = threadIdx.x; i < nr * WALK_COLS; i += WALK_THREADS) {
            const int r = i / WALK_COLS, cc = c0 + i % WALK_COLS;
            v_s[i] = cc < a.dv ? a.qkv[(size_t)(first + r0 + r) * a.C + 2 * a.kvh * a.d + (size_t)h * a.dv + cc] : 0.0f;
        }
        if (threadIdx.x < nr) b_s[threadIdx.x] = a.beta[(size_t)(first + r0 + threadIdx.x) * a.heads + h];
        __syncthreads();
        if (warp < nr) {
            float kq = 0.0f;
            for (int e = lane; e < DP; e += 32) kq = fmaf(k_s[warp * DP + e], q_s[warp * DP + e], kq);
            kq = warp_sum(kq);
            if (lane == 0) b_s[WALK_STAGE + warp] = kq;
        }
        __syncthreads();
        for (int r = 0; r < nr; ++r) {
            const float4* k4 = reinterpret_cast<const float4*>(k_s + r * DP) + sub;
            const float4* q4 = reinterpret_cast<const float4*>(q_s + r * DP) + sub;
            const float4* g4 = reinterpret_cast<const float4*>(g_s + r * DP) + sub;
            float4 ak = make_float4(0, 0, 0, 0), aq = ak;
#pragma unroll
            for (int j = 0; j < R4; ++j) {
                const float4 k = k4[WALK_LANES * j], q = q4[WALK_LANES * j], g = g4[WALK_LANES * j];
                S[j].x *= g.x; S[j].y *= g.y; S[j].z *= g.z; S[j].w *= g.w;
                ak.x = fmaf(S[j].x, k.x, ak.x); ak.y = fmaf(S[j].y, k.y, ak.y);
                ak.z = fmaf(S[j].z, k.z, ak.z); ak.w = fmaf(S[j].w, k.w, ak.w);
                aq.x = fmaf(S[j].x, q.x, aq.x); aq.y = fmaf(S[j].y, q.y, aq.y);
                aq.z = fmaf(S[j].z, q.z, aq.z); aq.w = fmaf(S[j].w, q.w, aq.w);
            }
            float dk = (ak.x + ak.y) + (ak.z + ak.w), dq = (aq.x + aq.y) + (aq.z + aq.w);
#pragma unroll
            for (int o = WALK_LANES / 2; o > 0; o >>= 1) {
                dk += __shfl_xor_sync(0xffffffffu, dk, o);
                dq += __shfl_xor_sync(0xffffffffu, dq, o);
            }
            const float u = b_s[r] * (v_s[r * WALK_COLS + col] - dk);
            if (sub == 0) o_s[r * WALK_COLS + col] = fmaf(b_s[WALK_STAGE + r], u, dq);
#pragma unroll
            for (int j = 0; j < R4; ++j) {
                const float4 k = k4[WALK_LANES * j];
                S[j].x = fmaf(k.x, u, S[j].x); S[j].y = fmaf(k.y, u, S[j].y);
                S[j].z = fmaf(k.z, u, S[j].z); S[j].w = fmaf(k.w, u, S[j].w);
            }
        }
        __syncthreads();
        for (int i = threadIdx.x; i < nr * WALK_COLS; i += WALK_THREADS) {
            const int r = i / WALK_COLS, cc = c0 + i % WALK_COLS;
            if (cc < a.dv) a.y[((size_t)(first + r0 + r) * a.heads + h) * a.dv + cc] = o_s[i];
        }
    }
#pragma unroll
    for (int j = 0; j < R4; ++j) {
        const int e = 4 * (sub + WALK_LANES * j);
        if (c < a.dv && e < a.dp) *reinterpret_cast<float4*>(st + e) = S[j];
    }
}

static bool fill_delta(DeltaArgs& a, const float* qkv, const float* beta, const float* z, int ldz, const float* dt_bias,
                       const float* a_log, const int* row_offsets, const int* state_slots, float* state,
                       long long state_stride, float* y, int kvh, int heads, int d, int dv) {
    if (kvh <= 0 || heads <= 0 || heads > 65535 || heads % kvh != 0 || d <= 0 || d > DELTA_MAX_KEY || dv <= 0 ||
        ldz < heads * d || state_stride % 4 != 0 || (reinterpret_cast<uintptr_t>(state) & 15) != 0)
        return false;
    a.qkv = qkv; a.beta = beta; a.z = z; a.ldz = ldz; a.dt_bias = dt_bias; a.a_log = a_log; a.row_offsets = row_offsets;
    a.state_slots = state_slots; a.requests = nullptr; a.chunks = nullptr; a.spans = nullptr; a.state = state;
    a.state_stride = state_stride; a.y = y; a.mats = nullptr; a.last = nullptr; a.u0 = nullptr;
    a.kvh = kvh; a.heads = heads; a.d = d; a.dp = (d + 3) / 4 * 4; a.dv = dv; a.C = 2 * kvh * d + heads * dv;
    return true;
}

template <int R4>
static int launch_delta_walk(const DeltaArgs& a, int n, int max_rows, cudaStream_t stream) {
    const dim3 grid((a.dv + WALK_COLS - 1) / WALK_COLS, a.heads, n);
    const size_t smem = (size_t)(WALK_STAGE * (3 * 32 * R4 + 2 * WALK_COLS) + 2 * WALK_STAGE) * sizeof(float);
    static bool configured = false;
    if (smem > 48 * 1024 && !configured) {
        if (cudaFuncSetAttribute(delta_walk_kernel<R4, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||
            cudaFuncSetAttribute(delta_walk_kernel<R4, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return SHARPI_LAUNCH_FAILED;
        configured = true;
    }
    if (max_rows > WALK_STAGE) {
        delta_walk_kernel<R4, true><<<grid, WALK_THREADS, smem, stream>>>(a);
        SHARPI_CHECK_LAUNCH();
    } else {
        SHARPI_LAUNCH_PDL((delta_walk_kernel<R4, false>), grid, WALK_THREADS, smem, stream, a);
    }
    return SHARPI_OK;
}

// `requests` (nullable): the `n` requests of the step to serve; null: requests 0 .. n - 1.  `max_rows`: the most rows one of
// them brings (how the kernel is launched; no result depends on it).
SHARPI_API int sharpi_delta_walk(const float* qkv, const float* beta, const float* z, int ldz, const float* dt_bias,
                                 const float* a_log, const int* row_offsets, const int* state_slots, const int* requests,
                                 int n, int max_rows, float* state, long long state_stride, float* y, int kvh, int heads,
                                 int d, int dv, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    DeltaArgs a;
    if (n > 65535 || !fill_delta(a, qkv, beta, z, ldz, dt_bias, a_log, row_offsets, state_slots, state, state_stride, y, kvh,
                                 heads, d, dv))
        return SHARPI_BAD_ARGUMENT;
    a.requests = requests;
    if (d <= 32) return launch_delta_walk<1>(a, n, max_rows, stream);
    if (d <= 64) return launch_delta_walk<2>(a, n, max_rows, stream);
    if (d <= 128) return launch_delta_walk<4>(a, n, max_rows, stream);
    if (d <= 256) return launch_delta_walk<8>(a, n, max_rows, stream);
    return launch_delta_walk<16>(a, n, max_rows, stream);
}

// -------------------------------------------------------------------------------------------------------------
// chunks
// -------------------------------------------------------------------------------------------------------------
constexpr int DC_ROWS = 16;
constexpr int DC_THREADS = 256;
constexpr int DC_MATS = 3 * DC_ROWS;      // floats of a key channel in `mats`

// lane l of the warp ends with the sum over all lanes of their acc[l]
__device__ __forceinline__ float transpose_sum32(float (&acc)[32], int lane) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const bool up = lane & o;
            const float give = up ? acc[i] : acc[i + o], keep = up ? acc[i + o] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    return acc[0];
}

// Two neighbouring elements in three bfloat16 pieces each (24 bits together), packed as an operand register.
struct Pieces {
    uint32_t v[3];
};
__device__ __forceinline__ Pieces split3(float x, float y) {
    Pieces r;
#pragma unroll
    for (int p = 0; p < 3; ++p) {
        r.v[p] = mma16::pack_bf16(x, y);
        if (p < 2) {
            x -= __uint_as_float(r.v[p] << 16);
            y -= __uint_as_float(r.v[p] & 0xffff0000u);
        }
    }
    return r;
}

// The operands of the tensor-core walk in the order in which its lanes (g = lane / 4, t = lane % 4) take them, 16 bytes each.
// Of the 32 rows -W | D q - B W, per 16 key channels, piece and pair of row tiles: words (tile 0: channels 2t, 2t + 1 of
// row g | the same 8 further | tile 1 likewise); of the decayed keys, per 16 key channels and piece: (channel g: rows 2t,
// 2t + 1 | 8 further | channel g + 8 likewise); then the dp products of decays.
constexpr int CM_M_WORDS = 3 * 2 * 128, CM_K_WORDS = 3 * 128;  // of 16 key channels
__host__ __device__ constexpr int cm_words(int dp) { return dp / 16 * (CM_M_WORDS + CM_K_WORDS) + dp; }
__device__ __forceinline__ int cm_m_half(int p, int row, int key) {            // index of a bfloat16
    const int k = key & 15, n = row >> 3;
    const int word = ((key >> 4) * 6 + p * 2 + (n >> 1)) * 128 + ((row & 7) * 4 + ((k & 7) >> 1)) * 4 + (n & 1) * 2 + (k >> 3);
    return 2 * word + (k & 1);
}
__device__ __forceinline__ int cm_k_word(int dp, int p, int pair, int key) {   // rows 2 pair, 2 pair + 1
    return dp / 16 * CM_M_WORDS + ((key >> 4) * 3 + p) * 128 + ((key & 7) * 4 + (pair & 3)) * 4 + ((key >> 3) & 1) * 2 + (pair >> 2);
}

// (1) one chunk of one head
template <bool SPLIT>
__global__ void __launch_bounds__(DC_THREADS, SPLIT ? 3 : 2) delta_chunk_kernel(DeltaArgs a) {
    extern __shared__ __align__(16) float chunk_smem[];
    const int d = a.d, dp = a.dp;
    float* k_s = chunk_smem;                                   // [DC_ROWS][dp] each
    float* q_s = k_s + DC_ROWS * dp;
    float* g_s = q_s + DC_ROWS * dp;
    uint32_t* ops_s = reinterpret_cast<uint32_t*>(g_s + DC_ROWS * dp);         // SPLIT: cm_words(dp)
    __shared__ __align__(16) float A_s[DC_ROWS][DC_ROWS];      // [s][t]: beta_t A_ts where t > s
    __shared__ __align__(16) float B_s[DC_ROWS][DC_ROWS];      // [s][t]: B_ts where t >= s
    __shared__ float b_s[DC_ROWS];
    const int h = blockIdx.y, hk = h / (a.heads / a.kvh);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float rate = expf(a.a_log[h]);
    pdl_wait();
    const int chunk = blockIdx.x;
    const int row0 = a.chunks[4 * chunk], rows = a.chunks[4 * chunk + 1];
#pragma unroll
    for (int r = warp; r < DC_ROWS; r += DC_THREADS / 32) {
        const size_t t = row0 + min(r, rows - 1);
        const float* row = a.qkv + t * a.C + hk * d;
        const float* z = a.z + t * a.ldz + h * d;
        const bool live = r < rows;                            // rows behind the chunk's last leave everything as it is
#pragma unroll 4
        for (int e = lane; e < dp; e += 32) {
            const bool in = e < d;
            const float q = in ? row[e] : 0.0f, k = in ? row[a.kvh * d + e] : 0.0f;
            const float g = in ? z[e] + a.dt_bias[h * d + e] : 0.0f;
            q_s[r * dp + e] = live ? q : 0.0f;
            k_s[r * dp + e] = live ? k : 0.0f;
            g_s[r * dp + e] = live ? delta_decay(g, rate) : 1.0f;
        }
    }
    if (threadIdx.x < DC_ROWS)
        b_s[threadIdx.x] = threadIdx.x < rows ? a.beta[(size_t)(row0 + threadIdx.x) * a.heads + h] : 0.0f;
    __syncthreads();
    // A and B: warp w forms the columns s = w and 15 - w (17 rows in all); a lane walks its channels down the rows
#pragma unroll 1
    for (int s = warp; s < DC_ROWS; s += DC_ROWS - 1 - 2 * warp) {
        float acc[32];                                         // [t] A, [16 + t] B
#pragma unroll
        for (int i = 0; i < 32; ++i) acc[i] = 0.0f;
        for (int e = lane; e < dp; e += 32) {
            float p = k_s[s * dp + e];
#pragma unroll
            for (int t = 0; t < DC_ROWS; ++t) {
                if (t < s) continue;
                if (t > s) p *= g_s[t * dp + e];
                acc[t] = fmaf(k_s[t * dp + e], p, acc[t]);
                acc[16 + t] = fmaf(q_s[t * dp + e], p, acc[16 + t]);
            }
        }
        const float m = transpose_sum32(acc, lane);
        if (lane < 16) A_s[s][lane] = b_s[lane] * m;
        else B_s[s][lane - 16] = m;
        if (s == DC_ROWS - 1 - warp) break;
    }
    __syncthreads();
    // a thread a column of [D k | v]: w <- the triangular system's solution, row by row into all rows below it, and b += B w
    const size_t at = (size_t)chunk * a.heads + h;
    for (int j = threadIdx.x; j < dp + a.dv; j += DC_THREADS) {
        float w[DC_ROWS], b[DC_ROWS];
        const bool key = j < dp;
        if (key) {
            float D = 1.0f;
#pragma unroll
            for (int t = 0; t < DC_ROWS; ++t) {
                D *= g_s[t * dp + j];
                w[t] = -b_s[t] * (D * k_s[t * dp + j]);        // the key columns are kept negated: -W
                b[t] = D * q_s[t * dp + j];
            }
            if (SPLIT) ops_s[cm_words(dp) - dp + j] = __float_as_uint(D);
            else a.last[at * dp + j] = D;
        } else {
            const float* v = a.qkv + (size_t)row0 * a.C + 2 * a.kvh * d + (size_t)h * a.dv + j - dp;
#pragma unroll
            for (int t = 0; t < DC_ROWS; ++t) {
                w[t] = t < rows ? b_s[t] * v[(size_t)t * a.C] : 0.0f;
                b[t] = 0.0f;
            }
        }
#pragma unroll
        for (int r = 0; r < DC_ROWS; ++r) {
#pragma unroll
            for (int t4 = r / 4 * 4; t4 < DC_ROWS; t4 += 4) {
                const float4 m = *reinterpret_cast<const float4*>(&A_s[r][t4]);
                const float4 n = *reinterpret_cast<const float4*>(&B_s[r][t4]);
                if (t4 > r) w[t4] = fmaf(-m.x, w[r], w[t4]);
                if (t4 + 1 > r) w[t4 + 1] = fmaf(-m.y, w[r], w[t4 + 1]);
                if (t4 + 2 > r) w[t4 + 2] = fmaf(-m.z, w[r], w[t4 + 2]);
                if (t4 + 3 > r) w[t4 + 3] = fmaf(-m.w, w[r], w[t4 + 3]);
                if (t4 >= r) b[t4] = fmaf(n.x, w[r], b[t4]);
                if (t4 + 1 >= r) b[t4 + 1] = fmaf(n.y, w[r], b[t4 + 1]);
                if (t4 + 2 >= r) b[t4 + 2] = fmaf(n.z, w[r], b[t4 + 2]);
                if (t4 + 3 >= r) b[t4 + 3] = fmaf(n.w, w[r], b[t4 + 3]);
            }
        }
        if (!key) {
            float* u0 = a.u0 + at * DC_ROWS * a.dv + j - dp;
            float* y = a.y + ((size_t)row0 * a.heads + h) * a.dv + j - dp;
#pragma unroll
            for (int t = 0; t < DC_ROWS; ++t) {
                u0[t * a.dv] = w[t];
                if (t < rows) y[(size_t)t * a.heads * a.dv] = b[t];
            }
            continue;
        }
        float* out = a.mats + (at * dp + j) * DC_MATS;
        uint16_t* half = reinterpret_cast<uint16_t*>(ops_s);
        if (SPLIT) {
#pragma unroll
            for (int t = 0; t < DC_ROWS; ++t) {                // the two rows of a pair go to different tiles
                const Pieces x = split3(w[t], b[t]);
#pragma unroll
                for (int p = 0; p < 3; ++p) {
                    half[cm_m_half(p, t, j)] = (uint16_t)x.v[p];
                    half[cm_m_half(p, DC_ROWS + t, j)] = (uint16_t)(x.v[p] >> 16);
                }
            }
        } else {
#pragma unroll
            for (int t = 0; t < DC_ROWS; t += 4) {
                *reinterpret_cast<float4*>(out + t) = make_float4(w[t], w[t + 1], w[t + 2], w[t + 3]);
                *reinterpret_cast<float4*>(out + DC_ROWS + t) = make_float4(b[t], b[t + 1], b[t + 2], b[t + 3]);
            }
        }
        float E = 1.0f;
#pragma unroll
        for (int t = DC_ROWS - 1; t >= 0; --t) {
            w[t] = E * k_s[t * dp + j];
            E *= g_s[t * dp + j];
        }
        if (SPLIT) {
#pragma unroll
            for (int t = 0; t < DC_ROWS / 2; ++t) {
                const Pieces x = split3(w[2 * t], w[2 * t + 1]);
#pragma unroll
                for (int p = 0; p < 3; ++p) ops_s[cm_k_word(dp, p, t, j)] = x.v[p];
            }
        } else {
#pragma unroll
            for (int t = 0; t < DC_ROWS; t += 4)
                *reinterpret_cast<float4*>(out + 2 * DC_ROWS + t) = make_float4(w[t], w[t + 1], w[t + 2], w[t + 3]);
        }
    }
    if (SPLIT) {
        __syncthreads();
        uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<uint32_t*>(a.mats) + at * cm_words(dp));
        for (int i = threadIdx.x; i < cm_words(dp) / 4; i += DC_THREADS) dst[i] = reinterpret_cast<const uint4*>(ops_s)[i];
    }
}

// (2) a portion's chunks one after the other; a block owns DC_COLS columns of one head's state
constexpr int DC_COLS = 16;
constexpr int DC_LD = DC_MATS + 4;        // floats between two key channels in shared memory (20 mod 32: no bank twice)
constexpr int DC_WARPS = DC_THREADS / 32;

__device__ __forceinline__ void copy16_async(float* dst, const float* src) {
    const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(d), "l"(src) : "memory");
}

__host__ __device__ constexpr int delta_carry_floats(int dp) {
    return 2 * dp * DC_LD + 2 * dp + dp * DC_COLS + DC_WARPS * 2 * DC_ROWS * DC_COLS + DC_ROWS * DC_COLS;
}

__global__ void __launch_bounds__(DC_THREADS) delta_carry_kernel(DeltaArgs a) {
    extern __shared__ __align__(16) float carry_smem[];
    const int dp = a.dp, dv = a.dv;
    float* mats_s = carry_smem;                                // [2][dp][DC_LD]
    float* last_s = mats_s + 2 * dp * DC_LD;                   // [2][dp]
    float* S_s = last_s + 2 * dp;                              // [dp][DC_COLS]
    float* part_s = S_s + dp * DC_COLS;                        // [DC_WARPS][2 DC_ROWS][DC_COLS]
    float* U_s = part_s + DC_WARPS * 2 * DC_ROWS * DC_COLS;    // [DC_ROWS][DC_COLS]
    pdl_wait_only();
    const int* span = a.spans + 4 * blockIdx.z;
    const int req = span[0], chunk0 = span[1], n = span[2];
    const int h = blockIdx.y, c0 = blockIdx.x * DC_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float* st = a.state + (size_t)a.state_slots[req] * a.state_stride + ((size_t)h * dv + c0) * dp;

    auto fetch = [&](int i) {                                  // chunk i of the span into buffer i & 1
        const size_t at = (size_t)(chunk0 + i) * a.heads + h;
        float* m = mats_s + (i & 1) * dp * DC_LD;
        const float* src = a.mats + at * dp * DC_MATS;
        for (int p = tid; p < dp * (DC_MATS / 4); p += DC_THREADS)
            copy16_async(m + (p / (DC_MATS / 4)) * DC_LD + (p % (DC_MATS / 4)) * 4, src + (size_t)p * 4);
        for (int p = tid; p < dp / 4; p += DC_THREADS) copy16_async(last_s + (i & 1) * dp + 4 * p, a.last + at * dp + 4 * p);
        asm volatile("cp.async.commit_group;\n" ::: "memory");
    };
    fetch(0);
    for (int i = tid; i < dp * DC_COLS; i += DC_THREADS) {     // columns of the state are contiguous
        const int c = i / dp, e = i % dp;
        S_s[e * DC_COLS + c] = c0 + c < dv ? st[(size_t)c * dp + e] : 0.0f;
    }
    const int per = (dp + DC_WARPS - 1) / DC_WARPS;            // key channels a warp adds up
    const int k_lo = min(warp * per, dp), k_hi = min(k_lo + per, dp);
    const int rg = lane >> 2, cg = lane & 3;                   // four rows, four columns
    const int o_row = tid >> 3, o_col = (tid & 7) * 2;         // the two sums a thread closes: rows 0 .. 15 of U, 16 .. 31 of o
    for (int i = 0; i < n; ++i) {
        const int row0 = a.chunks[4 * (chunk0 + i)], rows = a.chunks[4 * (chunk0 + i) + 1];
        // what the closing sums start from: asked for before the products
        float base[2] = {0.0f, 0.0f};
        float* y = nullptr;
        if (o_row < DC_ROWS) {
            const float* u0 = a.u0 + (((size_t)(chunk0 + i) * a.heads + h) * DC_ROWS + o_row) * dv + c0 + o_col;
            if (c0 + o_col < dv) base[0] = u0[0];
            if (c0 + o_col + 1 < dv) base[1] = u0[1];
        } else if (o_row - DC_ROWS < rows) {
            y = a.y + ((size_t)(row0 + o_row - DC_ROWS) * a.heads + h) * dv + c0 + o_col;
            if (c0 + o_col < dv) base[0] = y[0];
            if (c0 + o_col + 1 < dv) base[1] = y[1];
        }
        if (i + 1 < n) {
            fetch(i + 1);                                      // its buffer was last read before the previous chunk's last barrier
            asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::: "memory");
        }
        __syncthreads();                                       // the chunk is there, and S with the chunk before in it
        const float* m = mats_s + (i & 1) * dp * DC_LD;
        const float* last = last_s + (i & 1) * dp;
        float acc[4][4] = {};
#pragma unroll 4
        for (int k = k_lo; k < k_hi; ++k) {
            const float4 x = *reinterpret_cast<const float4*>(m + k * DC_LD + 4 * rg);
            const float4 s = *reinterpret_cast<const float4*>(S_s + k * DC_COLS + 4 * cg);
            const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
            for (int p = 0; p < 4; ++p) {
                acc[p][0] = fmaf(xs[p], s.x, acc[p][0]);
                acc[p][1] = fmaf(xs[p], s.y, acc[p][1]);
                acc[p][2] = fmaf(xs[p], s.z, acc[p][2]);
                acc[p][3] = fmaf(xs[p], s.w, acc[p][3]);
            }
        }
#pragma unroll
        for (int p = 0; p < 4; ++p)
            *reinterpret_cast<float4*>(part_s + (warp * 2 * DC_ROWS + 4 * rg + p) * DC_COLS + 4 * cg) =
                make_float4(acc[p][0], acc[p][1], acc[p][2], acc[p][3]);
        __syncthreads();
        {
            float2 sum = make_float2(base[0], base[1]);
#pragma unroll
            for (int w = 0; w < DC_WARPS; ++w) {
                const float2 v = *reinterpret_cast<const float2*>(part_s + (w * 2 * DC_ROWS + o_row) * DC_COLS + o_col);
                sum.x += v.x;
                sum.y += v.y;
            }
            if (o_row < DC_ROWS) {
                *reinterpret_cast<float2*>(U_s + o_row * DC_COLS + o_col) = sum;
            } else if (y) {
                if (c0 + o_col < dv) y[0] = sum.x;
                if (c0 + o_col + 1 < dv) y[1] = sum.y;
            }
        }
        __syncthreads();
        {   // S <- last * S + keys U: a thread four columns of key channels tid / 4, tid / 4 + 64, ...
            const int c4 = (tid & 3) * 4;
            for (int k0 = tid >> 2; k0 < dp; k0 += 2 * (DC_THREADS / 4)) {
                const int k1 = k0 + DC_THREADS / 4;
                const bool two = k1 < dp;
                float4 s0 = *reinterpret_cast<const float4*>(S_s + k0 * DC_COLS + c4), s1 = make_float4(0, 0, 0, 0);
                const float f0 = last[k0];
                s0.x *= f0; s0.y *= f0; s0.z *= f0; s0.w *= f0;
                if (two) {
                    s1 = *reinterpret_cast<const float4*>(S_s + k1 * DC_COLS + c4);
                    const float f1 = last[k1];
                    s1.x *= f1; s1.y *= f1; s1.z *= f1; s1.w *= f1;
                }
#pragma unroll
                for (int r = 0; r < DC_ROWS; r += 4) {
                    const float4 x0 = *reinterpret_cast<const float4*>(m + k0 * DC_LD + 2 * DC_ROWS + r);
                    float4 x1 = make_float4(0, 0, 0, 0);
                    if (two) x1 = *reinterpret_cast<const float4*>(m + k1 * DC_LD + 2 * DC_ROWS + r);
                    const float p0[4] = {x0.x, x0.y, x0.z, x0.w}, p1[4] = {x1.x, x1.y, x1.z, x1.w};
#pragma unroll
                    for (int p = 0; p < 4; ++p) {
                        const float4 u = *reinterpret_cast<const float4*>(U_s + (r + p) * DC_COLS + c4);
                        s0.x = fmaf(p0[p], u.x, s0.x); s0.y = fmaf(p0[p], u.y, s0.y);
                        s0.z = fmaf(p0[p], u.z, s0.z); s0.w = fmaf(p0[p], u.w, s0.w);
                        s1.x = fmaf(p1[p], u.x, s1.x); s1.y = fmaf(p1[p], u.y, s1.y);
                        s1.z = fmaf(p1[p], u.z, s1.z); s1.w = fmaf(p1[p], u.w, s1.w);
                    }
                }
                *reinterpret_cast<float4*>(S_s + k0 * DC_COLS + c4) = s0;
                if (two) *reinterpret_cast<float4*>(S_s + k1 * DC_COLS + c4) = s1;
            }
        }
        __syncthreads();                                       // the buffer may be filled again
    }
    for (int i = tid; i < dp * DC_COLS; i += DC_THREADS) {
        const int c = i / dp, e = i % dp;
        if (c0 + c < dv) st[(size_t)c * dp + e] = S_s[e * DC_COLS + c];
    }
}

// The same on the tensor cores.  A block owns DC_COLS columns of one head's state, a warp 16 KB of the key channels, as S^T
// in the layout of the accumulators of m16n8k16 (columns of S down, key channels across): two neighbouring tiles are at once
// the left operand of the product with the chunk's rows, so the state never leaves the registers.
//   P^T = S^T [-W | D q - B W]^T  (each warp its key channels; the parts are added in shared memory)
//   S^T <- last * S^T + U^T K     (U^T = U_0^T + P^T's first rows)
constexpr int CM_PART = 40;               // floats between two columns of a part (8 mod 32: no bank twice)

// acc[n] += a b[n] for N tiles, the six products of the pieces that count, a tile after the other for each of them
template <int N>
__device__ __forceinline__ void mma_split(float (*acc)[4], const uint32_t (&x)[3][4], const uint32_t (&b)[3][N][2]) {
    constexpr int order[6][2] = {{2, 0}, {0, 2}, {1, 1}, {1, 0}, {0, 1}, {0, 0}};
#pragma unroll
    for (int o = 0; o < 6; ++o)
#pragma unroll
        for (int n = 0; n < N; ++n) mma16::mma_bf16(acc[n], x[order[o][0]], b[order[o][1]][n][0], b[order[o][1]][n][1]);
}

// Two tiles: the three smaller products in sums of their own, so that no accumulator waits for six products in a row.
__device__ __forceinline__ void mma_split_pair(float (*acc)[4], const uint32_t (&x)[3][4], const uint32_t (&b)[3][2][2]) {
    float small[2][4] = {};
    constexpr int order[3][4] = {{2, 0, 1, 0}, {0, 2, 0, 1}, {1, 1, 0, 0}};
#pragma unroll
    for (int o = 0; o < 3; ++o) {
#pragma unroll
        for (int n = 0; n < 2; ++n) mma16::mma_bf16(small[n], x[order[o][0]], b[order[o][1]][n][0], b[order[o][1]][n][1]);
#pragma unroll
        for (int n = 0; n < 2; ++n) mma16::mma_bf16(acc[n], x[order[o][2]], b[order[o][3]][n][0], b[order[o][3]][n][1]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][e] += small[n][e];
}

constexpr int carry_mma_words(int warps, int kb) {             // 32-bit words of shared memory
    return 2 * cm_words(16 * warps * kb) + warps * DC_COLS * CM_PART + 3 * 128;
}

template <int WARPS, int KB>
__global__ void __launch_bounds__(WARPS * 32) delta_carry_mma_kernel(DeltaArgs a) {
    constexpr int THREADS = WARPS * 32, DP = 16 * WARPS * KB, BUF = cm_words(DP);
    extern __shared__ __align__(16) uint32_t cm_smem[];
    float* part_s = reinterpret_cast<float*>(cm_smem + 2 * BUF);               // [WARPS][DC_COLS][CM_PART]
    uint32_t* u_s = cm_smem + 2 * BUF + WARPS * DC_COLS * CM_PART;             // [3][32 lanes][4]: U^T as a left operand
    pdl_wait_only();
    const int* span = a.spans + 4 * blockIdx.z;
    const int req = span[0], chunk0 = span[1], n_chunks = span[2];
    const int h = blockIdx.y, c0 = blockIdx.x * DC_COLS, dv = a.dv;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    float* st = a.state + (size_t)a.state_slots[req] * a.state_stride + ((size_t)h * dv + c0) * DP;

    auto fetch = [&](int i) {                                  // chunk i of the span into buffer i & 1
        const uint32_t* src = reinterpret_cast<const uint32_t*>(a.mats) + ((size_t)(chunk0 + i) * a.heads + h) * BUF + 4 * tid;
        uint32_t* dst = cm_smem + (i & 1) * BUF + 4 * tid;
#pragma unroll
        for (int p = 0; p < (BUF / 4 + THREADS - 1) / THREADS; ++p)
            if (tid + p * THREADS < BUF / 4) mma16::cp_async_16(dst + 4 * p * THREADS, src + 4 * p * THREADS, 16);
        mma16::cp_async_commit();
    };
    fetch(0);
    const bool in0 = c0 + g < dv, in1 = c0 + g + 8 < dv;
    float S[2 * KB][4];
    float* own = st + (size_t)g * DP + 16 * KB * warp + 2 * t;                 // the warp's key channels
#pragma unroll
    for (int n = 0; n < 2 * KB; ++n) {
        const float2 x = in0 ? *reinterpret_cast<const float2*>(own + 8 * n) : make_float2(0.0f, 0.0f);
        const float2 y = in1 ? *reinterpret_cast<const float2*>(own + 8 * DP + 8 * n) : make_float2(0.0f, 0.0f);
        S[n][0] = x.x; S[n][1] = x.y; S[n][2] = y.x; S[n][3] = y.y;
    }
    // the closing sums: task (row tile n, column half) of 32 lanes each, a lane rows 8n + 2t, + 1 of column g + 8 half; tiles
    // 0 and 1 are U, 2 and 3 the outputs
    constexpr int TASKS = (8 + WARPS - 1) / WARPS;
    // what the sums start from, asked for a chunk ahead (a portion's chunks lie end to end, all but the last of DC_ROWS rows)
    const int first = a.chunks[4 * chunk0], total = (n_chunks - 1) * DC_ROWS + a.chunks[4 * (chunk0 + n_chunks - 1) + 1];
    float* from[TASKS];
    size_t step[TASKS], next_row[TASKS];                       // to the next chunk, to the second of the two rows
    float2 base[TASKS], ahead[TASKS];
#pragma unroll
    for (int k = 0; k < TASKS; ++k) {
        const int task = warp + k * WARPS, n = task >> 1, col = c0 + g + 8 * (task & 1), r = 8 * (n & 1) + 2 * t;
        const bool u = n < 2;
        next_row[k] = u ? dv : (size_t)a.heads * dv;
        step[k] = (size_t)DC_ROWS * a.heads * dv;
        from[k] = u ? a.u0 + (((size_t)chunk0 * a.heads + h) * DC_ROWS + r) * dv + col
                    : a.y + ((size_t)(first + r) * a.heads + h) * dv + col;
        if (task >= 8 || col >= dv) from[k] = nullptr;
    }
    auto ask = [&](int i) {
#pragma unroll
        for (int k = 0; k < TASKS; ++k) {
            const int n = (warp + k * WARPS) >> 1, r = 8 * (n & 1) + 2 * t;
            const int left = n < 2 ? DC_ROWS : total - i * DC_ROWS;
            const float* p = from[k] + i * step[k];
            ahead[k].x = from[k] && r < left ? p[0] : 0.0f;
            ahead[k].y = from[k] && r + 1 < left ? p[next_row[k]] : 0.0f;
        }
    };
    ask(0);
    for (int i = 0; i < n_chunks; ++i) {
#pragma unroll
        for (int k = 0; k < TASKS; ++k) base[k] = ahead[k];
        if (i + 1 < n_chunks) ask(i + 1);
        mma16::cp_async_wait<0>();
        __syncthreads();                                       // the chunk is there, and everyone is done with the one before
        if (i + 1 < n_chunks) fetch(i + 1);
        const uint4* M = reinterpret_cast<const uint4*>(cm_smem + (i & 1) * BUF) + lane;
        float P[4][4] = {};                                    // P^T: a tile eight of the 32 rows
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) {
            uint32_t b[3][4][2];
#pragma unroll
            for (int p = 0; p < 3; ++p)
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const uint4 v = M[(((warp * KB + kb) * 3 + p) * 2 + n) * 32];
                    b[p][2 * n][0] = v.x; b[p][2 * n][1] = v.y; b[p][2 * n + 1][0] = v.z; b[p][2 * n + 1][1] = v.w;
                }
            uint32_t x[3][4];
#pragma unroll
            for (int r = 0; r < 4; ++r) {                      // (g, 2t..), (g + 8, 2t..), (g, 2t + 8..), (g + 8, 2t + 8..)
                const float* s = S[2 * kb + (r >> 1)] + 2 * (r & 1);
                const Pieces v = split3(s[0], s[1]);
                x[0][r] = v.v[0]; x[1][r] = v.v[1]; x[2][r] = v.v[2];
            }
            mma_split<4>(P, x, b);
        }
        float* part = part_s + warp * DC_COLS * CM_PART + g * CM_PART + 2 * t;
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            *reinterpret_cast<float2*>(part + 8 * n) = make_float2(P[n][0], P[n][1]);
            *reinterpret_cast<float2*>(part + 8 * CM_PART + 8 * n) = make_float2(P[n][2], P[n][3]);
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TASKS; ++k) {
            const int task = warp + k * WARPS, n = task >> 1, half = task & 1;
            if (task >= 8) break;
            const float* src = part_s + (g + 8 * half) * CM_PART + 8 * n + 2 * t;
            float2 v[WARPS];
#pragma unroll
            for (int w = 0; w < WARPS; ++w) v[w] = *reinterpret_cast<const float2*>(src + w * DC_COLS * CM_PART);
            float2 sum = base[k];
#pragma unroll
            for (int w = 0; w < WARPS; w += 2) {
                sum.x += v[w].x + v[w + 1].x;
                sum.y += v[w].y + v[w + 1].y;
            }
            if (n < 2) {
                const Pieces x = split3(sum.x, sum.y);
#pragma unroll
                for (int p = 0; p < 3; ++p) u_s[(p * 32 + lane) * 4 + 2 * n + half] = x.v[p];
            } else if (from[k]) {
                const int r = 8 * (n & 1) + 2 * t, left = total - i * DC_ROWS;
                float* p = from[k] + i * step[k];
                if (r < left) p[0] = sum.x;
                if (r + 1 < left) p[next_row[k]] = sum.y;
            }
        }
        // what does not wait for U: the keys and the decay of the state
        const uint4* K = M + DP / 16 * CM_M_WORDS / 4;
        const float* last = reinterpret_cast<const float*>(cm_smem + (i & 1) * BUF + BUF - DP) + 16 * KB * warp + 2 * t;
        uint32_t b[KB][3][2][2];
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) {
#pragma unroll
            for (int p = 0; p < 3; ++p) {
                const uint4 v = K[((warp * KB + kb) * 3 + p) * 32];
                b[kb][p][0][0] = v.x; b[kb][p][0][1] = v.y; b[kb][p][1][0] = v.z; b[kb][p][1][1] = v.w;
            }
#pragma unroll
            for (int n = 2 * kb; n < 2 * kb + 2; ++n) {
                const float2 f = *reinterpret_cast<const float2*>(last + 8 * n);
                S[n][0] *= f.x; S[n][1] *= f.y; S[n][2] *= f.x; S[n][3] *= f.y;
            }
        }
        __syncthreads();
        uint32_t x[3][4];
#pragma unroll
        for (int p = 0; p < 3; ++p) {
            const uint4 v = *reinterpret_cast<const uint4*>(u_s + (p * 32 + lane) * 4);
            x[p][0] = v.x; x[p][1] = v.y; x[p][2] = v.z; x[p][3] = v.w;
        }
#pragma unroll
        for (int kb = 0; kb < KB; ++kb) mma_split_pair(S + 2 * kb, x, b[kb]);
    }
#pragma unroll
    for (int n = 0; n < 2 * KB; ++n) {
        if (in0) *reinterpret_cast<float2*>(own + 8 * n) = make_float2(S[n][0], S[n][1]);
        if (in1) *reinterpret_cast<float2*>(own + 8 * DP + 8 * n) = make_float2(S[n][2], S[n][3]);
    }
}

template <int WARPS, int KB>
static int launch_carry_mma(const DeltaArgs& a, int n_spans, cudaStream_t stream) {
    constexpr int smem = carry_mma_words(WARPS, KB) * 4;
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(delta_carry_mma_kernel<WARPS, KB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
            return SHARPI_LAUNCH_FAILED;
        configured = true;
    }
    delta_carry_mma_kernel<WARPS, KB><<<dim3((a.dv + DC_COLS - 1) / DC_COLS, a.heads, n_spans), WARPS * 32, smem, stream>>>(a);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// `chunks` int32 [n_chunks, 4] (first row, rows <= DC_ROWS, request, unused), a request's one after the other; `spans` int32
// [n_spans, 4] (request, first chunk, number of chunks, unused); scratch: `mats` [n_chunks * heads * dp * (split ? 73 : 48)],
// `last` [n_chunks * heads * dp], `u0` [n_chunks * heads * DC_ROWS * dv] floats, each on 16 bytes.  `split`: the walk over
// the chunks on the tensor cores (d a multiple of 64).
SHARPI_API int sharpi_delta_chunks(const float* qkv, const float* beta, const float* z, int ldz, const float* dt_bias,
                                   const float* a_log, const int* row_offsets, const int* state_slots, const int* chunks,
                                   int n_chunks, const int* spans, int n_spans, float* mats, float* last, float* u0,
                                   float* state, long long state_stride, float* y, int kvh, int heads, int d, int dv,
                                   int split, cudaStream_t stream) {
    if (n_chunks <= 0) return SHARPI_OK;
    DeltaArgs a;
    if (n_spans <= 0 || n_spans > 65535 || d > DELTA_MAX_CHUNK_KEY ||
        !fill_delta(a, qkv, beta, z, ldz, dt_bias, a_log, row_offsets, state_slots, state, state_stride, y, kvh, heads, d, dv))
        return SHARPI_BAD_ARGUMENT;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(mats) | reinterpret_cast<uintptr_t>(last);
    if ((ptrs & 15) != 0) return SHARPI_UNALIGNED;
    a.chunks = chunks; a.spans = spans; a.mats = mats; a.last = last; a.u0 = u0;
    if (split && d % 64 != 0) return SHARPI_BAD_ARGUMENT;
    const size_t smem1 = ((size_t)3 * DC_ROWS * a.dp + (split ? cm_words(a.dp) : 0)) * sizeof(float), smem2 = (size_t)delta_carry_floats(a.dp) * sizeof(float);
    static bool configured = false;
    if (!configured) {
        const int most = (int)((3 * DC_ROWS * DELTA_MAX_CHUNK_KEY + cm_words(DELTA_MAX_CHUNK_KEY)) * sizeof(float));
        if (cudaFuncSetAttribute(delta_chunk_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess ||
            cudaFuncSetAttribute(delta_chunk_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, most) != cudaSuccess ||
            cudaFuncSetAttribute(delta_carry_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                 (int)(delta_carry_floats(DELTA_MAX_CHUNK_KEY) * sizeof(float))) != cudaSuccess)
            return SHARPI_LAUNCH_FAILED;
        configured = true;
    }
    // the walk over the chunks is launched the plain way: its blocks run long and are to lie evenly over an empty GPU
    if (split) {
        SHARPI_LAUNCH_PDL(delta_chunk_kernel<true>, dim3(n_chunks, heads), DC_THREADS, smem1, stream, a);
        switch (d / 64) {
            case 1: return launch_carry_mma<4, 1>(a, n_spans, stream);
            case 2: return launch_carry_mma<8, 1>(a, n_spans, stream);
            case 3: return launch_carry_mma<6, 2>(a, n_spans, stream);
            default: return launch_carry_mma<8, 2>(a, n_spans, stream);
        }
    }
    SHARPI_LAUNCH_PDL(delta_chunk_kernel<false>, dim3(n_chunks, heads), DC_THREADS, smem1, stream, a);
    delta_carry_kernel<<<dim3((dv + DC_COLS - 1) / DC_COLS, heads, n_spans), DC_THREADS, smem2, stream>>>(a);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// -------------------------------------------------------------------------------------------------------------
// norm per head, weight, sigmoid gate
// -------------------------------------------------------------------------------------------------------------
constexpr int HNG_PER = 8;                // elements a lane keeps; longer heads are read twice

template <typename TO>
__global__ void __launch_bounds__(128)
head_norm_gate_kernel(const float* y, const float* gate, int ld_g, const float* __restrict__ w, float eps, int heads, int dv,
                      long long total, TO* out) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);        // row * heads + head
    if (i >= total) return;
    const int lane = threadIdx.x & 31, h = (int)(i % heads);
    const float* src = y + (size_t)i * dv;
    const float* g = gate + (size_t)(i / heads) * ld_g + (size_t)h * dv;
    float v[HNG_PER], gg[HNG_PER];
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < HNG_PER; ++k) {
        const int e = lane + 32 * k;
        v[k] = e < dv ? src[e] : 0.0f;
        gg[k] = e < dv ? g[e] : 0.0f;
    }
#pragma unroll
    for (int k = 0; k < HNG_PER; ++k) ss = fmaf(v[k], v[k], ss);
    for (int e = lane + 32 * HNG_PER; e < dv; e += 32) ss = fmaf(src[e], src[e], ss);
    const float f = 1.0f / sqrtf(warp_sum(ss) / (float)dv + eps);
    TO* o = out + (size_t)i * dv;
#pragma unroll
    for (int k = 0; k < HNG_PER; ++k) {
        const int e = lane + 32 * k;
        if (e < dv) o[e] = from_float<TO>(v[k] * f * w[e] * sigmoid_f(gg[k]));
    }
    for (int e = lane + 32 * HNG_PER; e < dv; e += 32) o[e] = from_float<TO>(src[e] * f * w[e] * sigmoid_f(g[e]));
}

SHARPI_API int sharpi_head_norm_gate(const float* y, const float* gate, int ld_g, const float* w, float eps, int T, int heads,
                                     int dv, void* out, int out_dtype, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (heads <= 0 || dv <= 0 || ld_g < heads * dv) return SHARPI_BAD_ARGUMENT;
    const long long total = (long long)T * heads;
    const unsigned blocks = (unsigned)((total + 3) / 4);
    if (out_dtype == SHARPI_F32)
        SHARPI_LAUNCH_PDL(head_norm_gate_kernel<float>, blocks, 128, 0, stream, y, gate, ld_g, w, eps, heads, dv, total, (float*)out);
    else if (out_dtype == SHARPI_BF16)
        SHARPI_LAUNCH_PDL(head_norm_gate_kernel<bf16>, blocks, 128, 0, stream, y, gate, ld_g, w, eps, heads, dv, total, (bf16*)out);
    else
        return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}
