// Blocks whose sublayer outputs are normed before they enter the residual stream, and what stands around them.
//
//   sharpi_add_normed     x[t] += y[t] / sqrt(mean(y[t]^2) + eps) * wy, then out[t] = x[t] / sqrt(mean(x[t]^2) + eps) * w, or
//                         x[t] itself where there is no w (a sublayer that reads the bare stream).  A layer scale is a
//                         factor of wy.  With `rows` only those rows are formed and x stays as it is.  `out32`
//                         (nullable): the same values unrounded.
//   sharpi_embed_pos      out[t] = table[id[t]] * scale + pos[position[t]]
//   sharpi_side_gate      out[t, j] = gelu_tanh(gate[t, j]) * table[id[t], col0 + j] for j < n, zeros up to n_out: a
//                         token's own vector through a gate that reads the stream.
//
// The stream, the updates, sums of squares and weights are float32.
#include "common.cuh"

// ---------------------------------------------------------------------------------------
// Rows of up to SW_VT * 4 * VPT elements in registers.  A row belongs to SW_VT "virtual" threads of VPT float4 each;
// THREADS real ones stand for SW_VT / THREADS of them.  The sums are formed per virtual warp and then over the virtual
// warps, so a row gives the same bits whichever block size a step of its size takes.
// ---------------------------------------------------------------------------------------
struct NormedArgs {
    float* x;
    const float* y;
    const float* wy;
    const float* w;
    const int* rows;
    float* out32;
    float eps;
    int H;
};

template <int NV, int VT, int THREADS>
__device__ __forceinline__ float virtual_block_sum(const float* ss, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float s[NV];
#pragma unroll
    for (int a = 0; a < NV; ++a) s[a] = warp_sum(ss[a]);
    __syncthreads();
    if (lane == 0) {
#pragma unroll
        for (int a = 0; a < NV; ++a) scratch[warp + (THREADS / 32) * a] = s[a];
    }
    __syncthreads();
    return warp_sum(lane < VT / 32 ? scratch[lane] : 0.0f);
}

template <typename TO> __device__ __forceinline__ void store4(TO* p, const float* v);
template <> __device__ __forceinline__ void store4<float>(float* p, const float* v) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float* v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 r;
    r.x = *reinterpret_cast<unsigned*>(&a);
    r.y = *reinterpret_cast<unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
}

template <typename TO, int VT, int THREADS, int VPT>
__global__ void __launch_bounds__(THREADS) add_normed_kernel(NormedArgs a, TO* __restrict__ out) {
    constexpr int NV = VT / THREADS;
    __shared__ float scratch[32];
    pdl_wait();
    const int t = blockIdx.x, H = a.H;
    const size_t src = (size_t)(a.rows ? a.rows[t] : t) * H;
    float4 x[NV][VPT], y[NV][VPT];
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int p = 0; p < VPT; ++p) {
            const int i = (threadIdx.x + n * THREADS + p * VT) * 4;
            y[n][p] = i < H ? *reinterpret_cast<const float4*>(a.y + src + i) : make_float4(0, 0, 0, 0);
            x[n][p] = i < H ? *reinterpret_cast<const float4*>(a.x + src + i) : make_float4(0, 0, 0, 0);
        }
    float ss[NV];
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        ss[n] = 0.0f;
#pragma unroll
        for (int p = 0; p < VPT; ++p)
            ss[n] += (y[n][p].x * y[n][p].x + y[n][p].y * y[n][p].y) + (y[n][p].z * y[n][p].z + y[n][p].w * y[n][p].w);
    }
    const float sy = 1.0f / sqrtf(virtual_block_sum<NV, VT, THREADS>(ss, scratch) / (float)H + a.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
        ss[n] = 0.0f;
#pragma unroll
        for (int p = 0; p < VPT; ++p) {
            const int i = (threadIdx.x + n * THREADS + p * VT) * 4;
            if (i < H) {
                const float4 wy = *reinterpret_cast<const float4*>(a.wy + i);
                x[n][p].x += y[n][p].x * sy * wy.x;
                x[n][p].y += y[n][p].y * sy * wy.y;
                x[n][p].z += y[n][p].z * sy * wy.z;
                x[n][p].w += y[n][p].w * sy * wy.w;
                if (!a.rows) *reinterpret_cast<float4*>(a.x + src + i) = x[n][p];
            }
            ss[n] += (x[n][p].x * x[n][p].x + x[n][p].y * x[n][p].y) + (x[n][p].z * x[n][p].z + x[n][p].w * x[n][p].w);
        }
    }
    float sx = 1.0f;
    if (a.w) sx = 1.0f / sqrtf(virtual_block_sum<NV, VT, THREADS>(ss, scratch) / (float)H + a.eps);
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int p = 0; p < VPT; ++p) {
            const int i = (threadIdx.x + n * THREADS + p * VT) * 4;
            if (i < H) {
                float v[4] = {x[n][p].x, x[n][p].y, x[n][p].z, x[n][p].w};
                if (a.w) {
                    const float4 w = *reinterpret_cast<const float4*>(a.w + i);
                    v[0] = v[0] * sx * w.x; v[1] = v[1] * sx * w.y; v[2] = v[2] * sx * w.z; v[3] = v[3] * sx * w.w;
                }
                store4<TO>(out + (size_t)t * H + i, v);
                if (a.out32) store4<float>(a.out32 + (size_t)t * H + i, v);
            }
        }
}

// Any width: the row is read again for every pass.
template <typename TO>
__global__ void __launch_bounds__(256) add_normed_general_kernel(NormedArgs a, TO* out) {
    __shared__ float scratch[32];
    pdl_wait();
    const int t = blockIdx.x, H = a.H;
    const size_t src = (size_t)(a.rows ? a.rows[t] : t) * H;
    const float* y = a.y + src;
    float* x = a.x + src;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < H; i += 256) ss += y[i] * y[i];
    const float sy = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + a.eps);
    ss = 0.0f;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = x[i] + y[i] * sy * a.wy[i];
        ss += v * v;
    }
    float sx = 1.0f;
    if (a.w) sx = 1.0f / sqrtf(block_sum(ss, scratch) / (float)H + a.eps);
    for (int i = threadIdx.x; i < H; i += 256) {
        float v = x[i] + y[i] * sy * a.wy[i];
        if (!a.rows) x[i] = v;
        if (a.w) v = v * sx * a.w[i];
        out[(size_t)t * H + i] = from_float<TO>(v);
        if (a.out32) a.out32[(size_t)t * H + i] = v;
    }
}

constexpr int SW_SMALL_STEP = 128;       // rows up to which a row gets a block as wide as it can be

template <typename TO>
static int launch_normed(const NormedArgs& a, TO* out, int T, cudaStream_t stream) {
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.y) | reinterpret_cast<uintptr_t>(a.wy) |
                           reinterpret_cast<uintptr_t>(a.w) | reinterpret_cast<uintptr_t>(a.out32) | reinterpret_cast<uintptr_t>(out);
    const int H = a.H;
    if (H % 4 != 0 || (ptrs & 15) != 0 || H > 16384) {
        SHARPI_LAUNCH_PDL(add_normed_general_kernel<TO>, T, 256, 0, stream, a, out);
        return SHARPI_OK;
    }
    if (H <= 1024) {
        SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 256, 256, 1>), T, 256, 0, stream, a, out);
    } else if (H <= 4096) {
        if (T <= SW_SMALL_STEP) SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 1024, 1024, 1>), T, 1024, 0, stream, a, out);
        else SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 1024, 256, 1>), T, 256, 0, stream, a, out);
    } else if (H <= 8192) {
        if (T <= SW_SMALL_STEP) SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 1024, 1024, 2>), T, 1024, 0, stream, a, out);
        else SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 1024, 512, 2>), T, 512, 0, stream, a, out);
    } else {
        SHARPI_LAUNCH_PDL((add_normed_kernel<TO, 1024, 1024, 4>), T, 1024, 0, stream, a, out);
    }
    return SHARPI_OK;
}

// `w` null: the bare stream; `rows` (nullable): T row indices, x is left as it is
SHARPI_API int sharpi_add_normed(float* x, const float* y, const float* wy, const float* w, float eps, const int* rows, int T,
                                 int H, void* out, int out_dtype, float* out32, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || !x || !y || !wy) return SHARPI_BAD_ARGUMENT;
    NormedArgs a;
    a.x = x; a.y = y; a.wy = wy; a.w = w; a.rows = rows; a.out32 = out32; a.eps = eps; a.H = H;
    if (out_dtype == SHARPI_F32) return launch_normed<float>(a, (float*)out, T, stream);
    if (out_dtype == SHARPI_BF16) return launch_normed<bf16>(a, (bf16*)out, T, stream);
    return SHARPI_BAD_ARGUMENT;
}

// ---------------------------------------------------------------------------------------
template <typename TT>
__global__ void __launch_bounds__(256)
embed_pos_kernel(const int* ids, const int* positions, const TT* __restrict__ table, const TT* __restrict__ pos, float scale,
                 float* out, int H, int V, int P) {
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t], p = positions[t];
    const bool ok = id >= 0 && id < V && p >= 0 && p < P;      // the host checks both before the launch
    const TT* e = table + (size_t)(ok ? id : 0) * H;
    const TT* q = pos + (size_t)(ok ? p : 0) * H;
    for (int i = threadIdx.x + blockIdx.y * 256; i < H; i += 256 * gridDim.y)
        out[(size_t)t * H + i] = ok ? to_float(e[i]) * scale + to_float(q[i]) : 0.0f;
}

SHARPI_API int sharpi_embed_pos(const int* ids, const int* positions, const void* table, const void* pos, int table_dtype,
                                float scale, float* out, int T, int H, int V, int P, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || V <= 0 || P <= 0) return SHARPI_BAD_ARGUMENT;
    const dim3 grid(T, H > 2048 ? (H + 2047) / 2048 : 1);
    if (table_dtype == SHARPI_F32)
        SHARPI_LAUNCH_PDL(embed_pos_kernel<float>, grid, 256, 0, stream, ids, positions, (const float*)table, (const float*)pos,
                          scale, out, H, V, P);
    else if (table_dtype == SHARPI_BF16)
        SHARPI_LAUNCH_PDL(embed_pos_kernel<bf16>, grid, 256, 0, stream, ids, positions, (const bf16*)table, (const bf16*)pos,
                          scale, out, H, V, P);
    else
        return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename TT, typename TO, int VEC>                    // VEC neighbouring columns a thread
__global__ void __launch_bounds__(128)
side_gate_kernel(const float* gate, int ld, const int* ids, const TT* __restrict__ table, long long ld_table, int col0, int n,
                 int n_out, TO* out, unsigned total, int V) {
    pdl_wait();
    const unsigned i = blockIdx.x * 128 + threadIdx.x;
    if (i >= total) return;
    const unsigned per = n_out / VEC;
    const int t = (int)(i / per), j = (int)(i % per) * VEC;
    const int id = ids[t];
    const bool ok = id >= 0 && id < V;
    const TT* e = table + (size_t)(ok ? id : 0) * ld_table + col0 + j;
    const float* z = gate + (size_t)t * ld + j;
    float g[VEC], v[VEC];
#pragma unroll
    for (int u = 0; u < VEC; ++u) g[u] = j + u < n ? z[u] : 0.0f;
#pragma unroll
    for (int u = 0; u < VEC; ++u) v[u] = ok && j + u < n ? to_float(e[u]) : 0.0f;
#pragma unroll
    for (int u = 0; u < VEC; ++u) v[u] *= gelu_tanh_f(g[u]);
    if (VEC == 4) {
        store4<TO>(out + (size_t)t * n_out + j, v);
    } else {
        out[(size_t)t * n_out + j] = from_float<TO>(v[0]);
    }
}

SHARPI_API int sharpi_side_gate(const float* gate, int ld, const int* ids, const void* table, int table_dtype, long long ld_table,
                                int col0, int n, int n_out, void* out, int out_dtype, int T, int V, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (n <= 0 || n_out < n || col0 < 0 || col0 + n > ld_table || ld < n || V <= 0) return SHARPI_BAD_ARGUMENT;
    const int vec = n_out % 4 == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0 ? 4 : 1;
    if ((long long)T * n_out > 0x7fffffffLL) return SHARPI_BAD_ARGUMENT;
    const unsigned total = (unsigned)T * (unsigned)(n_out / vec), blocks = (total + 127) / 128;
#define SIDE_CASE(TT, TO)                                                                                                      \
    do {                                                                                                                       \
        if (vec == 4)                                                                                                          \
            SHARPI_LAUNCH_PDL((side_gate_kernel<TT, TO, 4>), blocks, 128, 0, stream, gate, ld, ids, (const TT*)table, ld_table, \
                              col0, n, n_out, (TO*)out, total, V);                                                             \
        else                                                                                                                   \
            SHARPI_LAUNCH_PDL((side_gate_kernel<TT, TO, 1>), blocks, 128, 0, stream, gate, ld, ids, (const TT*)table, ld_table, \
                              col0, n, n_out, (TO*)out, total, V);                                                             \
    } while (0)
    if (table_dtype == SHARPI_F32 && out_dtype == SHARPI_F32) SIDE_CASE(float, float);
    else if (table_dtype == SHARPI_BF16 && out_dtype == SHARPI_BF16) SIDE_CASE(bf16, bf16);
    else if (table_dtype == SHARPI_F32 && out_dtype == SHARPI_BF16) SIDE_CASE(float, bf16);
    else if (table_dtype == SHARPI_BF16 && out_dtype == SHARPI_F32) SIDE_CASE(bf16, float);
    else return SHARPI_BAD_ARGUMENT;
#undef SIDE_CASE
    return SHARPI_OK;
}
