// Embedding lookup, residual-add + RMSNorm, SwiGLU and dtype casts.
//
// The residual stream is fp32 in both precisions; sums of squares, the rsqrt and the
// scaling are fp32.  Counterparts in the reference: llm_embed_lookup_f32
// (src/SharpInference.Cuda/CudaTextKernels.cs:944), llm_rmsnorm / llm_rmsnorm_batched
// (:199, :5819), add_inplace (src/SharpInference.Cuda/CudaKernels.cs:89) and llm_silu_mul
// (CudaTextKernels.cs:331); here the residual add is fused into the norm that follows it.
#include "common.cuh"

// ---------------------------------------------------------------------------------------
// out[t, :] = table[ids[t], :]           (fp32 residual stream)
// ---------------------------------------------------------------------------------------
template <typename TT>
__global__ void embed_gather_kernel(const int* __restrict__ ids, const TT* __restrict__ table,
                                    float* __restrict__ out, int H, int V) {
    const int t = blockIdx.x;
    int id = ids[t];
    const bool valid = (id >= 0 && id < V);
    const TT* row = table + (size_t)(valid ? id : 0) * H;
    float* dst = out + (size_t)t * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = valid ? to_float(row[i]) : 0.0f;
}

SHARPI_API int sharpi_embed_gather(const int* ids, const void* table, int table_dtype, float* out,
                                   int T, int H, int V, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || V <= 0) return SHARPI_BAD_ARGUMENT;
    const int threads = H >= 1024 ? 256 : 128;
    if (table_dtype == SHARPI_F32)
        embed_gather_kernel<float><<<T, threads, 0, stream>>>(ids, (const float*)table, out, H, V);
    else if (table_dtype == SHARPI_BF16)
        embed_gather_kernel<bf16><<<T, threads, 0, stream>>>(ids, (const bf16*)table, out, H, V);
    else
        return SHARPI_BAD_ARGUMENT;
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// Residual add + RMSNorm.
//   rows == nullptr:  x[t] += delta[t] (written back); out[t] = x[t] * rsqrt(mean(x[t]^2)+eps) * w
//                     (w == nullptr: the weightless norm, src/SharpInference.Cpu/SimdKernels.cs:4252-4283)
//   rows != nullptr:  r = rows[t]; v = x[r] + delta[r] (x untouched); out[t] = norm(v)
//   w2 / out2:        (sharpi_add_rmsnorm_pair) the same normalised row under a second weight, for blocks whose two
//                     sublayers read the same stream through norms of their own; `out32` is then the second's copy
// `out` has dtype out_dtype; `out32` (optional) receives the same values in fp32, for
// consumers that must not see them rounded (the expert router).
// One block of NORM_THREADS threads per row whatever the batch, so the order of the
// additions in the sum of squares never depends on what else is in the step.
// ---------------------------------------------------------------------------------------
constexpr int NORM_THREADS = 256;

// The row is read in pieces of NORM_UNROLL elements per thread whose loads are all issued before the first
// of them is used (a step of few rows is one block per row waiting for memory, nothing else), and kept in
// shared memory for the second pass when it fits (CACHED).  A thread still adds its squares in ascending
// order of the index, as a plain loop would.
constexpr int NORM_UNROLL = 8;
constexpr int NORM_CACHE_FLOATS = 12288;     // 48 KB

// WIDE_ORDER: the sum of squares is formed in the order of add_rmsnorm_wide_kernel below (as if 1024 threads each
// added their own elements and the block's tree were that of 32 warps), so that a row gives the same bits
// whichever of the two kernels a step of its size takes: this thread stands for the virtual threads
// t, t + 256, t + 512, t + 768.
template <typename TO, bool CACHED, bool WIDE_ORDER, bool PAIR = false>
__global__ void __launch_bounds__(NORM_THREADS)
add_rmsnorm_kernel(float* x, const float* __restrict__ delta, const float* __restrict__ w, float eps,
                   const int* __restrict__ rows, int H, TO* __restrict__ out, float* __restrict__ out32,
                   const float* __restrict__ w2, TO* __restrict__ out2) {
    __shared__ float scratch[32];
    extern __shared__ float row_s[];
    pdl_wait();
    const int t = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[t] : t) * H;
    float* xr = x + src;
    const float* dr = delta ? delta + src : nullptr;
    const bool write_back = dr && !rows;
    float ss = 0.0f;
    float ss4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
    for (int i0 = threadIdx.x; i0 < H; i0 += NORM_UNROLL * NORM_THREADS) {
        float v[NORM_UNROLL], d[NORM_UNROLL];
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            v[k] = (i < H) ? xr[i] : 0.0f;
            d[k] = (dr && i < H) ? dr[i] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            if (i < H) {
                if (dr) v[k] += d[k];
                if (write_back) xr[i] = v[k];
                if (CACHED) row_s[i] = v[k];
                if (WIDE_ORDER) ss4[k & 3] += v[k] * v[k];
                else ss += v[k] * v[k];
            }
        }
    }
    if (WIDE_ORDER) {
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
        for (int a = 0; a < 4; ++a) ss4[a] = warp_sum(ss4[a]);
        __syncthreads();
        if (lane == 0) {
#pragma unroll
            for (int a = 0; a < 4; ++a) scratch[warp + (NORM_THREADS / 32) * a] = ss4[a];   // virtual warp w + 8 a
        }
        __syncthreads();
        ss = warp_sum(scratch[lane]);
    } else {
        ss = block_sum(ss, scratch);
    }
    const float scale = 1.0f / sqrtf(ss / (float)H + eps);
    TO* orow = out + (size_t)t * H;
    float* o32 = out32 ? out32 + (size_t)t * H : nullptr;
    for (int i0 = threadIdx.x; i0 < H; i0 += NORM_UNROLL * NORM_THREADS) {
        float v[NORM_UNROLL], ww[NORM_UNROLL];
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            ww[k] = (i < H) ? (w ? w[i] : 1.0f) : 0.0f;
            if (CACHED) {
                v[k] = (i < H) ? row_s[i] : 0.0f;      // this thread wrote it
            } else {
                v[k] = (i < H) ? xr[i] : 0.0f;
                if (dr && rows && i < H) v[k] += dr[i];
            }
        }
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            if (i < H) {
                float y = v[k] * scale * ww[k];
                orow[i] = from_float<TO>(y);
                if (PAIR) {
                    y = v[k] * scale * w2[i];
                    out2[(size_t)t * H + i] = from_float<TO>(y);
                }
                if (o32) o32[i] = y;
            }
        }
    }
}

// Rows of up to NORM_WIDE_THREADS * NORM_UNROLL elements: 1024 threads hold the whole row in registers, so every
// load of the row, of the update and of the weight is issued before anything is used and the kernel is two trips to
// memory long (a decode step runs this kernel two or three times a layer with one block per row: its latency, not
// its bandwidth, is what counts there).  A thread adds its squares in ascending order of the index; the block's
// tree is fixed by the block size, so a row's result does not depend on the batch.
constexpr int NORM_WIDE_THREADS = 1024;
constexpr int NORM_WIDE_ROWS = 128;       // steps of up to this many rows take it

template <typename TO, bool PAIR = false>
__global__ void __launch_bounds__(NORM_WIDE_THREADS)
add_rmsnorm_wide_kernel(float* x, const float* __restrict__ delta, const float* __restrict__ w, float eps,
                        const int* __restrict__ rows, int H, TO* __restrict__ out, float* __restrict__ out32,
                        const float* __restrict__ w2, TO* __restrict__ out2) {
    __shared__ float scratch[32];
    // the weight is written by no kernel: it may be on its way before the kernel ahead has finished
    float ww[NORM_UNROLL], ww2[PAIR ? NORM_UNROLL : 1];
#pragma unroll
    for (int k = 0; k < NORM_UNROLL; ++k) {
        const int i = threadIdx.x + k * NORM_WIDE_THREADS;
        ww[k] = (i < H) ? (w ? w[i] : 1.0f) : 0.0f;
        if (PAIR) ww2[k] = (i < H) ? w2[i] : 0.0f;
    }
    pdl_wait();
    const int t = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[t] : t) * H;
    float* xr = x + src;
    const float* dr = delta ? delta + src : nullptr;
    const bool write_back = dr && !rows;
    float v[NORM_UNROLL], d[NORM_UNROLL];
#pragma unroll
    for (int k = 0; k < NORM_UNROLL; ++k) {
        const int i = threadIdx.x + k * NORM_WIDE_THREADS;
        v[k] = (i < H) ? xr[i] : 0.0f;
        d[k] = (dr && i < H) ? dr[i] : 0.0f;
    }
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NORM_UNROLL; ++k) {
        const int i = threadIdx.x + k * NORM_WIDE_THREADS;
        if (i < H) {
            if (dr) v[k] += d[k];
            if (write_back) xr[i] = v[k];
            ss += v[k] * v[k];
        }
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss / (float)H + eps);
    TO* orow = out + (size_t)t * H;
    float* o32 = out32 ? out32 + (size_t)t * H : nullptr;
#pragma unroll
    for (int k = 0; k < NORM_UNROLL; ++k) {
        const int i = threadIdx.x + k * NORM_WIDE_THREADS;
        if (i < H) {
            float y = v[k] * scale * ww[k];
            orow[i] = from_float<TO>(y);
            if (PAIR) {
                y = v[k] * scale * ww2[k];
                out2[(size_t)t * H + i] = from_float<TO>(y);
            }
            if (o32) o32[i] = y;
        }
    }
}

template <typename TO, bool PAIR = false>
static int launch_norm(float* x, const float* delta, const float* w, float eps, const int* rows, int T, int H, TO* out,
                       float* out32, cudaStream_t stream, const float* w2 = nullptr, TO* out2 = nullptr) {
    if (H <= NORM_WIDE_THREADS * NORM_UNROLL) {
        // few rows: latency counts (2.9 against 3.8 us at one row of 5120); many rows: bandwidth (33 against 49 us at
        // 2048 rows); the two kernels add in the same order, so the choice does not show in the result
        if (T <= NORM_WIDE_ROWS) {
            auto kern = add_rmsnorm_wide_kernel<TO, PAIR>;
            SHARPI_LAUNCH_PDL(kern, T, NORM_WIDE_THREADS, 0, stream, x, delta, w, eps, rows, H, out, out32, w2, out2);
        } else {
            auto kern = add_rmsnorm_kernel<TO, true, true, PAIR>;
            SHARPI_LAUNCH_PDL(kern, T, NORM_THREADS, (size_t)H * sizeof(float), stream, x, delta, w, eps, rows, H, out, out32, w2, out2);
        }
        return SHARPI_OK;
    }
    if (H <= NORM_CACHE_FLOATS) {
        auto kern = add_rmsnorm_kernel<TO, true, false, PAIR>;
        SHARPI_LAUNCH_PDL(kern, T, NORM_THREADS, (size_t)H * sizeof(float), stream, x, delta, w, eps, rows, H, out, out32, w2, out2);
    } else {
        auto kern = add_rmsnorm_kernel<TO, false, false, PAIR>;
        SHARPI_LAUNCH_PDL(kern, T, NORM_THREADS, 0, stream, x, delta, w, eps, rows, H, out, out32, w2, out2);
    }
    return SHARPI_OK;
}

SHARPI_API int sharpi_add_rmsnorm(float* x, const float* delta, const float* w, float eps, const int* rows,
                                  int T, int H, void* out, int out_dtype, float* out32, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0) return SHARPI_BAD_ARGUMENT;
    if (out_dtype == SHARPI_F32) return launch_norm<float>(x, delta, w, eps, rows, T, H, (float*)out, out32, stream);
    if (out_dtype == SHARPI_BF16) return launch_norm<bf16>(x, delta, w, eps, rows, T, H, (bf16*)out, out32, stream);
    return SHARPI_BAD_ARGUMENT;
}

SHARPI_API int sharpi_add_rmsnorm_pair(float* x, const float* delta, const float* w1, const float* w2, float eps, int T,
                                       int H, void* out1, void* out2, int out_dtype, float* out32, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || !w1 || !w2) return SHARPI_BAD_ARGUMENT;
    if (out_dtype == SHARPI_F32)
        return launch_norm<float, true>(x, delta, w1, eps, nullptr, T, H, (float*)out1, out32, stream, w2, (float*)out2);
    if (out_dtype == SHARPI_BF16)
        return launch_norm<bf16, true>(x, delta, w1, eps, nullptr, T, H, (bf16*)out1, out32, stream, w2, (bf16*)out2);
    return SHARPI_BAD_ARGUMENT;
}

// ---------------------------------------------------------------------------------------
// SwiGLU over a fused [M, 2I] gate|up product:  out[m, i] = silu(s*g) * (s*u),
// g = gate_up[m, i], u = gate_up[m, I + i], s = row_scale[scale_rows ? scale_rows[m] : m] or 1.
// The routed expert's router weight multiplies gate and up BEFORE the nonlinearity, which
// equals scaling the expert's input (src/SharpInference.Engine/ForwardPass.cs:2082-2088).
// ---------------------------------------------------------------------------------------
template <typename TO>
__global__ void swiglu_kernel(const float* __restrict__ gate_up, const float* __restrict__ row_scale,
                              const int* __restrict__ scale_rows, TO* __restrict__ out, int I) {
    const int m = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= I) return;
    const float s = row_scale ? row_scale[scale_rows ? scale_rows[m] : m] : 1.0f;
    const float g = gate_up[(size_t)m * 2 * I + i] * s;
    const float u = gate_up[(size_t)m * 2 * I + I + i] * s;
    const float act = g / (1.0f + expf(-g));
    out[(size_t)m * I + i] = from_float<TO>(act * u);
}

// Four elements per thread with 16-byte loads, for widths that are multiples of 4.
template <typename TO>
__global__ void swiglu_vec4_kernel(const float* __restrict__ gate_up, const float* __restrict__ row_scale,
                                   const int* __restrict__ scale_rows, TO* __restrict__ out, int I) {
    pdl_wait();
    const int m = blockIdx.x;
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (i >= I) return;
    const float s = row_scale ? row_scale[scale_rows ? scale_rows[m] : m] : 1.0f;
    const float4 g4 = *reinterpret_cast<const float4*>(gate_up + (size_t)m * 2 * I + i);
    const float4 u4 = *reinterpret_cast<const float4*>(gate_up + (size_t)m * 2 * I + I + i);
    const float g[4] = {g4.x * s, g4.y * s, g4.z * s, g4.w * s};
    const float u[4] = {u4.x * s, u4.y * s, u4.z * s, u4.w * s};
    TO* dst = out + (size_t)m * I + i;
#pragma unroll
    for (int j = 0; j < 4; ++j) dst[j] = from_float<TO>(g[j] / (1.0f + expf(-g[j])) * u[j]);
}

SHARPI_API int sharpi_swiglu(const float* gate_up, const float* row_scale, const int* scale_rows, void* out,
                             int out_dtype, int M, int I, cudaStream_t stream) {
    if (M <= 0) return SHARPI_OK;
    if (I <= 0 || (I + 255) / 256 > 65535) return SHARPI_BAD_ARGUMENT;
    if (I % 4 == 0 && (reinterpret_cast<uintptr_t>(gate_up) & 15) == 0) {
        dim3 grid4(M, (I / 4 + 255) / 256);
        if (out_dtype == SHARPI_F32)
            SHARPI_LAUNCH_PDL(swiglu_vec4_kernel<float>, grid4, 256, 0, stream, gate_up, row_scale, scale_rows, (float*)out, I);
        else if (out_dtype == SHARPI_BF16)
            SHARPI_LAUNCH_PDL(swiglu_vec4_kernel<bf16>, grid4, 256, 0, stream, gate_up, row_scale, scale_rows, (bf16*)out, I);
        else
            return SHARPI_BAD_ARGUMENT;
        SHARPI_CHECK_LAUNCH();
        return SHARPI_OK;
    }
    dim3 grid(M, (I + 255) / 256);
    if (out_dtype == SHARPI_F32)
        swiglu_kernel<float><<<grid, 256, 0, stream>>>(gate_up, row_scale, scale_rows, (float*)out, I);
    else if (out_dtype == SHARPI_BF16)
        swiglu_kernel<bf16><<<grid, 256, 0, stream>>>(gate_up, row_scale, scale_rows, (bf16*)out, I);
    else
        return SHARPI_BAD_ARGUMENT;
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// y[i] = a[i] + b[i] (fp32), used to combine a shared and a routed feed-forward output
// where no fused epilogue does it.
// ---------------------------------------------------------------------------------------
__global__ void add_kernel(const float* __restrict__ a, const float* __restrict__ b, float* __restrict__ y,
                           size_t n) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < n; i += stride) y[i] = a[i] + b[i];
}

SHARPI_API int sharpi_add(const float* a, const float* b, float* y, long long n, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    long long blocks = (n + 255) / 256;
    if (blocks > 148 * 32) blocks = 148 * 32;
    add_kernel<<<(int)blocks, 256, 0, stream>>>(a, b, y, (size_t)n);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// y[m, n] += bias[n]: the bias of a projection whose product came from the library.
__global__ void add_bias_kernel(float* __restrict__ y, const float* __restrict__ bias, int N) {
    pdl_wait();
    const int n = blockIdx.y * blockDim.x + threadIdx.x;
    if (n < N) y[(size_t)blockIdx.x * N + n] += bias[n];
}

SHARPI_API int sharpi_add_bias(float* y, const float* bias, int M, int N, cudaStream_t stream) {
    if (M <= 0 || N <= 0) return SHARPI_OK;
    if ((N + 255) / 256 > 65535) return SHARPI_BAD_ARGUMENT;
    dim3 grid(M, (N + 255) / 256);
    SHARPI_LAUNCH_PDL(add_bias_kernel, grid, 256, 0, stream, y, bias, N);
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// out[m, n] = act(y[m, n] + bias[n]): the activation of a feed-forward whose first product came back in fp32.
//   ACT_RELU2      max(z, 0)^2
//   ACT_GELU_TANH  0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
//   ACT_SILU       z / (1 + exp(-z))
//   ACT_SOFTPLUS   log(1 + exp(z))
// ---------------------------------------------------------------------------------------
enum SharpiAct : int { ACT_RELU2 = 0, ACT_GELU_TANH = 1, ACT_SILU = 2, ACT_SOFTPLUS = 3 };

template <int ACT> __device__ __forceinline__ float activate(float z) {
    if (ACT == ACT_RELU2) { const float r = fmaxf(z, 0.0f); return r * r; }
    if (ACT == ACT_GELU_TANH) return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    if (ACT == ACT_SOFTPLUS) return z > 20.0f ? z : log1pf(expf(z));
    return z / (1.0f + expf(-z));
}

template <typename TO, int ACT>
__global__ void bias_act_kernel(const float* __restrict__ y, const float* __restrict__ bias, TO* __restrict__ out,
                                int N) {
    pdl_wait();
    const size_t m = blockIdx.x;
    for (int n = blockIdx.y * blockDim.x + threadIdx.x; n < N; n += gridDim.y * blockDim.x) {
        const float z = y[m * N + n] + (bias ? bias[n] : 0.0f);
        out[m * N + n] = from_float<TO>(activate<ACT>(z));
    }
}

template <typename TO>
static int launch_bias_act(const float* y, const float* bias, TO* out, int M, int N, int act, cudaStream_t stream) {
    int by = (N + 255) / 256;
    if (by > 64) by = 64;
    const dim3 grid(M, by);
    if (act == ACT_RELU2) SHARPI_LAUNCH_PDL((bias_act_kernel<TO, ACT_RELU2>), grid, 256, 0, stream, y, bias, out, N);
    else if (act == ACT_GELU_TANH) SHARPI_LAUNCH_PDL((bias_act_kernel<TO, ACT_GELU_TANH>), grid, 256, 0, stream, y, bias, out, N);
    else if (act == ACT_SILU) SHARPI_LAUNCH_PDL((bias_act_kernel<TO, ACT_SILU>), grid, 256, 0, stream, y, bias, out, N);
    else if (act == ACT_SOFTPLUS) SHARPI_LAUNCH_PDL((bias_act_kernel<TO, ACT_SOFTPLUS>), grid, 256, 0, stream, y, bias, out, N);
    else return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

SHARPI_API int sharpi_bias_act(const float* y, const float* bias, void* out, int out_dtype, int M, int N, int act,
                               cudaStream_t stream) {
    if (M <= 0 || N <= 0) return SHARPI_OK;
    if (out_dtype == SHARPI_F32) return launch_bias_act<float>(y, bias, (float*)out, M, N, act, stream);
    if (out_dtype == SHARPI_BF16) return launch_bias_act<bf16>(y, bias, (bf16*)out, M, N, act, stream);
    return SHARPI_BAD_ARGUMENT;
}

// out[t, 0:H] = a[t] + delta[t] (delta nullable), out[t, H:2H] = b[t]: two streams side by side as the input of
// one product, in the dtype of that product's operand.
template <typename TO>
__global__ void concat2_kernel(const float* __restrict__ a, const float* __restrict__ delta,
                               const float* __restrict__ b, TO* __restrict__ out, int H) {
    pdl_wait();
    const size_t t = blockIdx.x;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = a[t * H + i] + (delta ? delta[t * H + i] : 0.0f);
        out[t * 2 * H + i] = from_float<TO>(v);
        out[t * 2 * H + H + i] = from_float<TO>(b[t * H + i]);
    }
}

SHARPI_API int sharpi_concat2(const float* a, const float* delta, const float* b, void* out, int out_dtype, int T,
                              int H, cudaStream_t stream) {
    if (T <= 0 || H <= 0) return SHARPI_OK;
    if (out_dtype == SHARPI_F32) SHARPI_LAUNCH_PDL(concat2_kernel<float>, T, 256, 0, stream, a, delta, b, (float*)out, H);
    else if (out_dtype == SHARPI_BF16) SHARPI_LAUNCH_PDL(concat2_kernel<bf16>, T, 256, 0, stream, a, delta, b, (bf16*)out, H);
    else return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

// The GPU's nanosecond clock into slot[index]: a marker between the launches of a stream, for timelines of a
// step taken inside a captured graph, where host-side timing sees nothing.
__global__ void timestamp_kernel(unsigned long long* slots, int index) {
    unsigned long long t;
    asm volatile("mov.u64 %0, %globaltimer;" : "=l"(t));
    slots[index] = t;
}

SHARPI_API int sharpi_timestamp(unsigned long long* slots, int index, cudaStream_t stream) {
    if (!slots || index < 0) return SHARPI_BAD_ARGUMENT;
    timestamp_kernel<<<1, 1, 0, stream>>>(slots, index);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// act(gate) * up over a fused [M, 2I] gate|up product, and tanh as one more plain activation
// (sharpi_act_only); a scale applied in place.
template <typename TO, int ACT>
__global__ void gated_act_kernel(const float* __restrict__ gate_up, TO* __restrict__ out, int I) {
    pdl_wait();
    const size_t m = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= I) return;
    const float g = gate_up[m * 2 * I + i], u = gate_up[m * 2 * I + I + i];
    out[m * I + i] = from_float<TO>(activate<ACT>(g) * u);
}

template <typename TO>
static int launch_gated_act(const float* gate_up, TO* out, int M, int I, int act, cudaStream_t stream) {
    const dim3 grid(M, (I + 255) / 256);
    if (act == ACT_RELU2) SHARPI_LAUNCH_PDL((gated_act_kernel<TO, ACT_RELU2>), grid, 256, 0, stream, gate_up, out, I);
    else if (act == ACT_GELU_TANH) SHARPI_LAUNCH_PDL((gated_act_kernel<TO, ACT_GELU_TANH>), grid, 256, 0, stream, gate_up, out, I);
    else if (act == ACT_SILU) SHARPI_LAUNCH_PDL((gated_act_kernel<TO, ACT_SILU>), grid, 256, 0, stream, gate_up, out, I);
    else return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

SHARPI_API int sharpi_gated_act(const float* gate_up, void* out, int out_dtype, int M, int I, int act,
                                cudaStream_t stream) {
    if (M <= 0 || I <= 0) return SHARPI_OK;
    if (out_dtype == SHARPI_F32) return launch_gated_act<float>(gate_up, (float*)out, M, I, act, stream);
    if (out_dtype == SHARPI_BF16) return launch_gated_act<bf16>(gate_up, (bf16*)out, M, I, act, stream);
    return SHARPI_BAD_ARGUMENT;
}

template <typename TO>
__global__ void tanh_kernel(const float* __restrict__ y, TO* __restrict__ out, long long n) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_float<TO>(tanhf(y[i]));
}

SHARPI_API int sharpi_tanh(const float* y, void* out, int out_dtype, long long n, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (out_dtype == SHARPI_F32) SHARPI_LAUNCH_PDL(tanh_kernel<float>, blocks, 256, 0, stream, y, (float*)out, n);
    else if (out_dtype == SHARPI_BF16) SHARPI_LAUNCH_PDL(tanh_kernel<bf16>, blocks, 256, 0, stream, y, (bf16*)out, n);
    else return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

__global__ void scale_kernel(float* y, float s, long long n) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) y[i] *= s;
}

SHARPI_API int sharpi_scale(float* y, float s, long long n, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    SHARPI_LAUNCH_PDL(scale_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, y, s, n);
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// Residual add fused with the element-wise squashing norm ("dynamic tanh"):
//   x += delta (in place unless `rows` gathers);  out = tanh(alpha * x) * w + b
// with one scalar alpha (read from device memory, so that a captured graph holds no copy of it), a weight and a
// bias vector.  No statistic of the row is formed, so every element stands alone: four elements a thread, rows
// in grid.y.  Same interface as sharpi_add_rmsnorm (optional unrounded float32 copy).
// ---------------------------------------------------------------------------------------
template <typename TO>
__global__ void __launch_bounds__(256)
add_dyt_kernel(float* x, const float* __restrict__ delta, const float* __restrict__ w, const float* __restrict__ b,
               const float* __restrict__ alpha, const int* __restrict__ rows, int H, TO* __restrict__ out,
               float* __restrict__ out32) {
    pdl_wait();
    const int t = blockIdx.y;
    const size_t src = (size_t)(rows ? rows[t] : t) * H;
    const float al = alpha[0];
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < H; i += gridDim.x * blockDim.x) {
        float v = x[src + i];
        if (delta) {
            v += delta[src + i];
            if (!rows) x[src + i] = v;
        }
        const float y = tanhf(al * v) * w[i] + (b ? b[i] : 0.0f);
        out[(size_t)t * H + i] = from_float<TO>(y);
        if (out32) out32[(size_t)t * H + i] = y;
    }
}

SHARPI_API int sharpi_add_dyt(float* x, const float* delta, const float* w, const float* b, const float* alpha,
                              const int* rows, int T, int H, void* out, int out_dtype, float* out32,
                              cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || T > 65535 * 1024 || !w || !alpha) return SHARPI_BAD_ARGUMENT;
    // rows in grid.y are limited to 65535: larger steps walk them in slices
    for (int t0 = 0; t0 < T; t0 += 65535) {
        const int n = T - t0 < 65535 ? T - t0 : 65535;
        const dim3 grid((H + 1023) / 1024 > 0 ? (H + 1023) / 1024 : 1, n);
        float* xs = rows ? x : x + (size_t)t0 * H;
        const float* ds = delta ? (rows ? delta : delta + (size_t)t0 * H) : nullptr;
        const int* rs = rows ? rows + t0 : nullptr;
        float* o32 = out32 ? out32 + (size_t)t0 * H : nullptr;
        if (out_dtype == SHARPI_F32)
            SHARPI_LAUNCH_PDL(add_dyt_kernel<float>, grid, 256, 0, stream, xs, ds, w, b, alpha, rs, H,
                              (float*)out + (size_t)t0 * H, o32);
        else if (out_dtype == SHARPI_BF16)
            SHARPI_LAUNCH_PDL(add_dyt_kernel<bf16>, grid, 256, 0, stream, xs, ds, w, b, alpha, rs, H,
                              (bf16*)out + (size_t)t0 * H, o32);
        else
            return SHARPI_BAD_ARGUMENT;
    }
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// Residual add fused with a layer norm that has a weight and a bias:
//   x += delta (in place unless `rows` gathers);  out = (x - mean) / sqrt(var + eps) * w + b
// with var the mean of the squared deviations from the mean (formed in a second pass over the row, not as
// E[x^2] - mean^2, so nothing cancels).  One block a row whatever the batch; a thread adds its elements in ascending
// order and the block's tree is fixed, so a row's numbers depend on the row alone.  The row stays in shared memory
// between the passes when it fits.  Same interface as sharpi_add_rmsnorm (optional unrounded float32 copy).
// ---------------------------------------------------------------------------------------
template <typename TO, bool CACHED>
__global__ void __launch_bounds__(NORM_THREADS)
add_layernorm_kernel(float* x, const float* __restrict__ delta, const float* __restrict__ w,
                     const float* __restrict__ b, float eps, const int* __restrict__ rows, int H,
                     TO* __restrict__ out, float* __restrict__ out32) {
    __shared__ float scratch[32];
    extern __shared__ float row_s[];
    pdl_wait();
    const int t = blockIdx.x;
    const size_t src = (size_t)(rows ? rows[t] : t) * H;
    float* xr = x + src;
    const float* dr = delta ? delta + src : nullptr;
    const bool write_back = dr && !rows;
    float sum = 0.0f;
    for (int i0 = threadIdx.x; i0 < H; i0 += NORM_UNROLL * NORM_THREADS) {
        float v[NORM_UNROLL], d[NORM_UNROLL];
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            v[k] = (i < H) ? xr[i] : 0.0f;
            d[k] = (dr && i < H) ? dr[i] : 0.0f;
        }
#pragma unroll
        for (int k = 0; k < NORM_UNROLL; ++k) {
            const int i = i0 + k * NORM_THREADS;
            if (i < H) {
                if (dr) v[k] += d[k];
                if (write_back) xr[i] = v[k];
                if (CACHED) row_s[i] = v[k];
                sum += v[k];
            }
        }
    }
    const float mean = block_sum(sum, scratch) / (float)H;
    // without the cache the row is read again: x already holds the sum unless the rows were gathered
    float sq = 0.0f;
    for (int i = threadIdx.x; i < H; i += NORM_THREADS) {
        const float v = CACHED ? row_s[i] : (xr[i] + ((dr && rows) ? dr[i] : 0.0f));
        sq += (v - mean) * (v - mean);
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)H + eps);
    TO* orow = out + (size_t)t * H;
    float* o32 = out32 ? out32 + (size_t)t * H : nullptr;
    for (int i = threadIdx.x; i < H; i += NORM_THREADS) {
        const float v = CACHED ? row_s[i] : (xr[i] + ((dr && rows) ? dr[i] : 0.0f));
        const float y = (v - mean) * inv * w[i] + (b ? b[i] : 0.0f);
        orow[i] = from_float<TO>(y);
        if (o32) o32[i] = y;
    }
}

template <typename TO>
static int launch_layernorm(float* x, const float* delta, const float* w, const float* b, float eps, const int* rows,
                            int T, int H, TO* out, float* out32, cudaStream_t stream) {
    if (H <= NORM_CACHE_FLOATS) {
        auto kern = add_layernorm_kernel<TO, true>;
        SHARPI_LAUNCH_PDL(kern, T, NORM_THREADS, (size_t)H * sizeof(float), stream, x, delta, w, b, eps, rows, H, out, out32);
    } else {
        auto kern = add_layernorm_kernel<TO, false>;
        SHARPI_LAUNCH_PDL(kern, T, NORM_THREADS, 0, stream, x, delta, w, b, eps, rows, H, out, out32);
    }
    return SHARPI_OK;
}

SHARPI_API int sharpi_add_layernorm(float* x, const float* delta, const float* w, const float* b, float eps,
                                    const int* rows, int T, int H, void* out, int out_dtype, float* out32,
                                    cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || !w) return SHARPI_BAD_ARGUMENT;
    if (out_dtype == SHARPI_F32) return launch_layernorm<float>(x, delta, w, b, eps, rows, T, H, (float*)out, out32, stream);
    if (out_dtype == SHARPI_BF16) return launch_layernorm<bf16>(x, delta, w, b, eps, rows, T, H, (bf16*)out, out32, stream);
    return SHARPI_BAD_ARGUMENT;
}

// out = o * sigmoid(g): a gate on the concatenated heads of a mixer, `o` in the activation dtype (the attention
// kernels' output), `g` the float32 product of the gate's projection ([rows, cols], rows `g_ld` floats apart); the
// sigmoid and the product are float32.
template <typename TO>
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(const TO* o, const float* g, TO* out, long long n, int cols,
                                                           int g_ld) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const long long gi = (g_ld == cols) ? i : (i / cols) * g_ld + i % cols;     // g may be a column range of a wider product
    out[i] = from_float<TO>(to_float(o[i]) / (1.0f + expf(-g[gi])));
}

SHARPI_API int sharpi_sigmoid_gate(const void* o, const float* g, void* out, int dtype, long long n, int cols, int g_ld,
                                   cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    if (cols <= 0 || g_ld < cols) return SHARPI_BAD_ARGUMENT;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (dtype == SHARPI_F32)
        SHARPI_LAUNCH_PDL(sigmoid_gate_kernel<float>, blocks, 256, 0, stream, (const float*)o, g, (float*)out, n, cols, g_ld);
    else if (dtype == SHARPI_BF16)
        SHARPI_LAUNCH_PDL(sigmoid_gate_kernel<bf16>, blocks, 256, 0, stream, (const bf16*)o, g, (bf16*)out, n, cols, g_ld);
    else
        return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

// ---------------------------------------------------------------------------------------
// The gated activation of a feed-forward with biases, written into a column range:
//   g = gate_up[m, i] + bias[i],  u = gate_up[m, I + i] + bias[I + i]        (bias nullable)
//   limit == 0:  out[m, i] = act(g) * u                                     (relu^2, tanh-GELU or SiLU)
//   limit > 0:   g = min(g, limit), u = clamp(u, -limit, limit), out[m, i] = g sigmoid(1.702 g) (u + 1)
// `out` rows are `ld` elements apart; behind the I elements `ones` columns of 1 and `zeros` columns of 0 are written (the
// product that reads the range can carry its bias as weight columns there, and a width its kernels like).
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ float clamped_gate(float g, float u, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}

template <typename TO, int ACT, bool CLAMP>
__global__ void __launch_bounds__(256)
gated_cols_kernel(const float* gate_up, const float* __restrict__ bias, TO* out, int I, int ld, int ones, int tail, float limit) {
    pdl_wait();
    const size_t m = blockIdx.x;
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= I + tail) return;
    float y;
    if (i < I) {
        const float g = gate_up[m * 2 * I + i] + (bias ? bias[i] : 0.0f);
        const float u = gate_up[m * 2 * I + I + i] + (bias ? bias[I + i] : 0.0f);
        y = CLAMP ? clamped_gate(g, u, limit) : activate<ACT>(g) * u;
    } else {
        y = i < I + ones ? 1.0f : 0.0f;
    }
    out[m * ld + i] = from_float<TO>(y);
}

// four elements a thread (16-byte loads), sizes and places that are multiples of four
template <typename TO, int ACT, bool CLAMP>
__global__ void __launch_bounds__(256)
gated_cols_vec4_kernel(const float* gate_up, const float* __restrict__ bias, TO* out, int I, int ld, int ones, int tail, float limit) {
    pdl_wait();
    const size_t m = blockIdx.x;
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (i >= I + tail) return;
    float y[4];
    if (i < I) {
        float4 g = *reinterpret_cast<const float4*>(gate_up + m * 2 * I + i);
        float4 u = *reinterpret_cast<const float4*>(gate_up + m * 2 * I + I + i);
        if (bias) {
            const float4 bg = *reinterpret_cast<const float4*>(bias + i), bu = *reinterpret_cast<const float4*>(bias + I + i);
            g.x += bg.x; g.y += bg.y; g.z += bg.z; g.w += bg.w;
            u.x += bu.x; u.y += bu.y; u.z += bu.z; u.w += bu.w;
        }
        const float gs[4] = {g.x, g.y, g.z, g.w}, us[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = CLAMP ? clamped_gate(gs[j], us[j], limit) : activate<ACT>(gs[j]) * us[j];
    } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = i + j < I + ones ? 1.0f : 0.0f;
    }
    TO* dst = out + m * ld + i;
#pragma unroll
    for (int j = 0; j < 4; ++j) dst[j] = from_float<TO>(y[j]);
}

template <typename TO, int ACT, bool CLAMP>
static int launch_gated_cols(const float* gate_up, const float* bias, TO* out, int M, int I, int ld, int ones, int tail,
                             float limit, cudaStream_t stream) {
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(gate_up) | reinterpret_cast<uintptr_t>(bias);
    if (I % 4 == 0 && tail % 4 == 0 && (ptrs & 15) == 0) {
        auto kern = gated_cols_vec4_kernel<TO, ACT, CLAMP>;
        SHARPI_LAUNCH_PDL(kern, dim3(M, ((I + tail) / 4 + 255) / 256), 256, 0, stream, gate_up, bias, out, I, ld, ones, tail, limit);
    } else {
        auto kern = gated_cols_kernel<TO, ACT, CLAMP>;
        SHARPI_LAUNCH_PDL(kern, dim3(M, (I + tail + 255) / 256), 256, 0, stream, gate_up, bias, out, I, ld, ones, tail, limit);
    }
    return SHARPI_OK;
}

SHARPI_API int sharpi_gated_cols(const float* gate_up, const float* bias, void* out, int out_dtype, int M, int I, int ld,
                                 int ones, int zeros, int act, float limit, cudaStream_t stream) {
    if (M <= 0 || I <= 0) return SHARPI_OK;
    const int tail = ones + zeros;
    if (ones < 0 || zeros < 0 || ld < I + tail || (I + tail + 255) / 256 > 65535 || !(limit >= 0.0f)) return SHARPI_BAD_ARGUMENT;
#define COLS_CASE(TO)                                                                                                       \
    do {                                                                                                                    \
        TO* o = (TO*)out;                                                                                                   \
        if (limit > 0.0f) return launch_gated_cols<TO, ACT_SILU, true>(gate_up, bias, o, M, I, ld, ones, tail, limit, stream); \
        if (act == ACT_RELU2) return launch_gated_cols<TO, ACT_RELU2, false>(gate_up, bias, o, M, I, ld, ones, tail, 0.0f, stream); \
        if (act == ACT_GELU_TANH) return launch_gated_cols<TO, ACT_GELU_TANH, false>(gate_up, bias, o, M, I, ld, ones, tail, 0.0f, stream); \
        if (act == ACT_SILU) return launch_gated_cols<TO, ACT_SILU, false>(gate_up, bias, o, M, I, ld, ones, tail, 0.0f, stream); \
        return SHARPI_BAD_ARGUMENT;                                                                                         \
    } while (0)
    if (out_dtype == SHARPI_F32) COLS_CASE(float);
    if (out_dtype == SHARPI_BF16) COLS_CASE(bf16);
#undef COLS_CASE
    return SHARPI_BAD_ARGUMENT;
}

// out[t, h dv + i] = o[t, h, i] * sigmoid(g[t, h]) * scale for i < dv: a gate of one number per head on attention outputs
// whose heads are D >= dv elements apart, laid side by side in a column range of a wider matrix.
template <typename TO>
__global__ void __launch_bounds__(256)
gate_heads_kernel(const TO* o, const float* g, int ld_g, TO* out, int ld_out, int heads, int D, int dv, float scale) {
    pdl_wait();
    const size_t t = blockIdx.x;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < heads * dv; i += gridDim.y * blockDim.x) {
        const int h = i / dv, e = i - h * dv;
        const float f = scale / (1.0f + expf(-g[t * ld_g + h]));
        out[t * ld_out + i] = from_float<TO>(to_float(o[(t * heads + h) * D + e]) * f);
    }
}

// the same eight elements a thread (16-byte accesses for 16-bit heads), sizes and places that are multiples of eight
template <typename TO>
__global__ void __launch_bounds__(256)
gate_heads_vec8_kernel(const TO* o, const float* g, int ld_g, TO* out, int ld_out, int heads, int D, int dv, float scale,
                       long long n) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const int per = dv / 8;
    const long long th = i / per;
    const int e = (int)(i - th * per) * 8;
    const int t = (int)(th / heads), h = (int)(th - (long long)t * heads);
    const float f = scale / (1.0f + expf(-g[(size_t)t * ld_g + h]));
    struct alignas(16) Eight { TO v[8]; };
    Eight x = *reinterpret_cast<const Eight*>(o + (size_t)th * D + e);
#pragma unroll
    for (int j = 0; j < 8; ++j) x.v[j] = from_float<TO>(to_float(x.v[j]) * f);
    *reinterpret_cast<Eight*>(out + (size_t)t * ld_out + (size_t)h * dv + e) = x;
}

SHARPI_API int sharpi_gate_heads(const void* o, const float* g, int ld_g, void* out, int ld_out, int dtype, int T, int heads,
                                 int D, int dv, float scale, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (heads <= 0 || dv <= 0 || D < dv || ld_g < heads || ld_out < heads * dv) return SHARPI_BAD_ARGUMENT;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(out);
    if (D % 8 == 0 && dv % 8 == 0 && ld_out % 8 == 0 && (ptrs & 15) == 0) {
        const long long n = (long long)T * heads * (dv / 8);
        const unsigned blocks = (unsigned)((n + 255) / 256);
        if (dtype == SHARPI_F32)
            SHARPI_LAUNCH_PDL(gate_heads_vec8_kernel<float>, blocks, 256, 0, stream, (const float*)o, g, ld_g, (float*)out, ld_out, heads, D, dv, scale, n);
        else if (dtype == SHARPI_BF16)
            SHARPI_LAUNCH_PDL(gate_heads_vec8_kernel<bf16>, blocks, 256, 0, stream, (const bf16*)o, g, ld_g, (bf16*)out, ld_out, heads, D, dv, scale, n);
        else
            return SHARPI_BAD_ARGUMENT;
        return SHARPI_OK;
    }
    int by = (heads * dv + 1023) / 1024;
    const dim3 grid(T, by > 64 ? 64 : by);
    if (dtype == SHARPI_F32)
        SHARPI_LAUNCH_PDL(gate_heads_kernel<float>, grid, 256, 0, stream, (const float*)o, g, ld_g, (float*)out, ld_out, heads, D, dv, scale);
    else if (dtype == SHARPI_BF16)
        SHARPI_LAUNCH_PDL(gate_heads_kernel<bf16>, grid, 256, 0, stream, (const bf16*)o, g, ld_g, (bf16*)out, ld_out, heads, D, dv, scale);
    else
        return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

// y = cap * tanh(y / cap), in place (float32): a cap on the logits
__global__ void softcap_kernel(float* y, float cap, long long n) {
    pdl_wait();
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) y[i] = cap * tanhf(y[i] / cap);
}

SHARPI_API int sharpi_softcap(float* y, float cap, long long n, cudaStream_t stream) {
    if (n <= 0) return SHARPI_OK;
    if (!(cap > 0.0f)) return SHARPI_BAD_ARGUMENT;
    SHARPI_LAUNCH_PDL(softcap_kernel, (unsigned)((n + 255) / 256), 256, 0, stream, y, cap, n);
    return SHARPI_OK;
}
