// Latent attention around the paged attention kernels: keys and values are two readings of one cached latent.
//
// Per token the cache holds one row of D elements for all heads: [c (rank) | k_rot (rot) | zeros], c the
// RMS-normed latent and k_rot the rotated key part that every head shares.  A head's score is
// q_plain . (W_uk c) + q_rot . k_rot = (W_uk^T q_plain) . c + q_rot . k_rot, so a query row of a head is
// [W_uk^T q_plain | q_rot | zeros] and the attention kernels see one key/value head of size D whose value is the
// key row itself; of a head's output the first `rank` elements are sum_j p_j c_j, which W_uv then expands.
//
//   sharpi_latent_down_post  one block a token over the fused down projection [q latent | c | k_rot]:
//                            RMS norm with a weight of the q latent (-> activation dtype) and of c, rotation of
//                            k_rot by the token's position (pairs (2i, 2i + 1) of its first `rot_dims` elements),
//                            and the store of [c | k_rot | 0] into the token's place in the pages (and of
//                            [c | 0] into the value plane when a page has one).
//   sharpi_head_major        columns [col0, col0 + n) of every head of src [T, heads, stride] (float32 or the
//                            activation dtype) as dst [heads, T, n] in the activation dtype: the operand of a
//                            per-head (grouped) product.
//   sharpi_head_minor        the way back: src float32 [heads, T, n] into columns [col0, col0 + n) of
//                            dst [T, heads, stride] in the activation dtype.
//   sharpi_latent_q_join     the query rows: dst[t, h] = [qa[h, t, :rank] | rotate(q[t, h, dim:dim + rot]) | 0].
//
// `ld` / `ldq`: the distance between two rows of the source when it is a column range of a wider product; `rot_amp`:
// a factor on the rotation's cosines and sines (frequency scalings that also stretch the amplitude); `gate` of
// head_minor: [T, gate_ld] float32 logits, head h of row t is multiplied by sigmoid(gate[t, h]), or element c of it by
// sigmoid(gate[t, h n + c]) (`gate_elem`).  Without `write_kv` (a layer that reads another one's latents) latent_down_post
// norms the query latent alone and the columns behind it may be absent.
//
// Norm sums, angles, sines and cosines are float32; a row's numbers depend on the row alone.
#include "common.cuh"

#include <initializer_list>

constexpr int LAT_THREADS = 128;

template <typename TO>
__global__ void __launch_bounds__(LAT_THREADS)
latent_down_post_kernel(const float* down, int ld, int q_rank, int rank, int rot, int rot_dims,
                        const float* __restrict__ wq, const float* __restrict__ wc, float eps,
                        const int* positions, const int* row_req, const int* block_table, int max_blocks,
                        int page_size, const float* __restrict__ inv_freq, TO* cq_out, TO* kv_base, int kv_planes,
                        int D, int write_kv, float rot_amp) {
    __shared__ float scratch[32];
    pdl_wait();
    const int t = blockIdx.x;
    const float* row = down + (size_t)t * ld;
    float ssq = 0.0f, ssc = 0.0f;
    for (int i = threadIdx.x; i < q_rank; i += LAT_THREADS) ssq += row[i] * row[i];
    if (write_kv)
        for (int i = threadIdx.x; i < rank; i += LAT_THREADS) ssc += row[q_rank + i] * row[q_rank + i];
    ssq = block_sum(ssq, scratch);
    if (write_kv) ssc = block_sum(ssc, scratch);
    if (q_rank > 0) {
        const float sq = 1.0f / sqrtf(ssq / (float)q_rank + eps);
        for (int i = threadIdx.x; i < q_rank; i += LAT_THREADS)
            cq_out[(size_t)t * q_rank + i] = from_float<TO>(row[i] * sq * wq[i]);
    }
    if (!write_kv) return;
    const int pos = positions[t];
    const int page = block_table[(size_t)row_req[t] * max_blocks + pos / page_size];
    if (page < 0) return;   // the host checks before the launch that every written position has a page
    const size_t plane = (size_t)page_size * D;
    TO* krow = kv_base + (size_t)page * kv_planes * plane + (size_t)(pos % page_size) * D;
    TO* vrow = kv_planes == 2 ? krow + plane : nullptr;
    const float sc = 1.0f / sqrtf(ssc / (float)rank + eps);
    const float* kr = row + q_rank + rank;
    for (int i = threadIdx.x; i < D; i += LAT_THREADS) {
        float k = 0.0f, v = 0.0f;
        if (i < rank) {
            k = v = row[q_rank + i] * sc * wc[i];
        } else if (i < rank + rot) {
            const int j = i - rank;
            k = kr[j];
            if (j < rot_dims && inv_freq) {
                float sn, cs;
                sincosf((float)pos * inv_freq[j >> 1], &sn, &cs);
                sn *= rot_amp;
                cs *= rot_amp;
                k = (j & 1) ? kr[j] * cs + kr[j - 1] * sn : kr[j] * cs - kr[j + 1] * sn;
            }
        }
        krow[i] = from_float<TO>(k);
        if (vrow) vrow[i] = from_float<TO>(v);
    }
}

SHARPI_API int sharpi_latent_down_post(const float* down, int ld, int q_rank, int rank, int rot, int rot_dims,
                                       const float* wq, const float* wc, float eps, const int* positions,
                                       const int* row_req, const int* block_table, int max_blocks, int page_size,
                                       const float* inv_freq, void* cq_out, void* kv_base, int kv_planes, int D,
                                       int write_kv, int out_dtype, int T, float rot_amp, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (q_rank < 0 || rank <= 0 || rot < 0 || rot_dims < 0 || rot_dims > rot || (rot_dims & 1) ||
        q_rank + (write_kv ? rank + rot : 0) > ld || rank + rot > D || (kv_planes != 1 && kv_planes != 2) ||
        page_size <= 0 || max_blocks <= 0 || (q_rank > 0 && !wq) || (write_kv && !wc))
        return SHARPI_BAD_ARGUMENT;
    if (out_dtype == SHARPI_F32)
        SHARPI_LAUNCH_PDL(latent_down_post_kernel<float>, T, LAT_THREADS, 0, stream, down, ld, q_rank, rank, rot,
                          rot_dims, wq, wc, eps, positions, row_req, block_table, max_blocks, page_size, inv_freq,
                          (float*)cq_out, (float*)kv_base, kv_planes, D, write_kv, rot_amp);
    else if (out_dtype == SHARPI_BF16)
        SHARPI_LAUNCH_PDL(latent_down_post_kernel<bf16>, T, LAT_THREADS, 0, stream, down, ld, q_rank, rank, rot,
                          rot_dims, wq, wc, eps, positions, row_req, block_table, max_blocks, page_size, inv_freq,
                          (bf16*)cq_out, (bf16*)kv_base, kv_planes, D, write_kv, rot_amp);
    else
        return SHARPI_BAD_ARGUMENT;
    return SHARPI_OK;
}

// Four neighbouring elements a thread where sizes, strides and addresses allow it.
template <int VEC> __device__ __forceinline__ void load_vec(const float* p, float* v) {
    if (VEC == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x; v[1 % VEC] = x.y; v[2 % VEC] = x.z; v[3 % VEC] = x.w;
    } else {
        v[0] = *p;
    }
}
template <int VEC> __device__ __forceinline__ void load_vec(const bf16* p, float* v) {
    if (VEC == 4) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        v[0] = __uint_as_float(x.x << 16); v[1 % VEC] = __uint_as_float(x.x & 0xffff0000u);
        v[2 % VEC] = __uint_as_float(x.y << 16); v[3 % VEC] = __uint_as_float(x.y & 0xffff0000u);
    } else {
        v[0] = to_float(*p);
    }
}
template <int VEC> __device__ __forceinline__ void store_vec(float* p, const float* v) {
    if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]);
    else *p = v[0];
}
template <int VEC> __device__ __forceinline__ void store_vec(bf16* p, const float* v) {
    if (VEC == 4) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % VEC]), b = __floats2bfloat162_rn(v[2 % VEC], v[3 % VEC]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
    } else {
        *p = from_float<bf16>(v[0]);
    }
}
static inline bool fours(std::initializer_list<long long> sizes, std::initializer_list<const void*> pointers) {
    for (long long n : sizes)
        if (n % 4 != 0) return false;
    for (const void* p : pointers)
        if (reinterpret_cast<uintptr_t>(p) & 15) return false;
    return true;
}

template <typename TS, typename TO, int VEC>
__global__ void __launch_bounds__(256)
head_major_kernel(const TS* src, int T, int heads, int stride, int col0, int n, TO* dst, int ld) {
    pdl_wait();
    const int t = blockIdx.x, i = blockIdx.y * blockDim.x + threadIdx.x, per = n / VEC;
    const int h = i / per, c = i % per * VEC;
    if (h >= heads) return;
    float v[VEC];
    load_vec<VEC>(src + (size_t)t * ld + (size_t)h * stride + col0 + c, v);
    store_vec<VEC>(dst + ((size_t)h * T + t) * n + c, v);
}

SHARPI_API int sharpi_head_major(const void* src, int src_dtype, int T, int heads, int stride, int col0, int n,
                                 void* dst, int dst_dtype, int ld, cudaStream_t stream) {
    if (T <= 0 || n <= 0) return SHARPI_OK;
    if (ld <= 0) ld = heads * stride;          // rows lie end to end
    if (heads <= 0 || col0 < 0 || col0 + n > stride || ld < heads * stride) return SHARPI_BAD_ARGUMENT;
    const bool vec = fours({n, stride, col0, ld}, {src, dst});
    const dim3 grid(T, ((long long)heads * (n / (vec ? 4 : 1)) + 255) / 256);
#define MAJOR_CASE(TS, TO)                                                                                                       \
    do {                                                                                                                         \
        if (vec) SHARPI_LAUNCH_PDL((head_major_kernel<TS, TO, 4>), grid, 256, 0, stream, (const TS*)src, T, heads, stride, col0, n, (TO*)dst, ld); \
        else SHARPI_LAUNCH_PDL((head_major_kernel<TS, TO, 1>), grid, 256, 0, stream, (const TS*)src, T, heads, stride, col0, n, (TO*)dst, ld); \
    } while (0)
    if (src_dtype == SHARPI_F32 && dst_dtype == SHARPI_F32) MAJOR_CASE(float, float);
    else if (src_dtype == SHARPI_F32 && dst_dtype == SHARPI_BF16) MAJOR_CASE(float, bf16);
    else if (src_dtype == SHARPI_BF16 && dst_dtype == SHARPI_BF16) MAJOR_CASE(bf16, bf16);
    else
        return SHARPI_BAD_ARGUMENT;
#undef MAJOR_CASE
    return SHARPI_OK;
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(256)
head_minor_kernel(const float* src, int T, int heads, int stride, int col0, int n, TO* dst, const float* gate,
                  int gate_ld, int gate_elem) {
    pdl_wait();
    const int t = blockIdx.x, i = blockIdx.y * blockDim.x + threadIdx.x, per = n / VEC;
    const int h = i / per, c = i % per * VEC;
    if (h >= heads) return;
    float v[VEC], z[VEC];
    load_vec<VEC>(src + ((size_t)h * T + t) * n + c, v);
    if (gate) {                                                        // times sigmoid(gate logit)
        if (gate_elem) {
            load_vec<VEC>(gate + (size_t)t * gate_ld + h * n + c, z);
#pragma unroll
            for (int u = 0; u < VEC; ++u) v[u] = v[u] / (1.0f + expf(-z[u]));
        } else {
            const float e = expf(-gate[(size_t)t * gate_ld + h]);
#pragma unroll
            for (int u = 0; u < VEC; ++u) v[u] = v[u] / (1.0f + e);
        }
    }
    store_vec<VEC>(dst + ((size_t)t * heads + h) * stride + col0 + c, v);
}

SHARPI_API int sharpi_head_minor(const float* src, int T, int heads, int stride, int col0, int n, void* dst,
                                 int dst_dtype, const float* gate, int gate_ld, int gate_elem, cudaStream_t stream) {
    if (T <= 0 || n <= 0) return SHARPI_OK;
    if (heads <= 0 || col0 < 0 || col0 + n > stride) return SHARPI_BAD_ARGUMENT;
    const bool vec = fours({n, stride, col0, gate && gate_elem ? gate_ld : 0}, {src, dst, gate && gate_elem ? gate : nullptr});
    const dim3 grid(T, ((long long)heads * (n / (vec ? 4 : 1)) + 255) / 256);
#define MINOR_CASE(TO)                                                                                                           \
    do {                                                                                                                         \
        if (vec) SHARPI_LAUNCH_PDL((head_minor_kernel<TO, 4>), grid, 256, 0, stream, src, T, heads, stride, col0, n, (TO*)dst, gate, gate_ld, gate_elem); \
        else SHARPI_LAUNCH_PDL((head_minor_kernel<TO, 1>), grid, 256, 0, stream, src, T, heads, stride, col0, n, (TO*)dst, gate, gate_ld, gate_elem); \
    } while (0)
    if (dst_dtype == SHARPI_F32) MINOR_CASE(float);
    else if (dst_dtype == SHARPI_BF16) MINOR_CASE(bf16);
    else
        return SHARPI_BAD_ARGUMENT;
#undef MINOR_CASE
    return SHARPI_OK;
}

template <typename TO, int VEC>                        // VEC 4: rank, rot and D are multiples of 4
__global__ void __launch_bounds__(256)
latent_q_join_kernel(const float* qa, const float* q, const int* positions, const float* __restrict__ inv_freq, int T,
                     int heads, int dim, int rank, int rot, int rot_dims, int D, TO* dst, int ldq, float rot_amp) {
    pdl_wait();
    const int t = blockIdx.x, i = blockIdx.y * blockDim.x + threadIdx.x, per = D / VEC;
    const int h = i / per, c0 = i % per * VEC;
    if (h >= heads) return;
    float v[VEC];
    if (c0 + VEC <= rank) {
        load_vec<VEC>(qa + ((size_t)h * T + t) * rank + c0, v);
    } else {
#pragma unroll
        for (int u = 0; u < VEC; ++u) {
            const int j = c0 + u - rank;
            v[u] = 0.0f;
            if (j < 0 || j >= rot) continue;
            const float* qr = q + (size_t)t * ldq + (size_t)h * (dim + rot) + dim;
            v[u] = qr[j];
            if (j < rot_dims && inv_freq) {
                float sn, cs;
                sincosf((float)positions[t] * inv_freq[j >> 1], &sn, &cs);
                sn *= rot_amp;
                cs *= rot_amp;
                v[u] = (j & 1) ? qr[j] * cs + qr[j - 1] * sn : qr[j] * cs - qr[j + 1] * sn;
            }
        }
    }
    store_vec<VEC>(dst + ((size_t)t * heads + h) * D + c0, v);
}

SHARPI_API int sharpi_latent_q_join(const float* qa, const float* q, const int* positions, const float* inv_freq,
                                    int T, int heads, int dim, int rank, int rot, int rot_dims, int D, void* dst,
                                    int dst_dtype, int ldq, float rot_amp, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (ldq <= 0) ldq = heads * (dim + rot);   // rows lie end to end
    if (heads <= 0 || dim <= 0 || rank <= 0 || rot < 0 || rot_dims < 0 || rot_dims > rot || (rot_dims & 1) ||
        rank + rot > D)
        return SHARPI_BAD_ARGUMENT;
    const bool vec = fours({rank, rot, D}, {qa, dst});
    const dim3 grid(T, ((long long)heads * (D / (vec ? 4 : 1)) + 255) / 256);
#define JOIN_CASE(TO)                                                                                                            \
    do {                                                                                                                         \
        if (vec) SHARPI_LAUNCH_PDL((latent_q_join_kernel<TO, 4>), grid, 256, 0, stream, qa, q, positions, inv_freq, T, heads, dim, rank, rot, rot_dims, D, (TO*)dst, ldq, rot_amp); \
        else SHARPI_LAUNCH_PDL((latent_q_join_kernel<TO, 1>), grid, 256, 0, stream, qa, q, positions, inv_freq, T, heads, dim, rank, rot, rot_dims, D, (TO*)dst, ldq, rot_amp); \
    } while (0)
    if (dst_dtype == SHARPI_F32) JOIN_CASE(float);
    else if (dst_dtype == SHARPI_BF16) JOIN_CASE(bf16);
    else
        return SHARPI_BAD_ARGUMENT;
#undef JOIN_CASE
    return SHARPI_OK;
}
