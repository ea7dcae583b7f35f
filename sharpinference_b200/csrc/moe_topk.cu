// Routing of a mixture of experts in which every row uses k experts.
//
//   router_topk   z = h Wr^T (float32), s = sigmoid(z); the k experts with the largest s + correction (the lowest
//                 index among equals) are chosen; each weight is scale * s (without the correction), divided by the
//                 sum of the chosen s first when `renormalize`.  A row's logits are one fixed sequence of additions
//                 whatever else the step holds.  `bias` [E] (optional) is added to the logits.  `scoring` = 1
//                 (softmax over the chosen): the k experts with the largest logits z are chosen and their weights are
//                 scale * exp(z_i - max) / sum over the chosen of exp(z_j - max): the other experts' logits do not
//                 enter.
//                 `scoring` = 2 (softmax over all): s = softmax(z) over every expert; the choice score is s + correction;
//                 with `n_groups` > 1 the experts form equal groups of neighbours, a group's score is its largest choice
//                 score, and only experts of the `keep` best groups may be chosen (the lowest index among equal groups).
//                 Weights as for the sigmoid (scale * s / (sum + 1e-20) when `renormalize`).
//                 `scoring` = 3: s = sigmoid(z) with the groups of 2.  `group_top` = 2: a group's score is the sum of its two
//                 largest choice scores (of its only one in groups of one) in place of the largest.
//                 `gate_w` [H] (optional): one more row, gate_out[t] = sigmoid(gate_w . h_t), the gate of a shared expert.
//   pair_tokens   after the (row, choice) pairs have been sorted by expert: the row each sorted pair belongs to.
//   combine       out[t] = add[t] + sum over the row's k pairs of y[pair], in the order of the choices.
//   combine_full  out[t] = add[t] + gate[t] shared[t] + sum over the row's k pairs of (y[pair], or weight[pair] h[t] for a
//                 choice beyond the experts that have weights: an identity expert), in the order of the choices.
//
// The reference routes on the host, one row at a time (src/SharpInference.Engine/ForwardPass.cs:2021-2098); here
// routing stays on the device so that a step's rows can be sorted by expert for grouped products.
#include "common.cuh"

constexpr int TOPK_MANY_ROWS = 512;   // steps of more rows than this put four rows in a CTA (a router row is fetched
                                      // once for all of them); smaller steps one, for more CTAs

// One CTA per TOPK_ROWS rows (1 or 4): warp w forms the logits of experts w, w + warps, ... for each of the CTA's rows: lane
// l adds the elements 128 i + 4 l + u in ascending i into chain u = 0 .. 3, the chains and then the lanes are added in a
// fixed order, so a row's logits depend on neither its neighbours nor the number of warps.  Then warp r picks the k best of
// row r.
template <int TOPK_ROWS>
__global__ void __launch_bounds__(1024)
router_topk_kernel(const float* __restrict__ h, const float* __restrict__ wr, const float* __restrict__ correction,
                   int T, int H, int E, int k, float scale, int renormalize, int* __restrict__ expert_id,
                   float* __restrict__ weight, float* __restrict__ scores_out, int stage_rows,
                   const float* __restrict__ bias, int scoring, int n_groups, int keep, int group_top, const float* __restrict__ gate_w,
                   float* __restrict__ gate_out, int vec) {
    extern __shared__ __align__(16) float smem[];         // the rows [ROWS][H] if they fit; per row s [E], choice [E]; group scores
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int t0 = blockIdx.x * TOPK_ROWS;
    const int rows = min(TOPK_ROWS, T - t0);
    float* const score_s = smem + (stage_rows ? ((size_t)TOPK_ROWS * H + 3) / 4 * 4 : 0);
    const float* row[TOPK_ROWS];
#pragma unroll
    for (int r = 0; r < TOPK_ROWS; ++r) row[r] = h + (size_t)(t0 + min(r, rows - 1)) * H;
    if (stage_rows) {                                     // the rows are read from memory once, by all warps together
        if (vec) {
            const float4* src = reinterpret_cast<const float4*>(h + (size_t)t0 * H);
            for (int i = threadIdx.x; i < rows * H / 4; i += blockDim.x) reinterpret_cast<float4*>(smem)[i] = src[i];
        } else {
            for (int i = threadIdx.x; i < rows * H; i += blockDim.x) smem[i] = h[(size_t)t0 * H + i];
        }
        __syncthreads();
#pragma unroll
        for (int r = 0; r < TOPK_ROWS; ++r) row[r] = smem + (size_t)min(r, rows - 1) * H;
    }
    for (int e = warp; e < E + (gate_w ? 1 : 0); e += warps) {
        const float* w = e < E ? wr + (size_t)e * H : gate_w;
        float acc[TOPK_ROWS][4];
#pragma unroll
        for (int r = 0; r < TOPK_ROWS; ++r)
#pragma unroll
            for (int u = 0; u < 4; ++u) acc[r][u] = 0.0f;
        if (vec) {
#pragma unroll 4
            for (int i = 4 * lane; i < H; i += 128) {
                const float4 wv = *reinterpret_cast<const float4*>(w + i);
#pragma unroll
                for (int r = 0; r < TOPK_ROWS; ++r) {
                    const float4 x = *reinterpret_cast<const float4*>(row[r] + i);
                    acc[r][0] = fmaf(x.x, wv.x, acc[r][0]);
                    acc[r][1] = fmaf(x.y, wv.y, acc[r][1]);
                    acc[r][2] = fmaf(x.z, wv.z, acc[r][2]);
                    acc[r][3] = fmaf(x.w, wv.w, acc[r][3]);
                }
            }
        } else {
            for (int i = 4 * lane; i < H; i += 128) {
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                    if (i + u < H) {
                        const float wv = w[i + u];
#pragma unroll
                        for (int r = 0; r < TOPK_ROWS; ++r) acc[r][u] = fmaf(row[r][i + u], wv, acc[r][u]);
                    }
                }
            }
        }
#pragma unroll
        for (int r = 0; r < TOPK_ROWS; ++r) {
            const float z = warp_sum((acc[r][0] + acc[r][1]) + (acc[r][2] + acc[r][3])) + (bias && e < E ? bias[e] : 0.0f);
            if (lane == 0 && r < rows && e == E) gate_out[t0 + r] = 1.0f / (1.0f + expf(-z));
            if (lane == 0 && r < rows && e < E) {
                const float s = scoring == 1 || scoring == 2 ? z : 1.0f / (1.0f + expf(-z));
                score_s[(size_t)r * 2 * E + e] = s;
                score_s[(size_t)r * 2 * E + E + e] = correction ? s + correction[e] : s;
                if (scores_out && scoring != 2) scores_out[(size_t)(t0 + r) * E + e] = s;
            }
        }
    }
    __syncthreads();
    if (warp >= rows) return;
    const int t = t0 + warp;
    float* s_s = score_s + (size_t)warp * 2 * E;
    float* c_s = s_s + E;
    if (scoring == 2) {
        float m = -INFINITY, sum = 0.0f;
        for (int e = lane; e < E; e += 32) m = fmaxf(m, s_s[e]);
        m = warp_max(m);
        for (int e = lane; e < E; e += 32) {
            const float x = expf(s_s[e] - m);
            s_s[e] = x;
            sum += x;
        }
        sum = warp_sum(sum);
        for (int e = lane; e < E; e += 32) {
            const float s = s_s[e] / sum;
            s_s[e] = s;
            c_s[e] = correction ? s + correction[e] : s;
            if (scores_out) scores_out[(size_t)t * E + e] = s;
        }
        __syncwarp();
    }
    if (scoring >= 2) {
        if (n_groups > 1 && keep < n_groups) {
            float* g_s = score_s + (size_t)TOPK_ROWS * 2 * E + (size_t)warp * n_groups;       // the groups' scores
            const int per = E / n_groups;
            for (int g = lane; g < n_groups; g += 32) {
                float best = -INFINITY, second = -INFINITY;
                for (int e = g * per; e < (g + 1) * per; ++e) {
                    const float c = c_s[e];
                    second = fmaxf(second, fminf(best, c));
                    best = fmaxf(best, c);
                }
                g_s[g] = group_top == 2 && per > 1 ? best + second : best;
            }
            __syncwarp();
            // a group stays when fewer than `keep` groups are ahead of it (larger score, or equal and lower index)
            for (int g = lane; g < n_groups; g += 32) {
                int ahead = 0;
                for (int o = 0; o < n_groups; ++o) ahead += g_s[o] > g_s[g] || (g_s[o] == g_s[g] && o < g);
                if (ahead >= keep)
                    for (int e = g * per; e < (g + 1) * per; ++e) c_s[e] = -INFINITY;
            }
            __syncwarp();
        }
    }
    float total = 0.0f, top = 0.0f;
    int mine = 0;                                          // lane j keeps the j-th choice
    for (int j = 0; j < k; ++j) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float c = c_s[e];
            if (c > best) { best = c; at = e; }          // ascending e: the first of equals stays
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (ob > best || (ob == best && oa < at)) { best = ob; at = oa; }
        }
        if (at >= E) at = j < E ? j : 0;                   // every score was NaN: any expert, but a valid one
        if (lane == 0) {
            expert_id[(size_t)t * k + j] = at;
            c_s[at] = -INFINITY;
        }
        if (lane == j) mine = at;
        if (scoring == 1) {                                // the first choice has the largest logit
            if (j == 0) top = s_s[at];
            total += expf(s_s[at] - top);
        } else {
            total += s_s[at];
        }
        __syncwarp();
    }
    if (scoring == 1) {
        if (lane < k) weight[(size_t)t * k + lane] = expf(s_s[mine] - top) * (scale / total);
        return;
    }
    const float factor = renormalize ? scale / (scoring == 2 ? total + 1e-20f : total) : scale;
    if (lane < k) weight[(size_t)t * k + lane] = s_s[mine] * factor;      // k <= 32 is checked by the host
}

static int router_topk_impl(const float* h, const float* wr, const float* correction, int T, int H, int E, int k,
                            float scale, int renormalize, int* expert_id, float* weight, float* scores_out,
                            const float* bias, int scoring, int n_groups, int keep, int group_top, const float* gate_w,
                            float* gate_out, cudaStream_t stream) {
    if (T <= 0) return SHARPI_OK;
    if (H <= 0 || E <= 0 || k <= 0 || k > E || k > 32) return SHARPI_BAD_ARGUMENT;
    const int per_cta = T > TOPK_MANY_ROWS ? 4 : 1;
    size_t smem = (size_t)per_cta * (2 * E + n_groups) * sizeof(float);
    if (smem > 48 * 1024) return SHARPI_BAD_ARGUMENT;
    const size_t copies = ((size_t)per_cta * H + 3) / 4 * 4 * sizeof(float);
    const int stage_rows = smem + copies <= 48 * 1024;
    if (stage_rows) smem += copies;
    const int vec = H % 4 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(wr) |
                                    reinterpret_cast<uintptr_t>(gate_w)) & 15) == 0;
    // a warp an expert where the step is small (the wait is what counts), eight where its CTAs fill the GPU
    const int experts = E + (gate_w ? 1 : 0);
    const int warps = T > TOPK_MANY_ROWS ? 8 : experts < 8 ? 8 : experts > 32 ? 32 : experts;
    if (per_cta == 4)
        router_topk_kernel<4><<<(T + 3) / 4, warps * 32, smem, stream>>>(
            h, wr, correction, T, H, E, k, scale, renormalize, expert_id, weight, scores_out, stage_rows, bias, scoring,
            n_groups, keep, group_top, gate_w, gate_out, vec);
    else
        router_topk_kernel<1><<<T, warps * 32, smem, stream>>>(
            h, wr, correction, T, H, E, k, scale, renormalize, expert_id, weight, scores_out, stage_rows, bias, scoring,
            n_groups, keep, group_top, gate_w, gate_out, vec);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

SHARPI_API int sharpi_router_topk(const float* h, const float* wr, const float* correction, int T, int H, int E, int k,
                                  float scale, int renormalize, int* expert_id, float* weight, float* scores_out,
                                  const float* bias, int scoring, cudaStream_t stream) {
    if (scoring != 0 && scoring != 1) return SHARPI_BAD_ARGUMENT;
    return router_topk_impl(h, wr, correction, T, H, E, k, scale, renormalize, expert_id, weight, scores_out, bias, scoring,
                            0, 0, 1, nullptr, nullptr, stream);
}

// The softmax over all experts (`scoring` 2) or the sigmoid of each (3), with groups (n_groups >= 1, keep of them; k must fit
// the kept groups' experts) whose score is the sum of their `group_top` largest choice scores, and the gate row
SHARPI_API int sharpi_router_groups(const float* h, const float* wr, const float* correction, int T, int H, int E, int k,
                                    float scale, int renormalize, int n_groups, int keep, int scoring, int group_top,
                                    const float* gate_w, float* gate_out, int* expert_id, float* weight, float* scores_out,
                                    cudaStream_t stream) {
    if (n_groups < 1 || E % n_groups != 0 || keep < 1 || keep > n_groups || k > keep * (E / n_groups) ||
        (scoring != 2 && scoring != 3) || (group_top != 1 && group_top != 2) || (gate_w == nullptr) != (gate_out == nullptr))
        return SHARPI_BAD_ARGUMENT;
    return router_topk_impl(h, wr, correction, T, H, E, k, scale, renormalize, expert_id, weight, scores_out, nullptr,
                            scoring, n_groups, keep, group_top, gate_w, gate_out, stream);
}

__global__ void pair_tokens_kernel(const int* __restrict__ sorted_pairs, int P, int k, int* __restrict__ tokens) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < P) tokens[i] = sorted_pairs[i] / k;
}

SHARPI_API int sharpi_moe_pair_tokens(const int* sorted_pairs, int P, int k, int* tokens, cudaStream_t stream) {
    if (P <= 0) return SHARPI_OK;
    if (k <= 0) return SHARPI_BAD_ARGUMENT;
    pair_tokens_kernel<<<(P + 255) / 256, 256, 0, stream>>>(sorted_pairs, P, k, tokens);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

__global__ void moe_combine_kernel(const float* __restrict__ y, const float* add, float* out,      // out may be add
                                   int k, int H) {
    const int t = blockIdx.x;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < H; i += gridDim.y * blockDim.x) {
        float acc = add ? add[(size_t)t * H + i] : 0.0f;
        for (int j = 0; j < k; ++j) acc += y[((size_t)t * k + j) * H + i];
        out[(size_t)t * H + i] = acc;
    }
}

__global__ void moe_combine_vec4_kernel(const float4* __restrict__ y, const float4* add, float4* out, int k, int H4) {
    const int t = blockIdx.x;
    for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < H4; i += gridDim.y * blockDim.x) {
        float4 acc = add ? add[(size_t)t * H4 + i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        for (int j = 0; j < k; ++j) {
            const float4 v = y[((size_t)t * k + j) * H4 + i];
            acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
        }
        out[(size_t)t * H4 + i] = acc;
    }
}

SHARPI_API int sharpi_moe_combine(const float* y, const float* add, float* out, int T, int k, int H,
                                  cudaStream_t stream) {
    if (T <= 0 || H <= 0) return SHARPI_OK;
    if (k <= 0) return SHARPI_BAD_ARGUMENT;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(add) | reinterpret_cast<uintptr_t>(out);
    if (H % 4 == 0 && (ptrs & 15) == 0) {               // same additions in the same order, four columns a thread
        int by4 = (H / 4 + 255) / 256;
        if (by4 > 64) by4 = 64;
        moe_combine_vec4_kernel<<<dim3(T, by4), 256, 0, stream>>>((const float4*)y, (const float4*)add, (float4*)out, k, H / 4);
        SHARPI_CHECK_LAUNCH();
        return SHARPI_OK;
    }
    int by = (H + 255) / 256;
    if (by > 64) by = 64;
    moe_combine_kernel<<<dim3(T, by), 256, 0, stream>>>(y, add, out, k, H);
    SHARPI_CHECK_LAUNCH();
    return SHARPI_OK;
}

template <int VEC>
__global__ void __launch_bounds__(256)
moe_combine_full_kernel(const float* y, const int* expert, const float* weight, const float* h, const float* shared,
                        const float* gate, const float* add, float* out, int E, int k, int H) {
    pdl_wait();
    const int t = blockIdx.x;
    const float gt = shared ? (gate ? gate[t] : 1.0f) : 0.0f;
    for (int i = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; i < H; i += gridDim.y * blockDim.x * VEC) {
        float acc[VEC];
        const size_t at = (size_t)t * H + i;
        auto read = [&](const float* p, float* v) {
            if (VEC == 4) {
                const float4 x = *reinterpret_cast<const float4*>(p);
                v[0] = x.x; v[1 % VEC] = x.y; v[2 % VEC] = x.z; v[3 % VEC] = x.w;
            } else {
                v[0] = *p;
            }
        };
        float v[VEC], x[VEC];
        read(h + at, x);
#pragma unroll
        for (int u = 0; u < VEC; ++u) acc[u] = 0.0f;
        if (add) read(add + at, acc);
        if (shared) {
            read(shared + at, v);
#pragma unroll
            for (int u = 0; u < VEC; ++u) acc[u] = fmaf(gt, v[u], acc[u]);
        }
        for (int j = 0; j < k; ++j) {
            const size_t pair = (size_t)t * k + j;
            if (expert[pair] < E) {
                read(y + pair * H + i, v);
#pragma unroll
                for (int u = 0; u < VEC; ++u) acc[u] += v[u];
            } else {
                const float w = weight[pair];
#pragma unroll
                for (int u = 0; u < VEC; ++u) acc[u] = fmaf(w, x[u], acc[u]);
            }
        }
        if (VEC == 4) *reinterpret_cast<float4*>(out + at) = make_float4(acc[0], acc[1 % VEC], acc[2 % VEC], acc[3 % VEC]);
        else out[at] = acc[0];
    }
}

// `shared`, `gate` and `add` may be null; `out` may be `add`.  Choices >= E are identity experts.
SHARPI_API int sharpi_moe_combine_full(const float* y, const int* expert, const float* weight, const float* h,
                                       const float* shared, const float* gate, const float* add, float* out, int T, int E,
                                       int k, int H, cudaStream_t stream) {
    if (T <= 0 || H <= 0) return SHARPI_OK;
    if (k <= 0 || E < 0) return SHARPI_BAD_ARGUMENT;
    const uintptr_t ptrs = reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(shared) |
                           reinterpret_cast<uintptr_t>(add) | reinterpret_cast<uintptr_t>(out);
    const bool vec = H % 4 == 0 && (ptrs & 15) == 0;
    int by = (H / (vec ? 4 : 1) + 255) / 256;
    if (by > 64) by = 64;
    if (by < 1) by = 1;
    if (vec) SHARPI_LAUNCH_PDL(moe_combine_full_kernel<4>, dim3(T, by), 256, 0, stream, y, expert, weight, h, shared, gate, add, out, E, k, H);
    else SHARPI_LAUNCH_PDL(moe_combine_full_kernel<1>, dim3(T, by), 256, 0, stream, y, expert, weight, h, shared, gate, add, out, E, k, H);
    return SHARPI_OK;
}
