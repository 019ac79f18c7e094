// Kernels around retention layers and heads that share their attention weights, beside ops_gated.cu:
//   * the embedding rows under an RMS norm, straight into the float32 stream;
//   * the output of a retention layer: every head over its root mean square, under a silu gate;
//   * talking heads: each head's output as a mixture over the heads' attention weights, under a sigmoid gate;
//   * the weighted sum of two branches, each under an RMS norm of its own.
// Norms, gates and mixtures are float32; T is the compute type of projections and activations.
#include "common.cuh"

namespace {

// silu(z), with the approximate exponential and division for bfloat16 values (their error is far below the rounding)
template <typename T>
__device__ __forceinline__ float silu_of(float z) {
    return sizeof(T) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));
}
__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
}
__device__ __forceinline__ void load4(const bf16* p, float (&v)[4]) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    v[0] = __uint_as_float(t.x << 16); v[1] = __uint_as_float(t.x & 0xffff0000u);
    v[2] = __uint_as_float(t.y << 16); v[3] = __uint_as_float(t.y & 0xffff0000u);
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

}  // namespace

// ---------------------------------------------------------------- embedding rows under a norm
//
// out[t] = e / sqrt(mean(e^2) + eps) * weight with e = scale * table[ids[t]], float32.  A block per token.
template <typename T>
__global__ void __launch_bounds__(256)
embedding_norm_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, const float* __restrict__ weight,
                      float* __restrict__ out, int hidden, int vocab, float scale, float eps, int* err) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[33];
    int id = ids[blockIdx.x];
    if (id < 0 || id >= vocab) {
        if (threadIdx.x == 0) atomicOr(err, SS_ERR_TOKEN_RANGE);
        id = 0;
    }
    const T* row = table + (int64_t)id * hidden;
    float* dst = out + (int64_t)blockIdx.x * hidden;
    if (hidden % 4 == 0 && hidden <= 4 * 4 * 256) {  // the row in registers, all loads of a thread in flight
        float v[4][4], ss = 0.f;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int j = (threadIdx.x + u * blockDim.x) * 4;
            if (j < hidden) load4(row + j, v[u]);
            else v[u][0] = v[u][1] = v[u][2] = v[u][3] = 0.f;
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                v[u][e] *= scale;
                ss = fmaf(v[u][e], v[u][e], ss);
            }
        const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int j = (threadIdx.x + u * blockDim.x) * 4;
            if (j >= hidden) break;
            float w[4];
            load4(weight + j, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] *= v[u][e] * f;
            store4(dst + j, w);
        }
        return;
    }
    float ss = 0.f;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
        const float v = to_float(row[j]) * scale;
        ss = fmaf(v, v, ss);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps);
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) dst[j] = to_float(row[j]) * scale * f * weight[j];
}

extern "C" int ss_embedding_norm(const int32_t* ids, const void* table, const float* weight, float* out, int n_tokens,
                                 int hidden, int vocab, int dtype, float scale, float eps, int* err, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (hidden < 1 || vocab < 1 || !weight) return (int)cudaErrorInvalidValue;
    if (dtype == SS_BF16)
        ss_launch(embedding_norm_kernel<bf16>, dim3(n_tokens), dim3(256), 0, stream, ids, (const bf16*)table, weight, out, hidden, vocab, scale, eps, err);
    else
        ss_launch(embedding_norm_kernel<float>, dim3(n_tokens), dim3(256), 0, stream, ids, (const float*)table, weight, out, hidden, vocab, scale, eps, err);
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- heads over their root mean square, under a silu gate
//
// out[t][h][j] = x[t][h][j] / sqrt(mean_j(x[t][h]^2) + eps) * silu(gate[t][h][j]); x float32 [rows][heads * dim], gate a
// view with rows gate_stride apart.  A warp per head.  VEC: four elements a lane, dim a multiple of 4 up to 256.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* __restrict__ x, const T* __restrict__ gate, int64_t gate_stride, T* __restrict__ out,
                      int64_t pairs, int heads, int dim, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const int64_t p = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (p >= pairs) return;
    const int64_t t = p / heads;
    const float* src = x + p * dim;
    const T* g = gate + t * gate_stride + (p - t * heads) * dim;
    T* dst = out + p * dim;
    if constexpr (VEC) {
        float v[2][4], gv[2][4], ss = 0.f;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int j = (lane + 32 * u) * 4;
#pragma unroll
            for (int e = 0; e < 4; ++e) v[u][e] = 0.f;
            if (j < dim) {
                load4(src + j, v[u]);
                load4(g + j, gv[u]);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) ss = fmaf(v[u][e], v[u][e], ss);
        }
        const float f = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int j = (lane + 32 * u) * 4;
            if (j >= dim) break;
#pragma unroll
            for (int e = 0; e < 4; ++e) v[u][e] *= f * silu_of<T>(gv[u][e]);
            store4(dst + j, v[u]);
        }
    } else {
        float ss = 0.f;
        for (int j = lane; j < dim; j += 32) ss = fmaf(src[j], src[j], ss);
        const float f = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
        for (int j = lane; j < dim; j += 32) dst[j] = from_float<T>(src[j] * f * silu_of<T>(to_float(g[j])));
    }
}

extern "C" int ss_head_norm_gate(const float* x, const void* gate, int64_t gate_stride, void* out, int n_tokens, int heads,
                                 int dim, float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (heads < 1 || dim < 1) return (int)cudaErrorInvalidValue;
    const int64_t pairs = (int64_t)n_tokens * heads;
    const int warps = pairs >= 8 * ss_sm_count() ? 8 : 2;
    const dim3 grid((unsigned)((pairs + warps - 1) / warps)), block(warps * 32);
    const int size = dtype == SS_BF16 ? 2 : 4;
    const bool vec = dim % 4 == 0 && dim <= 256 && gate_stride % 4 == 0 && (((uintptr_t)x | (uintptr_t)out | (uintptr_t)gate) & (4 * size - 1)) == 0 && ((uintptr_t)x & 15) == 0;
#define HN_GO(T, VEC) ss_launch(head_norm_gate_kernel<T, VEC>, grid, block, 0, stream, x, (const T*)gate, gate_stride, (T*)out, pairs, heads, dim, eps)
    if (dtype == SS_BF16) {
        if (vec) HN_GO(bf16, true); else HN_GO(bf16, false);
    } else {
        if (vec) HN_GO(float, true); else HN_GO(float, false);
    }
#undef HN_GO
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- talking heads
//
// The attention kernels leave, for every query head g and kv head c, head g's weights applied to the values of c:
// x[t][a][c][r][:] with g = a * G + r (common.cuh: head_pair).  Mixing the heads' weights before they meet the values
// is the same sum in another order:
//   out[t][h] = sigmoid(gate[t][h]) * sum_g table[h][g] x[t][g's a][h's c][g's r],      c = h / G.
// table_t: the table transposed, float32 [g][h].  A warp takes TH_OUT heads of one kv head c of one token; a lane four
// elements of D (a multiple of 16, padding behind the values included).
#define TH_OUT 8
template <typename T>
__global__ void __launch_bounds__(128)
talk_heads_kernel(const float* __restrict__ x, const float* __restrict__ table_t, const T* __restrict__ gate,
                  int64_t gate_stride, T* __restrict__ out, int64_t units, int n_kv, int G, int D) {
    pdl_launch_dependents();
    const int lane = threadIdx.x & 31;
    const int64_t unit = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    pdl_wait();
    if (unit >= units) return;
    const int chunks = (G + TH_OUT - 1) / TH_OUT, H = n_kv * G;
    const int chunk = (int)(unit % chunks);
    const int64_t tc = unit / chunks;
    const int c = (int)(tc % n_kv);
    const int64_t t = tc / n_kv;
    const int h0 = c * G + chunk * TH_OUT, n_out = min(TH_OUT, G - chunk * TH_OUT);
    const float* xt = x + t * n_kv * H * D;
    for (int j = lane * 4; j < D; j += 128) {
        float acc[TH_OUT][4];
#pragma unroll
        for (int o = 0; o < TH_OUT; ++o) acc[o][0] = acc[o][1] = acc[o][2] = acc[o][3] = 0.f;
        for (int a = 0; a < n_kv; ++a) {
            const float* xa = xt + (int64_t)(a * n_kv + c) * G * D + j;
            const float* ta = table_t + (int64_t)a * G * H + h0;
#pragma unroll 4
            for (int r = 0; r < G; ++r) {
                float v[4];
                load4(xa + (int64_t)r * D, v);
#pragma unroll
                for (int o = 0; o < TH_OUT; ++o) {
                    const float w = o < n_out ? __ldg(ta + (int64_t)r * H + o) : 0.f;
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[o][e] = fmaf(w, v[e], acc[o][e]);
                }
            }
        }
#pragma unroll
        for (int o = 0; o < TH_OUT; ++o) {
            if (o >= n_out) break;
            if (gate) {
                float g[4];
                load4(gate + t * gate_stride + (int64_t)(h0 + o) * D + j, g);
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[o][e] = gated<sizeof(T) == 2>(acc[o][e], g[e]);
            }
            store4(out + (t * H + h0 + o) * D + j, acc[o]);
        }
    }
}

extern "C" int ss_talk_heads(const float* x, const float* table_t, const void* gate, int64_t gate_stride, void* out, int n_tokens,
                             int n_kv, int G, int D, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int size = dtype == SS_BF16 ? 2 : 4;
    if (n_kv < 1 || G < 1 || D < 4 || D % 4 || ((uintptr_t)x & 15) || (((uintptr_t)gate | (uintptr_t)out) & (4 * size - 1)) || gate_stride % 4)
        return (int)cudaErrorInvalidValue;
    const int64_t units = (int64_t)n_tokens * n_kv * ((G + TH_OUT - 1) / TH_OUT);
    const dim3 grid((unsigned)((units + 3) / 4));
    if (dtype == SS_BF16)
        ss_launch(talk_heads_kernel<bf16>, grid, dim3(128), 0, stream, x, table_t, (const bf16*)gate, gate_stride, (bf16*)out, units, n_kv, G, D);
    else
        ss_launch(talk_heads_kernel<float>, grid, dim3(128), 0, stream, x, table_t, (const float*)gate, gate_stride, (float*)out, units, n_kv, G, D);
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- two branches, each under a norm of its own
//
// out = scale * (a / sqrt(mean(a^2) + eps) * wa + b / sqrt(mean(b^2) + eps) * wb).  A block per row.
template <typename T>
__global__ void __launch_bounds__(256)
normed_pair_kernel(const T* __restrict__ a, const float* __restrict__ wa, const T* __restrict__ b, const float* __restrict__ wb,
                   T* __restrict__ out, int hidden, float eps, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float scratch[2][33];
    const int64_t at = (int64_t)blockIdx.x * hidden;
    float sa = 0.f, sb = 0.f;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
        const float x = to_float(a[at + j]), y = to_float(b[at + j]);
        sa = fmaf(x, x, sa);
        sb = fmaf(y, y, sb);
    }
    const float fa = scale / sqrtf(block_sum(sa, scratch[0]) / (float)hidden + eps);
    const float fb = scale / sqrtf(block_sum(sb, scratch[1]) / (float)hidden + eps);
    for (int j = threadIdx.x; j < hidden; j += blockDim.x)
        out[at + j] = from_float<T>(to_float(a[at + j]) * fa * wa[j] + to_float(b[at + j]) * fb * wb[j]);
}

extern "C" int ss_normed_pair(const void* a, const float* wa, const void* b, const float* wb, void* out, int n_rows, int hidden,
                              float eps, float scale, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (hidden < 1) return (int)cudaErrorInvalidValue;
    if (dtype == SS_BF16)
        ss_launch(normed_pair_kernel<bf16>, dim3(n_rows), dim3(256), 0, stream, (const bf16*)a, wa, (const bf16*)b, wb, (bf16*)out, hidden, eps, scale);
    else
        ss_launch(normed_pair_kernel<float>, dim3(n_rows), dim3(256), 0, stream, (const float*)a, wa, (const float*)b, wb, (float*)out, hidden, eps, scale);
    return SS_LAUNCH_CHECK();
}
