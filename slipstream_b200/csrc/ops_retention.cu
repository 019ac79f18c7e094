// Kernels around retention layers and heads that share their attention weights, beside ops_gated.cu:
//   * the embedding rows under an RMS norm, straight into the float32 stream;
//   * retention over prompt portions on the tensor cores, a chunk of tokens at a time;
//   * the output of a retention layer: every head over its root mean square, under a silu gate;
//   * talking heads: each head's output as a mixture over the heads' attention weights, under a sigmoid gate;
//   * the weighted sum of two branches, each under an RMS norm of its own.
// Norms, gates and mixtures are float32; T is the compute type of projections and activations.
#include "mma_sync.cuh"

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
// table_t: the table transposed, float32 [g][h].  A block takes TH_OUT heads of one kv head c of TH_ROWS tokens, with the part of
// the table it needs in shared memory; LP lanes share a token's row of D elements (a multiple of 4, padding behind the values
// included), four elements a lane and pass.
#define TH_OUT 8
#define TH_WARPS 8
template <typename T, int LP>
__global__ void __launch_bounds__(TH_WARPS * 32)
talk_heads_kernel(const float* __restrict__ x, const float* __restrict__ table_t, const T* __restrict__ gate,
                  int64_t gate_stride, T* __restrict__ out, int n_tokens, int n_kv, int G, int D) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float th_smem[];  // [g][TH_OUT]
    const int chunks = (G + TH_OUT - 1) / TH_OUT, H = n_kv * G;
    const int c = blockIdx.y / chunks, chunk = blockIdx.y - c * chunks;
    const int h0 = c * G + chunk * TH_OUT, n_out = min(TH_OUT, G - chunk * TH_OUT);
    for (int i = threadIdx.x; i < H * TH_OUT; i += TH_WARPS * 32) {
        const int g = i / TH_OUT, o = i % TH_OUT;
        th_smem[i] = o < n_out ? table_t[(int64_t)g * H + h0 + o] : 0.f;
    }
    __syncthreads();
    pdl_wait();
    const int sub = threadIdx.x % LP;
    const int t = blockIdx.x * (TH_WARPS * 32 / LP) + threadIdx.x / LP;
    if (t >= n_tokens) return;
    const int64_t a_stride = (int64_t)n_kv * G * D;
    const float* xt = x + (int64_t)t * n_kv * a_stride + (int64_t)c * G * D;
    for (int j = sub * 4; j < D; j += LP * 4) {
        float acc[TH_OUT][4];
#pragma unroll
        for (int o = 0; o < TH_OUT; ++o) acc[o][0] = acc[o][1] = acc[o][2] = acc[o][3] = 0.f;
        for (int a = 0; a < n_kv; ++a) {
            const float* xa = xt + a * a_stride + j;
            const float* ta = th_smem + a * G * TH_OUT;
            for (int r0 = 0; r0 < G; r0 += 8) {
                float v[8][4];  // eight rows in flight
#pragma unroll
                for (int r = 0; r < 8; ++r)
                    if (r0 + r < G) load4(xa + (r0 + r) * D, v[r]);
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    if (r0 + r >= G) break;
                    float w[TH_OUT];
                    *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(ta + (r0 + r) * TH_OUT);
                    *reinterpret_cast<float4*>(w + 4) = *reinterpret_cast<const float4*>(ta + (r0 + r) * TH_OUT + 4);
#pragma unroll
                    for (int o = 0; o < TH_OUT; ++o)
#pragma unroll
                        for (int e = 0; e < 4; ++e) acc[o][e] = fmaf(w[o], v[r][e], acc[o][e]);
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
            store4(out + ((int64_t)t * H + h0 + o) * D + j, acc[o]);
        }
    }
}

template <typename T, int LP>
static int launch_talk_heads(const float* x, const float* table_t, const void* gate, int64_t gate_stride, void* out, int n_tokens,
                             int n_kv, int G, int D, cudaStream_t stream) {
    const int smem = n_kv * G * TH_OUT * 4, rows = TH_WARPS * 32 / LP;
    if (smem > 48 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid((n_tokens + rows - 1) / rows, n_kv * ((G + TH_OUT - 1) / TH_OUT));
    ss_launch(talk_heads_kernel<T, LP>, grid, dim3(TH_WARPS * 32), smem, stream, x, table_t, (const T*)gate, gate_stride, (T*)out, n_tokens, n_kv, G, D);
    return SS_LAUNCH_CHECK();
}

extern "C" int ss_talk_heads(const float* x, const float* table_t, const void* gate, int64_t gate_stride, void* out, int n_tokens,
                             int n_kv, int G, int D, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    const int size = dtype == SS_BF16 ? 2 : 4;
    if (n_kv < 1 || G < 1 || D < 4 || D % 4 || ((uintptr_t)x & 15) || (((uintptr_t)gate | (uintptr_t)out) & (4 * size - 1)) || gate_stride % 4)
        return (int)cudaErrorInvalidValue;
#define TH_GO(T)                                                                                                      \
    do {                                                                                                              \
        if (D <= 16) return launch_talk_heads<T, 4>(x, table_t, gate, gate_stride, out, n_tokens, n_kv, G, D, stream);  \
        if (D <= 32) return launch_talk_heads<T, 8>(x, table_t, gate, gate_stride, out, n_tokens, n_kv, G, D, stream);  \
        if (D <= 64) return launch_talk_heads<T, 16>(x, table_t, gate, gate_stride, out, n_tokens, n_kv, G, D, stream); \
        return launch_talk_heads<T, 32>(x, table_t, gate, gate_stride, out, n_tokens, n_kv, G, D, stream);              \
    } while (0)
    if (dtype == SS_BF16) TH_GO(bf16);
    TH_GO(float);
#undef TH_GO
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

// ---------------------------------------------------------------- retention over prompt portions, a chunk at a time
//
// The recurrence S <- g S + k v^T, o = S^T q of a head (g its decay) over a chunk of C tokens from the state S_0 in front
// of it is, exactly:
//   o_t = g^(t+1) S_0^T q_t + sum_{s <= t} g^(t-s) (q_t . k_s) v_s,        S_C = g^C S_0 + sum_s g^(C-1-s) k_s v_s^T,
// products of matrices instead of C dependent steps.  q and k are rotated (pairs (i, i + half), k times k_scale) and the
// state is kept in float32; every float32 operand of a product is cut into two bfloat16 parts, x = hi + lo with a remainder
// below 2^-17 |x|, and the products hi hi + hi lo + lo hi are accumulated in float32 (the values v are bfloat16 as projected).
//
// A block of 16 warps takes RC_COLS value columns of a head of a request and walks its tokens in chunks of RC_T:
//   * the chunk's rows arrive in shared memory by asynchronous copies issued while the chunk in front is computed;
//   * they are rotated and cut in two: a thread has one run of 8 pairs of a row of q and of k, and the cosines and sines of
//     that row's offset in the chunk in registers, those of the chunk's first position are formed once a chunk; k_scale is
//     left to the factors that the scores and the values meet anyway;
//   * four warps share 16 rows: each takes 16 keys of the scores and a quarter of the state's rows, and their sums meet in
//     shared memory;
//   * the state stays in registers as accumulators, cut in two in shared memory once a chunk.
// proj, state, out as for the token-by-token kernel (ops_gated.cu).  D: 64 or 128, at least the head's dim; zeros behind it.
#define RC_T 64
#define RC_COLS 32
#define RC_THREADS 512

template <int D>
struct RcSmem {
    static constexpr int S = D + 8, V = RC_COLS + 8;          // strides that spread ldmatrix over all banks
    static constexpr int raw_qk = 0;                          // bf16 [2][RC_T][D]
    static constexpr int raw_v = raw_qk + 2 * RC_T * D * 2;   // bf16 [RC_T][RC_COLS]
    static constexpr int qk = raw_v + RC_T * RC_COLS * 2;     // bf16 [q hi, q lo, k hi, k lo][RC_T][S]
    static constexpr int v = qk + 4 * RC_T * S * 2;           // bf16 [v, g^(n-1-s) v: hi, lo][RC_T][V]
    static constexpr int st = v + 3 * RC_T * V * 2;           // bf16 [state hi, lo][D][V]
    static constexpr int sum = st + 2 * D * V * 2;            // float [4][RC_T][V]
    static constexpr int pw = sum + 4 * RC_T * V * 4;         // float [RC_T + 4]: powers of the decay
    static constexpr int pk = pw + (RC_T + 4) * 4;            // float [RC_T + 4]: the same times k_scale
    static constexpr int base = pk + (RC_T + 4) * 4;          // float2 [D / 2]: the chunk's first position
    static constexpr int bytes = base + D / 2 * 8;
};

__device__ __forceinline__ void cut_in_two(const float (&x)[8], uint4& hi, uint4& lo) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        h[e] = pack_bf16(x[2 * e], x[2 * e + 1]);
        l[e] = pack_bf16(x[2 * e] - __uint_as_float(h[e] << 16), x[2 * e + 1] - __uint_as_float(h[e] & 0xffff0000u));
    }
    hi = make_uint4(h[0], h[1], h[2], h[3]);
    lo = make_uint4(l[0], l[1], l[2], l[3]);
}
__device__ __forceinline__ void eight(const uint4& r, float (&v)[8]) {
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        v[2 * e] = __uint_as_float(w[e] << 16);
        v[2 * e + 1] = __uint_as_float(w[e] & 0xffff0000u);
    }
}

template <int D>
__global__ void __launch_bounds__(RC_THREADS)
retention_chunks_kernel(const bf16* __restrict__ proj, int64_t stride, const float* __restrict__ decay, float* __restrict__ state,
                        float* __restrict__ out, const int32_t* __restrict__ q_start, const int32_t* __restrict__ seq_lens,
                        const int32_t* __restrict__ slots, int heads, int dim, int vdim, int n_slots, int* err,
                        const float* __restrict__ inv_freq, int half, float k_scale) {
    using M = RcSmem<D>;
    constexpr int S = M::S, V = M::V, KS = D / 16, NT = RC_COLS / 8;
    constexpr int UT = NT / 2;  // column tiles of the state a warp holds (of 16 rows); with D = 64 half of the warps hold any
    extern __shared__ __align__(16) unsigned char smem[];
    bf16* raw = reinterpret_cast<bf16*>(smem + M::raw_qk);
    bf16* raw_v = reinterpret_cast<bf16*>(smem + M::raw_v);
    bf16* Qh = reinterpret_cast<bf16*>(smem + M::qk);
    bf16* Ql = Qh + RC_T * S;
    bf16* Kh = Ql + RC_T * S;
    bf16* Kl = Kh + RC_T * S;
    bf16* Vs = reinterpret_cast<bf16*>(smem + M::v);
    bf16* Wh = Vs + RC_T * V;
    bf16* Wl = Wh + RC_T * V;
    bf16* Sh = reinterpret_cast<bf16*>(smem + M::st);
    bf16* Sl = Sh + D * V;
    float* sums = reinterpret_cast<float*>(smem + M::sum);
    float* pw = reinterpret_cast<float*>(smem + M::pw);
    float2* base = reinterpret_cast<float2*>(smem + M::base);
    float* pk = reinterpret_cast<float*>(smem + M::pk);

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int col_blocks = (vdim + RC_COLS - 1) / RC_COLS;
    const int h = blockIdx.x / col_blocks, c0 = (blockIdx.x % col_blocks) * RC_COLS, r = blockIdx.y;
    const float g = decay[h];
    const int half8 = half / 8;
    pdl_launch_dependents();
    // this thread's run of pairs: elements 8 tc .. and half further of row tt of a chunk
    static_assert(RC_T * (D / 16) <= RC_THREADS, "a thread has at most one run of pairs");
    const bool turns = tid < RC_T * half8;
    const int tt = turns ? tid / half8 : 0, tc = turns ? tid - tt * half8 : 0;
    float2 off[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) off[e] = make_float2(1.f, 0.f);
    if (turns) {  // (constants of the layer: before the kernels in front are complete)
#pragma unroll 1
        for (int e = 0; e < 8; ++e) {
            float sn, cs;
            sincosf(__fmul_rn((float)tt, inv_freq[tc * 8 + e]), &sn, &cs);
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (k == e) off[k] = make_float2(cs, sn);
        }
    }
    for (int i = tid; i <= RC_T; i += RC_THREADS) {
        pw[i] = powf(g, (float)i);
        pk[i] = pw[i] * k_scale;
    }
    pdl_wait();
    const int q0 = q_start[r], q_len = q_start[r + 1] - q0, seq_len = seq_lens[r];
    if (q_len <= 0 || seq_len <= 0) return;
    const int slot = slots[r];
    if (slot < 0 || slot >= n_slots) {
        if (tid == 0) atomicOr(err, SS_ERR_SLOT_RANGE);
        return;
    }
    const int pos0 = seq_len - q_len;
    const int64_t k_off = (int64_t)heads * dim, v_off = 2 * k_off + (int64_t)h * vdim + c0;

    // a chunk's rows into shared memory, 16 bytes a copy; zeros behind the last row, the head's last element and its last column
    constexpr int RUNS = D / 8, ROWS = RC_THREADS / RUNS;  // runs of 8 elements of a row; rows a pass over the threads covers
    const int ft = tid / RUNS, fc = (tid % RUNS) * 8;
    const bf16* f_src = proj + (int64_t)(q0 + ft) * stride + (int64_t)h * dim + (fc < dim ? fc : 0);
    const int vt = tid / (RC_COLS / 8), vc = (tid % (RC_COLS / 8)) * 8;  // (the values: a quarter or half of the threads)
    auto fetch = [&](int t0) {
#pragma unroll
        for (int w = 0; w < RC_T / ROWS; ++w) {
            const bool ok = t0 + ft + w * ROWS < q_len && fc < dim;
            const bf16* src = ok ? f_src + (int64_t)(t0 + w * ROWS) * stride : proj;
            cp_async16(raw + (ft + w * ROWS) * D + fc, src, ok);
            cp_async16(raw + (RC_T + ft + w * ROWS) * D + fc, ok ? src + k_off : proj, ok);
        }
        if (tid < RC_T * (RC_COLS / 8)) {
            const bool ok = t0 + vt < q_len && c0 + vc < vdim;
            cp_async16(raw_v + vt * RC_COLS + vc, ok ? proj + (int64_t)(q0 + t0 + vt) * stride + v_off + vc : proj, ok);
        }
        cp_async_commit();
    };
    fetch(0);

    // the state as accumulators: this warp's 16 rows and UT column tiles
    const int s_row = (warp % (D / 16)) * 16 + (lane >> 2), s_nt = warp / (D / 16) * UT;
    const bool s_mine = s_nt < NT && s_row - (lane >> 2) < dim;
    float* sp = state + ((int64_t)slot * heads + h) * dim * vdim;
    float acc_s[UT][4];
#pragma unroll
    for (int n = 0; n < UT; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int row = s_row + e * 8, col = c0 + (s_nt + n) * 8 + (lane & 3) * 2;
            float2 x = make_float2(0.f, 0.f);
            if (s_mine && row < dim && col < vdim) x = *reinterpret_cast<const float2*>(sp + (int64_t)row * vdim + col);
            acc_s[n][2 * e] = x.x;
            acc_s[n][2 * e + 1] = x.y;
        }
    const int rt = warp & 3, part = warp >> 2;  // rows 16 rt .. of the chunk; which keys and which of the state's rows

    for (int t0 = 0; t0 < q_len; t0 += RC_T) {
        const int nb = min(RC_T, q_len - t0);
        for (int i = tid; i < half; i += RC_THREADS) {
            float sn, cs;
            sincosf(__fmul_rn((float)(pos0 + t0), inv_freq[i]), &sn, &cs);
            base[(i & 7) * half8 + (i >> 3)] = make_float2(cs, sn);
        }
        cp_async_wait<0>();
        __syncthreads();  // the rows and the chunk's first angles; and the chunk in front is done with everything below
        // rotated pairs
        if (turns) {
            float cs[8], sn[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const float2 b = base[e * half8 + tc];
                cs[e] = off[e].x * b.x - off[e].y * b.y;
                sn[e] = off[e].y * b.x + off[e].x * b.y;
            }
#pragma unroll
            for (int which = 0; which < 2; ++which) {
                const bf16* src = raw + (which * RC_T + tt) * D + tc * 8;
                bf16* hi = (which ? Kh : Qh) + tt * S + tc * 8;
                bf16* lo = (which ? Kl : Ql) + tt * S + tc * 8;
                float u[8], v[8];
                eight(*reinterpret_cast<const uint4*>(src), u);
                eight(*reinterpret_cast<const uint4*>(src + half), v);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float x = u[e] * cs[e] - v[e] * sn[e];
                    v[e] = v[e] * cs[e] + u[e] * sn[e];
                    u[e] = x;
                }
                uint4 ph, pl;
                cut_in_two(u, ph, pl);
                *reinterpret_cast<uint4*>(hi) = ph;
                *reinterpret_cast<uint4*>(lo) = pl;
                cut_in_two(v, ph, pl);
                *reinterpret_cast<uint4*>(hi + half) = ph;
                *reinterpret_cast<uint4*>(lo + half) = pl;
            }
        }
        // elements that are not rotated (and the zeros behind the head): bfloat16 as they came
        const int rest8 = D / 8 - 2 * half8;
        for (int i = tid; i < 2 * RC_T * rest8; i += RC_THREADS) {
            const int row = i / rest8, c = 2 * half + (i - row * rest8) * 8, t = row % RC_T;
            const bool keys = row >= RC_T;
            *reinterpret_cast<uint4*>((keys ? Kh : Qh) + t * S + c) = *reinterpret_cast<const uint4*>(raw + row * D + c);
            *reinterpret_cast<uint4*>((keys ? Kl : Ql) + t * S + c) = make_uint4(0u, 0u, 0u, 0u);
        }
        if (tid < RC_T * (RC_COLS / 8)) {
            const uint4 w = *reinterpret_cast<const uint4*>(raw_v + vt * RC_COLS + vc);
            *reinterpret_cast<uint4*>(Vs + vt * V + vc) = w;
            float u[8];
            eight(w, u);
            const float f = vt < nb ? pk[nb - 1 - vt] : 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) u[e] *= f;
            uint4 ph, pl;
            cut_in_two(u, ph, pl);
            *reinterpret_cast<uint4*>(Wh + vt * V + vc) = ph;
            *reinterpret_cast<uint4*>(Wl + vt * V + vc) = pl;
        }
        if (s_nt < NT) {
#pragma unroll
            for (int n = 0; n < UT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int at = (s_row + e * 8) * V + (s_nt + n) * 8 + (lane & 3) * 2;
                    const float x = acc_s[n][2 * e], y = acc_s[n][2 * e + 1];
                    const uint32_t hi = pack_bf16(x, y);
                    *reinterpret_cast<uint32_t*>(Sh + at) = hi;
                    *reinterpret_cast<uint32_t*>(Sl + at) = pack_bf16(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
                }
        }
        __syncthreads();
        if (t0 + RC_T < q_len) fetch(t0 + RC_T);  // the rows as they came have been used up

        // scores of 16 rows with 16 keys up to the diagonal, and a quarter of q S_0
        const bool rows_on = rt * 16 < nb, keys_on = part <= rt;
        float sc[2][4], o[NT][4];
#pragma unroll
        for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
#pragma unroll
        for (int n = 0; n < 2; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
        if (rows_on) {
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                const bool state_on = ks / (KS / 4) == part;
                if (!keys_on && !state_on) continue;
                uint32_t qh[4], ql[4];
                const int qa = (rt * 16 + (lane & 15)) * S + ks * 16 + ((lane >> 4) << 3);
                ldmatrix_x4(qh, Qh + qa);
                ldmatrix_x4(ql, Ql + qa);
                if (keys_on) {
                    uint32_t kh[4], kl[4];
                    const int ka = (part * 16 + (lane & 7) + ((lane >> 4) << 3)) * S + ks * 16 + (((lane >> 3) & 1) << 3);
                    ldmatrix_x4(kh, Kh + ka);
                    ldmatrix_x4(kl, Kl + ka);
#pragma unroll
                    for (int n = 0; n < 2; ++n) {
                        mma_bf16(sc[n], qh, kh[2 * n], kh[2 * n + 1]);
                        mma_bf16(sc[n], qh, kl[2 * n], kl[2 * n + 1]);
                        mma_bf16(sc[n], ql, kh[2 * n], kh[2 * n + 1]);
                    }
                }
                if (state_on) {
#pragma unroll
                    for (int n = 0; n < NT; n += 2) {
                        uint32_t sh[4], sl[4];
                        const int sa = (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * V + n * 8 + ((lane >> 4) << 3);
                        ldmatrix_x4_trans(sh, Sh + sa);
                        ldmatrix_x4_trans(sl, Sl + sa);
#pragma unroll
                        for (int m = 0; m < 2; ++m) {
                            mma_bf16(o[n + m], qh, sh[2 * m], sh[2 * m + 1]);
                            mma_bf16(o[n + m], qh, sl[2 * m], sl[2 * m + 1]);
                            mma_bf16(o[n + m], ql, sh[2 * m], sh[2 * m + 1]);
                        }
                    }
                }
            }
            const int row_lo = rt * 16 + (lane >> 2), row_hi = row_lo + 8;
            const float f_lo = pw[row_lo + 1], f_hi = pw[row_hi + 1];
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                o[n][0] *= f_lo; o[n][1] *= f_lo;
                o[n][2] *= f_hi; o[n][3] *= f_hi;
            }
            if (keys_on) {
                uint32_t ah[4], al[4];
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const int key = part * 16 + n * 8 + ((lane & 3) << 1);
                    float x[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int back = (e < 2 ? row_lo : row_hi) - (key + (e & 1));
                        x[e] = back >= 0 ? sc[n][e] * pk[back] : 0.f;
                    }
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const uint32_t hi = pack_bf16(x[2 * e], x[2 * e + 1]);
                        ah[2 * n + e] = hi;
                        al[2 * n + e] = pack_bf16(x[2 * e] - __uint_as_float(hi << 16), x[2 * e + 1] - __uint_as_float(hi & 0xffff0000u));
                    }
                }
#pragma unroll
                for (int n = 0; n < NT; n += 2) {
                    uint32_t vv[4];
                    ldmatrix_x4_trans(vv, Vs + (part * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * V + n * 8 + ((lane >> 4) << 3));
#pragma unroll
                    for (int m = 0; m < 2; ++m) {
                        mma_bf16(o[n + m], ah, vv[2 * m], vv[2 * m + 1]);
                        mma_bf16(o[n + m], al, vv[2 * m], vv[2 * m + 1]);
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    *reinterpret_cast<float2*>(sums + (part * RC_T + row_lo + e * 8) * V + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * e], o[n][2 * e + 1]);
        }
        // the state behind the chunk
        if (s_mine) {
            const float f = pw[nb];
#pragma unroll
            for (int n = 0; n < UT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc_s[n][e] *= f;
            const int m0 = s_row - (lane >> 2);
#pragma unroll
            for (int ks = 0; ks < RC_T / 16; ++ks) {
                if (ks * 16 >= nb) break;
                uint32_t kh[4], kl[4];
                const int ka = (ks * 16 + (lane & 7) + ((lane >> 4) << 3)) * S + m0 + (((lane >> 3) & 1) << 3);
                ldmatrix_x4_trans(kh, Kh + ka);
                ldmatrix_x4_trans(kl, Kl + ka);
#pragma unroll
                for (int n = 0; n < UT; n += 2) {
                    uint32_t wh[4], wl[4];
                    const int wa = (ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3)) * V + (s_nt + n) * 8 + ((lane >> 4) << 3);
                    ldmatrix_x4_trans(wh, Wh + wa);
                    ldmatrix_x4_trans(wl, Wl + wa);
#pragma unroll
                    for (int m = 0; m < 2; ++m) {
                        mma_bf16(acc_s[n + m], kh, wh[2 * m], wh[2 * m + 1]);
                        mma_bf16(acc_s[n + m], kh, wl[2 * m], wl[2 * m + 1]);
                        mma_bf16(acc_s[n + m], kl, wh[2 * m], wh[2 * m + 1]);
                    }
                }
            }
        }
        __syncthreads();
        {
            const int t = tid / (RC_COLS / 4), c = (tid % (RC_COLS / 4)) * 4;
            static_assert(RC_THREADS == RC_T * (RC_COLS / 4), "a thread adds four neighbouring sums");
            if (t < nb && c0 + c < vdim) {
                float4 x = *reinterpret_cast<const float4*>(sums + t * V + c);
#pragma unroll
                for (int p = 1; p < 4; ++p) {
                    const float4 y = *reinterpret_cast<const float4*>(sums + (p * RC_T + t) * V + c);
                    x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
                }
                *reinterpret_cast<float4*>(out + ((int64_t)(q0 + t0 + t) * heads + h) * vdim + c0 + c) = x;
            }
        }
    }
#pragma unroll
    for (int n = 0; n < UT; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int row = s_row + e * 8, col = c0 + (s_nt + n) * 8 + (lane & 3) * 2;
            if (s_mine && row < dim && col < vdim) *reinterpret_cast<float2*>(sp + (int64_t)row * vdim + col) = make_float2(acc_s[n][2 * e], acc_s[n][2 * e + 1]);
        }
}

template <int D>
static int launch_retention_chunks(const bf16* proj, int64_t stride, const float* decay, float* state, float* out, const int32_t* q_start,
                                   const int32_t* seq_lens, const int32_t* slots, int R, int heads, int dim, int vdim, int n_slots, int* err,
                                   cudaStream_t stream, const float* inv_freq, int half, float k_scale) {
    constexpr int smem = RcSmem<D>::bytes;
    static SsPerDevice opted;
    if (int rc = ss_opt_in_smem(retention_chunks_kernel<D>, smem, opted)) return rc;
    ss_launch(retention_chunks_kernel<D>, dim3(heads * ((vdim + RC_COLS - 1) / RC_COLS), R), dim3(RC_THREADS), smem, stream, proj, stride, decay,
              state, out, q_start, seq_lens, slots, heads, dim, vdim, n_slots, err, inv_freq, half, k_scale);
    return SS_LAUNCH_CHECK();
}

// bfloat16 rows; dim at most 128, dim, vdim, stride and half in steps of 8, proj, state and out on 16-byte boundaries.
extern "C" int ss_retention_chunks(const void* proj, int64_t stride, const float* decay, float* state, float* out, const int32_t* q_start,
                                   const int32_t* seq_lens, const int32_t* slots, int R, int heads, int dim, int vdim, int n_slots, int* err,
                                   cudaStream_t stream, const float* inv_freq, int half, float k_scale) {
    if (R <= 0) return 0;
    if (heads < 1 || dim < 8 || dim > 128 || vdim < 8 || dim % 8 || vdim % 8 || stride % 8 || half < 0 || half % 8 || 2 * half > dim ||
        (half > 0 && !inv_freq) || (((uintptr_t)proj | (uintptr_t)state | (uintptr_t)out) & 15))
        return (int)cudaErrorInvalidValue;
    if (dim <= 64)
        return launch_retention_chunks<64>((const bf16*)proj, stride, decay, state, out, q_start, seq_lens, slots, R, heads, dim, vdim, n_slots, err,
                                           stream, inv_freq, half, k_scale);
    return launch_retention_chunks<128>((const bf16*)proj, stride, decay, state, out, q_start, seq_lens, slots, R, heads, dim, vdim, n_slots, err,
                                        stream, inv_freq, half, k_scale);
}

// ---------------------------------------------------------------- retention of single tokens, head norm and gate included
//
// A decode step: every request brings one token.  S <- g S + k v^T, o = S^T q as above, then o / sqrt(mean(o^2) + eps) *
// silu(gate) head by head, in T.  A block takes a head of a request whole: a thread holds four neighbouring columns of every
// RG-th row of the state, all its loads in flight before the first is used; the row groups' sums meet in shared memory.
// vdim a multiple of 4 up to 256.
#define RD_THREADS 512
#define RD_ROWS 8  // rows of the state a thread has in flight
template <typename T>
__global__ void __launch_bounds__(RD_THREADS, 2)
retention_token_kernel(const T* __restrict__ proj, int64_t stride, const float* __restrict__ decay, float* __restrict__ state,
                       T* __restrict__ out, const int32_t* __restrict__ q_start, const int32_t* __restrict__ seq_lens,
                       const int32_t* __restrict__ slots, int heads, int dim, int vdim, int n_slots, int* err,
                       const float* __restrict__ inv_freq, int half, float k_scale, float eps) {
    __shared__ float qs[256], ks[256], scratch[33];
    __shared__ __align__(16) float sums[4 * RD_THREADS];
    const int tid = threadIdx.x, h = blockIdx.x, r = blockIdx.y;
    const int cols4 = vdim >> 2, groups = RD_THREADS / cols4;
    const int c4 = tid % cols4, rg = tid / cols4;
    const bool on = rg < groups;
    const float g = decay[h];
    pdl_launch_dependents();
    pdl_wait();
    const int seq_len = seq_lens[r];
    if (q_start[r + 1] <= q_start[r] || seq_len <= 0) return;
    const int slot = slots[r];
    if (slot < 0 || slot >= n_slots) {
        if (tid == 0) atomicOr(err, SS_ERR_SLOT_RANGE);
        return;
    }
    float4* sp = reinterpret_cast<float4*>(state + ((int64_t)slot * heads + h) * dim * vdim) + c4;
    float4 s[RD_ROWS];
#pragma unroll
    for (int i = 0; i < RD_ROWS; ++i) {
        const int row = rg + i * groups;
        if (on && row < dim) s[i] = sp[(int64_t)row * cols4];
    }
    const int64_t row_q = q_start[r];
    const T* src = proj + row_q * stride;
    const int64_t k_off = (int64_t)heads * dim;
    for (int i = tid; i < dim; i += RD_THREADS) {
        if (i < half) {
            float sn, cs;
            sincosf(__fmul_rn((float)(seq_len - 1), inv_freq[i]), &sn, &cs);
            const float q1 = to_float(src[(int64_t)h * dim + i]), q2 = to_float(src[(int64_t)h * dim + i + half]);
            const float k1 = to_float(src[k_off + (int64_t)h * dim + i]), k2 = to_float(src[k_off + (int64_t)h * dim + i + half]);
            qs[i] = q1 * cs - q2 * sn;
            qs[i + half] = q2 * cs + q1 * sn;
            ks[i] = (k1 * cs - k2 * sn) * k_scale;
            ks[i + half] = (k2 * cs + k1 * sn) * k_scale;
        } else if (i >= 2 * half) {
            qs[i] = to_float(src[(int64_t)h * dim + i]);
            ks[i] = to_float(src[k_off + (int64_t)h * dim + i]) * k_scale;
        }
    }
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    const T* vp = src + 2 * k_off + (int64_t)h * vdim;
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = to_float(vp[c4 * 4 + e]);
    __syncthreads();
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    auto row_of = [&](const float4& old, int row) {
        const float k = ks[row], q = qs[row];
        float4 n;
        n.x = fmaf(k, v[0], g * old.x); n.y = fmaf(k, v[1], g * old.y);
        n.z = fmaf(k, v[2], g * old.z); n.w = fmaf(k, v[3], g * old.w);
        o[0] = fmaf(n.x, q, o[0]); o[1] = fmaf(n.y, q, o[1]);
        o[2] = fmaf(n.z, q, o[2]); o[3] = fmaf(n.w, q, o[3]);
        sp[(int64_t)row * cols4] = n;
    };
    if (on) {
#pragma unroll
        for (int i = 0; i < RD_ROWS; ++i) {
            const int row = rg + i * groups;
            if (row < dim) row_of(s[i], row);
        }
        for (int row = rg + RD_ROWS * groups; row < dim; row += groups) row_of(sp[(int64_t)row * cols4], row);
        *reinterpret_cast<float4*>(sums + (rg * cols4 + c4) * 4) = make_float4(o[0], o[1], o[2], o[3]);
    }
    __syncthreads();
    float x = 0.f;
    if (tid < vdim)
        for (int i = 0; i < groups; ++i) x += sums[i * vdim + tid];
    const float f = 1.0f / sqrtf(block_sum(x * x, scratch) / (float)vdim + eps);
    if (tid < vdim) {
        const int64_t at = (int64_t)h * vdim + tid;
        const float gate = to_float(src[2 * k_off + (int64_t)heads * vdim + at]);
        out[row_q * heads * vdim + at] = from_float<T>(x * f * silu_of<T>(gate));
    }
}

// proj row: [q | k | v | gate], heads * (2 dim + 2 vdim) elements; out [rows][heads * vdim] in the type of proj.
extern "C" int ss_retention_token(const void* proj, int64_t stride, const float* decay, float* state, void* out, const int32_t* q_start,
                                  const int32_t* seq_lens, const int32_t* slots, int R, int heads, int dim, int vdim, int n_slots, int dtype,
                                  int* err, cudaStream_t stream, const float* inv_freq, int half, float k_scale, float eps) {
    if (R <= 0) return 0;
    if (heads < 1 || dim < 1 || dim > 256 || vdim < 4 || vdim > 256 || vdim % 4 || half < 0 || 2 * half > dim || (half > 0 && !inv_freq) ||
        ((uintptr_t)state & 15))
        return (int)cudaErrorInvalidValue;
    const dim3 grid(heads, R), block(RD_THREADS);
    if (dtype == SS_BF16)
        ss_launch(retention_token_kernel<bf16>, grid, block, 0, stream, (const bf16*)proj, stride, decay, state, (bf16*)out, q_start, seq_lens,
                  slots, heads, dim, vdim, n_slots, err, inv_freq, half, k_scale, eps);
    else
        ss_launch(retention_token_kernel<float>, grid, block, 0, stream, (const float*)proj, stride, decay, state, (float*)out, q_start, seq_lens,
                  slots, heads, dim, vdim, n_slots, err, inv_freq, half, k_scale, eps);
    return SS_LAUNCH_CHECK();
}
