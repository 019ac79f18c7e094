// Kernels between a layer's products and its attention, and behind them:
//  * heads_to_pages: projected queries, keys and values into the forms the paged attention kernels read;
//  * diff_combine: the two maps of differential heads into one output;
//  * branch_norm: a branch's normed output joins the stream, and the next norm of the stream.
// All arithmetic is float32 and rounds once where it is written.
#include "common.cuh"

// Sum over the block with one barrier: every thread adds the warps' sums in the same order.  `scratch` (32 floats) may
// not be written again before the next barrier of the block.
__device__ __forceinline__ float block_sum_once(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    return warp_sum(lane < n_warps ? scratch[lane] : 0.f);
}

__device__ __forceinline__ void unpack8(const uint4& r, float (&v)[8]) {
    const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        v[2 * e] = __uint_as_float(w[e] << 16);
        v[2 * e + 1] = __uint_as_float(w[e] & 0xffff0000u);
    }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
    uint32_t w[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const __nv_bfloat162 p = __floats2bfloat162_rn(v[2 * e], v[2 * e + 1]);
        w[e] = *reinterpret_cast<const uint32_t*>(&p);
    }
    return make_uint4(w[0], w[1], w[2], w[3]);
}
__device__ __forceinline__ void load8f(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
__device__ __forceinline__ void store8f(float* p, const float (&v)[8]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

// ---------------------------------------------------------------- projected heads -> queries and pages
//
// A row holds n_q * M query parts and (from k_col) n_kv * M key parts of d elements, M the maps of a head (1, or 2 for
// differential heads: [map 1 | map 2] head by head), and from v_col n_kv values of dv elements (v_col may be k_col: the
// values are then the keys as projected).  Per token:
//   norm      with q_weight / k_weight: x / sqrt(mean(x^2) + eps) * w over ALL queries of the token at once, and over all
//             its keys at once (not the values);
//   rotation  of the first rot_dim elements of every part by position * inv_freq, in pairs of neighbours (2i, 2i + 1) or,
//             not interleaved, (i, i + rot_dim / 2);
//   queries   to q_out [token][n_q * M][D]: the part of map m of a head lies at m * d of its D elements, zeros elsewhere;
//   keys      to their page: all maps of a kv head side by side in one row of D elements, zeros behind them;
//   values    to theirs: dv elements, zeros behind them.
// The score of query (head, map m) with such a key row is that of map m alone, so the attention kernels run n_q * M
// query heads over n_kv key/value heads of D >= max(M * d, dv) elements.  kv: [page][2][kv head][offset][D].
// Two kernels: one with 16-byte accesses (bfloat16, sizes in runs of 8, pairs of neighbours), one for any type and size.
struct HeadsArgs {
    const void* rows;
    int64_t row_stride;
    const int32_t* positions;
    const int32_t* slots;
    const float* inv_freq;
    const float* q_weight;
    const float* k_weight;
    void* q_out;
    void* kv;
    int n_q, n_kv, maps, d, dv, D, k_col, v_col, rot_dim, interleaved, page_size;
    float eps;
    int64_t pool_slots;
    int* err;
};

// Any type and size: a block per token, a thread per element.
template <typename T>
__global__ void __launch_bounds__(256) heads_to_pages_kernel(const HeadsArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float cos_s[128], sin_s[128], scratch[2][32];
    const int t = blockIdx.x;
    const T* row = reinterpret_cast<const T*>(a.rows) + (int64_t)t * a.row_stride;
    const float pos = (float)a.positions[t];
    for (int i = threadIdx.x; i < a.rot_dim / 2; i += blockDim.x) sincosf(__fmul_rn(pos, a.inv_freq[i]), &sin_s[i], &cos_s[i]);
    int64_t slot = (a.slots && a.kv) ? (int64_t)a.slots[t] : -1;
    if (slot >= a.pool_slots) {
        if (threadIdx.x == 0) atomicOr(a.err, SS_ERR_SLOT_RANGE);
        slot = -1;
    }
    const int md = a.maps * a.d, D = a.D;
    const int q_len = a.n_q * md, k_len = a.n_kv * md;
    float q_rstd = 1.f, k_rstd = 1.f;
    if (a.q_weight) {
        float sq = 0.f, sk = 0.f;
        for (int c = threadIdx.x; c < q_len; c += blockDim.x) sq = fmaf(to_float(row[c]), to_float(row[c]), sq);
        for (int c = threadIdx.x; c < k_len; c += blockDim.x) sk = fmaf(to_float(row[a.k_col + c]), to_float(row[a.k_col + c]), sk);
        q_rstd = 1.0f / sqrtf(block_sum_once(sq, scratch[0]) / (float)q_len + a.eps);
        k_rstd = 1.0f / sqrtf(block_sum_once(sk, scratch[1]) / (float)k_len + a.eps);
    } else {
        __syncthreads();
    }
    const int64_t page = slot >= 0 ? slot / a.page_size : 0;
    const int off = slot >= 0 ? (int)(slot % a.page_size) : 0;
    const int q_runs = a.n_q * a.maps * D, kv_runs = slot >= 0 ? a.n_kv * D : 0;
    T* const q_out = reinterpret_cast<T*>(a.q_out) + (int64_t)t * q_runs;
    T* const kv = reinterpret_cast<T*>(a.kv);
    for (int run = threadIdx.x; run < q_runs + 2 * kv_runs; run += blockDim.x) {
        const bool is_q = run < q_runs, is_v = run >= q_runs + kv_runs;
        const int r = is_q ? run : (is_v ? run - q_runs - kv_runs : run - q_runs);
        const int head = r / D, o = r - head * D;
        T* dst;
        int from = -1;  // place of the element among its projection's; -1: zero
        int in_part = 0;
        if (is_q) {
            dst = q_out + r;
            const int m = head % a.maps, h = head / a.maps;
            in_part = o - m * a.d;
            if (in_part >= 0 && in_part < a.d) from = h * md + o;
        } else {
            dst = kv + ((((page * 2 + (is_v ? 1 : 0)) * a.n_kv + head) * a.page_size + off) * (int64_t)D) + o;
            if (is_v) {
                if (o < a.dv) from = head * a.dv + o;
            } else if (o < md) {
                in_part = o % a.d;
                from = head * md + o;
            }
        }
        float v = 0.f;
        if (from >= 0) {
            const T* src = row + (is_q ? 0 : (is_v ? a.v_col : a.k_col)) + from;
            const float* w = is_q ? a.q_weight : a.k_weight;
            const float rstd = is_q ? q_rstd : k_rstd;
            const bool normed = w != nullptr && !is_v;
            v = to_float(*src);
            if (normed) v = v * rstd * w[from];
            if (!is_v && in_part < a.rot_dim) {
                const int half = a.rot_dim >> 1;
                const bool second = a.interleaved ? (in_part & 1) != 0 : in_part >= half;
                const int to = a.interleaved ? (second ? -1 : 1) : (second ? -half : half);
                const int i = a.interleaved ? in_part >> 1 : (second ? in_part - half : in_part);
                float other = to_float(src[to]);
                if (normed) other = other * rstd * w[from + to];
                // (u, v) -> (u c - v s, v c + u s)
                v = __fadd_rn(__fmul_rn(v, cos_s[i]), __fmul_rn(second ? other : -other, sin_s[i]));
            }
        }
        *dst = from_float<T>(v);
    }
}

// bfloat16 in runs of 8 elements (16 bytes): a block per token (without a norm the runs of a token may be spread over
// blocks along y), R runs a thread, read once: a run's source is in registers before the angles and the sums of squares
// are formed, and every source run serves exactly one run of the queries or keys, so the sums come from the same loads.
template <int R>
__global__ void __launch_bounds__(1024) heads_to_pages_bf16x8_kernel(const HeadsArgs a, unsigned per_head_inverse) {
    pdl_launch_dependents();
    __shared__ float cos_s[128], sin_s[128], scratch[2][32];
    const int t = blockIdx.x, D = a.D, md = a.maps * a.d, per_head = D / 8;
    const int q_runs = a.n_q * a.maps * per_head, kv_runs = a.n_kv * per_head, runs = q_runs + 2 * kv_runs;
    const int run0 = blockIdx.y * blockDim.x * R + threadIdx.x;
    int from[R], head_of[R], at[R];  // source (place in the row; -1: zeros), output head, first element in it
#pragma unroll
    for (int k = 0; k < R; ++k) {
        const int run = run0 + k * blockDim.x;
        const bool is_q = run < q_runs, is_v = run >= q_runs + kv_runs;
        const int r = is_q ? run : (is_v ? run - q_runs - kv_runs : run - q_runs);
        const int head = (int)__umulhi((unsigned)r, per_head_inverse), o = (r - head * per_head) * 8;
        head_of[k] = head;
        at[k] = o;
        from[k] = -1;
        if (run < runs) {
            if (is_q) {
                const int m = a.maps == 1 ? 0 : (head & 1), h = a.maps == 1 ? head : head >> 1, in_part = o - m * a.d;
                if (in_part >= 0 && in_part < a.d) from[k] = h * md + o;
            } else if (is_v) {
                if (o < a.dv) from[k] = a.v_col + head * a.dv + o;
            } else if (o < md) {
                from[k] = a.k_col + head * md + o;
            }
        }
    }
    pdl_wait();
    const bf16* row = reinterpret_cast<const bf16*>(a.rows) + (int64_t)t * a.row_stride;
    uint4 raw[R];
#pragma unroll
    for (int k = 0; k < R; ++k) raw[k] = from[k] >= 0 ? *reinterpret_cast<const uint4*>(row + from[k]) : make_uint4(0u, 0u, 0u, 0u);
    const float pos = (float)a.positions[t];
    int64_t slot = (a.slots && a.kv) ? (int64_t)a.slots[t] : -1;
    for (int i = threadIdx.x; i < a.rot_dim / 2; i += blockDim.x) sincosf(__fmul_rn(pos, a.inv_freq[i]), &sin_s[i], &cos_s[i]);
    if (slot >= a.pool_slots) {
        if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(a.err, SS_ERR_SLOT_RANGE);
        slot = -1;
    }
    float q_rstd = 1.f, k_rstd = 1.f;
    if (a.q_weight) {
        float sq = 0.f, sk = 0.f;
#pragma unroll
        for (int k = 0; k < R; ++k) {
            const int run = run0 + k * blockDim.x;
            if (run >= q_runs + kv_runs) continue;
            float v[8], s = 0.f;
            unpack8(raw[k], v);
#pragma unroll
            for (int e = 0; e < 8; ++e) s = fmaf(v[e], v[e], s);
            if (run < q_runs) sq += s; else sk += s;
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
        if (lane == 0) { scratch[0][warp] = sq; scratch[1][warp] = sk; }
        __syncthreads();
        q_rstd = 1.0f / sqrtf(warp_sum(lane < n_warps ? scratch[0][lane] : 0.f) / (float)(a.n_q * md) + a.eps);
        k_rstd = 1.0f / sqrtf(warp_sum(lane < n_warps ? scratch[1][lane] : 0.f) / (float)(a.n_kv * md) + a.eps);
    } else {
        __syncthreads();
    }
    const int page_size = a.page_size, page = slot >= 0 ? (int)slot / page_size : 0, off = slot >= 0 ? (int)slot - page * page_size : 0;
#pragma unroll
    for (int k = 0; k < R; ++k) {
        const int run = run0 + k * blockDim.x;
        const bool is_q = run < q_runs, is_v = run >= q_runs + kv_runs;
        if (run >= runs || (!is_q && slot < 0)) continue;
        bf16* dst;
        if (is_q) dst = reinterpret_cast<bf16*>(a.q_out) + (int64_t)t * a.n_q * a.maps * D + run * 8;
        else dst = reinterpret_cast<bf16*>(a.kv) + ((((int64_t)page * 2 + (is_v ? 1 : 0)) * a.n_kv + head_of[k]) * page_size + off) * D + at[k];
        const int second = a.maps == 2 && (is_q ? (head_of[k] & 1) : at[k] >= a.d) ? a.d : 0, in_part = at[k] - second;
        const bool turned = in_part < a.rot_dim;
        if (from[k] < 0 || is_v || (!a.q_weight && !turned)) {
            *reinterpret_cast<uint4*>(dst) = raw[k];
            continue;
        }
        float v[8];
        unpack8(raw[k], v);
        if (a.q_weight) {
            float w8[8];
            load8f(is_q ? a.q_weight + from[k] : a.k_weight + from[k] - a.k_col, w8);
            const float rstd = is_q ? q_rstd : k_rstd;
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = v[e] * rstd * w8[e];
        }
        if (turned) {
#pragma unroll
            for (int e = 0; e < 8; e += 2) {
                if (in_part + e < a.rot_dim) {
                    const int i = (in_part + e) >> 1;
                    const float c = cos_s[i], s = sin_s[i], x = v[e], y = v[e + 1];
                    v[e] = __fadd_rn(__fmul_rn(x, c), __fmul_rn(-y, s));
                    v[e + 1] = __fadd_rn(__fmul_rn(y, c), __fmul_rn(x, s));
                }
            }
        }
        *reinterpret_cast<uint4*>(dst) = pack8(v);
    }
}

extern "C" int ss_heads_to_pages(const void* rows, int64_t row_stride, const int32_t* positions, const int32_t* slots,
                                 const float* inv_freq, const float* q_weight, const float* k_weight, void* q_out, void* kv,
                                 int n_tokens, int n_q, int n_kv, int maps, int d, int dv, int D, int k_col, int v_col,
                                 int rot_dim, int interleaved, float eps, int page_size, int64_t num_pages, int dtype, int* err,
                                 cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n_q < 1 || n_kv < 0 || (maps != 1 && maps != 2) || d < 1 || dv < 1 || D < 16 || D % 8 != 0 || maps * d > D || dv > D || rot_dim < 0 ||
        rot_dim > d || rot_dim % 2 || rot_dim > 256 || (rot_dim > 0 && !inv_freq) || (!q_weight != !k_weight && n_kv > 0) || page_size < 1)
        return (int)cudaErrorInvalidValue;
    HeadsArgs a;
    a.rows = rows; a.row_stride = row_stride; a.positions = positions; a.slots = slots; a.inv_freq = inv_freq;
    a.q_weight = q_weight; a.k_weight = k_weight; a.q_out = q_out; a.kv = kv; a.n_q = n_q; a.n_kv = n_kv; a.maps = maps;
    a.d = d; a.dv = dv; a.D = D; a.k_col = k_col; a.v_col = v_col; a.rot_dim = rot_dim; a.interleaved = interleaved;
    a.page_size = page_size; a.eps = eps; a.pool_slots = num_pages * page_size; a.err = err;
    if (a.pool_slots > 0x7fffffff) return (int)cudaErrorInvalidValue;  // slots are 32-bit
    const bool wide = dtype == SS_BF16 && (interleaved || rot_dim == 0) && d % 8 == 0 && dv % 8 == 0 && k_col % 8 == 0 &&
                      v_col % 8 == 0 && row_stride % 8 == 0 && ((uintptr_t)rows & 15) == 0 && ((uintptr_t)q_out & 15) == 0 &&
                      ((uintptr_t)kv & 15) == 0 && ((uintptr_t)q_weight & 15) == 0 && ((uintptr_t)k_weight & 15) == 0;
    const int runs = (n_q * maps + 2 * n_kv) * (D / 8);
    // few tokens want a short chain per thread, many tokens several loads in flight per thread and several blocks an SM
    const bool many = n_tokens >= 2 * ss_sm_count();
    if (wide && runs <= 4 * 1024) {
        const unsigned inverse = (unsigned)((((uint64_t)1 << 32) + D / 8 - 1) / (D / 8));  // exact for the small numbers here (D >= 16)
        if (!q_weight) {  // nothing is summed over the token: its runs over as many blocks as keep one run a thread
            const int threads = runs >= 256 ? 256 : 128;
            if (many && runs > threads)
                ss_launch(heads_to_pages_bf16x8_kernel<2>, dim3(n_tokens, (runs + 2 * threads - 1) / (2 * threads)), dim3(threads), 0, stream, a, inverse);
            else
                ss_launch(heads_to_pages_bf16x8_kernel<1>, dim3(n_tokens, (runs + threads - 1) / threads), dim3(threads), 0, stream, a, inverse);
        } else {
            const int r = runs <= 1024 && !many ? 1 : (runs <= 512 || (runs <= 2048 && !many) ? 2 : 4);
            const int threads = ((runs + r - 1) / r + 31) / 32 * 32;
            if (r == 1) ss_launch(heads_to_pages_bf16x8_kernel<1>, dim3(n_tokens), dim3(threads), 0, stream, a, inverse);
            else if (r == 2) ss_launch(heads_to_pages_bf16x8_kernel<2>, dim3(n_tokens), dim3(threads), 0, stream, a, inverse);
            else ss_launch(heads_to_pages_bf16x8_kernel<4>, dim3(n_tokens), dim3(threads), 0, stream, a, inverse);
        }
    } else if (dtype == SS_BF16) {
        ss_launch(heads_to_pages_kernel<bf16>, dim3(n_tokens), dim3(256), 0, stream, a);
    } else {
        ss_launch(heads_to_pages_kernel<float>, dim3(n_tokens), dim3(256), 0, stream, a);
    }
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- the two maps of differential heads
//
// x: float32 [token][2 * heads][D], maps 2h and 2h + 1 of head h.  out [token][heads * dv]: with o = x_2h - lam * x_2h+1
// over the first dv elements, o * mult / sqrt(mean(o^2) + eps).  A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
diff_combine_kernel(const float* __restrict__ x, T* __restrict__ out, int64_t pairs, int D, int dv, float lam, float mult, float eps) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const int64_t p = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (p >= pairs) return;
    const float* x1 = x + p * 2 * D;
    constexpr int EPL = 8;  // dv is at most 256
    float o[EPL];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < EPL; ++c) {
        const int e = lane + 32 * c;
        o[c] = e < dv ? x1[e] - lam * x1[D + e] : 0.f;
        ss = fmaf(o[c], o[c], ss);
    }
    const float f = mult / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll
    for (int c = 0; c < EPL; ++c) {
        const int e = lane + 32 * c;
        if (e < dv) out[p * dv + e] = from_float<T>(o[c] * f);
    }
}

extern "C" int ss_diff_combine(const float* x, void* out, int64_t n_tokens, int heads, int D, int dv, float lam, float mult,
                               float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (heads < 1 || dv < 1 || dv > D || dv > 256) return (int)cudaErrorInvalidValue;
    const int64_t pairs = n_tokens * heads;
    const int warps = pairs >= 8 * ss_sm_count() ? 8 : 2;
    const dim3 grid((unsigned)((pairs + warps - 1) / warps)), block(warps * 32);
    if (dtype == SS_BF16) ss_launch(diff_combine_kernel<bf16>, grid, block, 0, stream, x, (bf16*)out, pairs, D, dv, lam, mult, eps);
    else ss_launch(diff_combine_kernel<float>, grid, block, 0, stream, x, (float*)out, pairs, D, dv, lam, mult, eps);
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- a branch's normed output, and the next norm
//
// residual += mult * (y / sqrt(mean(y^2) + eps_y) * w_y) [+ anchor], then out = residual / sqrt(mean(residual^2) + eps) * w.
// y is a branch's output, or one that has not been formed yet (SRC): the weighted sum of two outputs under norms of their
// own, pair_scale * (a / rms(a) * wa + b / rms(b) * wb), or the sum over a token's chosen experts of weight * output (float32
// [token][choice][hidden], or bfloat16 rows in sorted order with the place of every (token, choice)).
// y null: the second half only.  With `rows` only those rows are produced and the stream stays as it is.  Weights are
// float32.  A block per row.  VEC 8: hidden a multiple of 8, at most 8 elements a thread, each row read once; VEC 1: any.
struct BranchArgs {
    float* residual;
    const void* y;
    const float* y_weight;
    const float* anchor;
    const float* weight;
    void* out;
    const int32_t* rows;
    int hidden;
    float mult, y_eps, eps;
    const void* y2;  // SRC_PAIR: y is a, y2 is b
    const float* pair_weight[2];
    float pair_eps, pair_scale;
    const float* term_weight;  // SRC_TERMS: [token][top]
    const int32_t* place;      // y holds sorted rows (of type T); null: y is float32 in order
    int top;
};
enum { SRC_PLAIN = 0, SRC_PAIR = 1, SRC_TERMS = 2 };

// EARLY (few rows): the weights are in registers before the kernels in front are complete; with many rows they are read
// where they are used, which leaves room for more blocks on an SM.
template <typename T, int VEC, bool EARLY, int SRC>
__global__ void __launch_bounds__(1024) branch_norm_kernel(const BranchArgs a) {
    pdl_launch_dependents();
    __shared__ float scratch[4][32];
    const int hidden = a.hidden;
    if constexpr (VEC == 8) {
        const int j = threadIdx.x * 8;
        const bool on = j < hidden;
        float wy[8], w[8];
        if (EARLY && on) {  // weights do not depend on the kernels in front
            load8f(a.weight + j, w);
            if (a.y) load8f(a.y_weight + j, wy);
        }
        pdl_wait();
        const int64_t src = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = 0.f;
        if (on) load8f(a.residual + src * hidden + j, v);
        if (a.y) {
            float y[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) y[e] = 0.f;
            float ss = 0.f;
            auto row8 = [&](const void* p, int64_t row, float (&x)[8]) {
                if constexpr (sizeof(T) == 2) unpack8(*reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(p) + row * hidden + j), x);
                else load8f(reinterpret_cast<const float*>(p) + row * hidden + j, x);
            };
            if constexpr (SRC == SRC_PLAIN) {
                if (on) row8(a.y, src, y);
            } else if constexpr (SRC == SRC_PAIR) {
                float b[8], sa = 0.f, sb = 0.f;
#pragma unroll
                for (int e = 0; e < 8; ++e) b[e] = 0.f;
                if (on) {
                    row8(a.y, src, y);
                    row8(a.y2, src, b);
                }
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    sa = fmaf(y[e], y[e], sa);
                    sb = fmaf(b[e], b[e], sb);
                }
                const float fa = a.pair_scale / sqrtf(block_sum_once(sa, scratch[2]) / (float)hidden + a.pair_eps);
                const float fb = a.pair_scale / sqrtf(block_sum_once(sb, scratch[3]) / (float)hidden + a.pair_eps);
                if (on) {
                    float wa[8], wb[8];
                    load8f(a.pair_weight[0] + j, wa);
                    load8f(a.pair_weight[1] + j, wb);
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] = fmaf(y[e] * fa, wa[e], b[e] * fb * wb[e]);
                }
            } else if (on) {
                for (int k = 0; k < a.top; ++k) {
                    const int64_t at = src * a.top + k;
                    float t[8];
                    if (a.place) row8(a.y, a.place[at], t);
                    else load8f(reinterpret_cast<const float*>(a.y) + at * hidden + j, t);
                    const float w = a.term_weight[at];
#pragma unroll
                    for (int e = 0; e < 8; ++e) y[e] = fmaf(w, t[e], y[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(y[e], y[e], ss);
            float anchor[8];
            if (on && a.anchor) load8f(a.anchor + src * hidden + j, anchor);
            const float f = 1.0f / sqrtf(block_sum_once(ss, scratch[0]) / (float)hidden + a.y_eps);
            if (!EARLY && on) load8f(a.y_weight + j, wy);
            if (on) {
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = fmaf(a.mult, y[e] * f * wy[e], v[e]);
                if (a.anchor) {
#pragma unroll
                    for (int e = 0; e < 8; ++e) v[e] += anchor[e];
                }
                if (!a.rows) store8f(a.residual + src * hidden + j, v);
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
        const float f = 1.0f / sqrtf(block_sum_once(ss, scratch[1]) / (float)hidden + a.eps);
        if (!EARLY && on) load8f(a.weight + j, w);
        if (on) {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = v[e] * f * w[e];
            T* out = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * hidden + j;
            if constexpr (sizeof(T) == 2) *reinterpret_cast<uint4*>(out) = pack8(v);
            else store8f(reinterpret_cast<float*>(out), v);
        }
    } else {
        pdl_wait();
        const int64_t src = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
        float* res = a.residual + src * hidden;
        float fa = 0.f, fb = 0.f;
        auto branch = [&](int j) -> float {  // element j of the branch's output
            const T* y = reinterpret_cast<const T*>(a.y);
            if constexpr (SRC == SRC_PLAIN) {
                return to_float(y[src * hidden + j]);
            } else if constexpr (SRC == SRC_PAIR) {
                return fmaf(to_float(y[src * hidden + j]) * fa, a.pair_weight[0][j],
                            to_float(reinterpret_cast<const T*>(a.y2)[src * hidden + j]) * fb * a.pair_weight[1][j]);
            } else {
                float sum = 0.f;
                for (int k = 0; k < a.top; ++k) {
                    const int64_t at = src * a.top + k;
                    const float t = a.place ? to_float(y[(int64_t)a.place[at] * hidden + j]) : reinterpret_cast<const float*>(a.y)[at * hidden + j];
                    sum = fmaf(a.term_weight[at], t, sum);
                }
                return sum;
            }
        };
        if constexpr (SRC == SRC_PAIR) {
            float sa = 0.f, sb = 0.f;
            for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
                const float x = to_float(reinterpret_cast<const T*>(a.y)[src * hidden + j]), z = to_float(reinterpret_cast<const T*>(a.y2)[src * hidden + j]);
                sa = fmaf(x, x, sa);
                sb = fmaf(z, z, sb);
            }
            fa = a.pair_scale / sqrtf(block_sum_once(sa, scratch[2]) / (float)hidden + a.pair_eps);
            fb = a.pair_scale / sqrtf(block_sum_once(sb, scratch[3]) / (float)hidden + a.pair_eps);
        }
        const float* anchor = a.anchor ? a.anchor + src * hidden : nullptr;
        T* out = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * hidden;
        float fy = 0.f;
        if (a.y) {
            float ss = 0.f;
            for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
                const float v = branch(j);
                ss = fmaf(v, v, ss);
            }
            fy = 1.0f / sqrtf(block_sum_once(ss, scratch[0]) / (float)hidden + a.y_eps);
        }
        auto joined = [&](int j) {
            float v = res[j];
            if (a.y) {
                v = fmaf(a.mult, branch(j) * fy * a.y_weight[j], v);
                if (anchor) v += anchor[j];
            }
            return v;
        };
        float ss = 0.f;
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
            const float v = joined(j);
            ss = fmaf(v, v, ss);
        }
        const float f = 1.0f / sqrtf(block_sum_once(ss, scratch[1]) / (float)hidden + a.eps);
        for (int j = threadIdx.x; j < hidden; j += blockDim.x) {  // every thread meets its own elements again
            const float v = joined(j);
            if (a.y && !a.rows) res[j] = v;
            out[j] = from_float<T>(v * f * a.weight[j]);
        }
    }
}

template <int SRC>
static int launch_branch_norm(const BranchArgs& a, int n_rows, int dtype, bool aligned, cudaStream_t stream) {
    const int hidden = a.hidden;
    if (hidden % 8 == 0 && hidden <= 8192 && aligned) {
        const dim3 block((hidden / 8 + 31) / 32 * 32);
        const bool many = n_rows >= 2 * ss_sm_count();
        if (dtype == SS_BF16 && many) ss_launch(branch_norm_kernel<bf16, 8, false, SRC>, dim3(n_rows), block, 0, stream, a);
        else if (dtype == SS_BF16) ss_launch(branch_norm_kernel<bf16, 8, true, SRC>, dim3(n_rows), block, 0, stream, a);
        else ss_launch(branch_norm_kernel<float, 8, true, SRC>, dim3(n_rows), block, 0, stream, a);
    } else {
        const dim3 block(hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128));
        if (dtype == SS_BF16) ss_launch(branch_norm_kernel<bf16, 1, false, SRC>, dim3(n_rows), block, 0, stream, a);
        else ss_launch(branch_norm_kernel<float, 1, false, SRC>, dim3(n_rows), block, 0, stream, a);
    }
    return SS_LAUNCH_CHECK();
}

// y2 with pair_a, pair_b: SRC_PAIR.  term_weight: SRC_TERMS.
extern "C" int ss_branch_norm(float* residual, const void* y, const float* y_weight, float y_eps, float mult, const float* anchor,
                              const float* weight, float eps, void* out, const int32_t* rows, int n_rows, int hidden, int dtype,
                              cudaStream_t stream, const void* y2, const float* pair_a, const float* pair_b, float pair_eps, float pair_scale,
                              const float* term_weight, const int32_t* place, int top) {
    if (n_rows <= 0) return 0;
    if (hidden < 1 || (y && !y_weight) || (!y && anchor) || (y2 && (!y || !pair_a || !pair_b || term_weight)) || (term_weight && (!y || top < 1)))
        return (int)cudaErrorInvalidValue;
    BranchArgs a;
    a.residual = residual; a.y = y; a.y_weight = y_weight; a.anchor = anchor; a.weight = weight; a.out = out; a.rows = rows;
    a.hidden = hidden; a.mult = mult; a.y_eps = y_eps; a.eps = eps;
    a.y2 = y2; a.pair_weight[0] = pair_a; a.pair_weight[1] = pair_b; a.pair_eps = pair_eps; a.pair_scale = pair_scale;
    a.term_weight = term_weight; a.place = place; a.top = top;
    const bool aligned = (((uintptr_t)residual | (uintptr_t)y | (uintptr_t)y_weight | (uintptr_t)anchor | (uintptr_t)weight | (uintptr_t)out |
                           (uintptr_t)y2 | (uintptr_t)pair_a | (uintptr_t)pair_b) & 15) == 0;
    if (y2) return launch_branch_norm<SRC_PAIR>(a, n_rows, dtype, aligned, stream);
    if (term_weight) return launch_branch_norm<SRC_TERMS>(a, n_rows, dtype, aligned, stream);
    return launch_branch_norm<SRC_PLAIN>(a, n_rows, dtype, aligned, stream);
}
