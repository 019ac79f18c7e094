// Split-KV paged decode attention over the values of ALL kv heads, and the mixture of heads behind it: requests that bring
// ONE token, bfloat16, head size 64 or 128, 2 to 8 kv heads of at most 16 query heads, page sizes 8, 16, 32 and 64.
//
// Heads whose softmax weights are mixed before they meet the values (talking heads) need every query head's weights at the
// values of every kv head.  A block per pair of kv heads would read every key and value n_kv times.  Here a block takes a
// slice of a request's keys for all of its kv heads at once, so that every tile of keys and values is fetched once:
//   * a tile is AX_BN keys: their K rows of all n_kv heads and their V rows of the block's `nc` heads (all of them up to four;
//     more than four are shared by blocks along grid.y), moved by TMA, one box per page, head and 64-element half, into a ring;
//   * a consumer warp has one kv head of keys (whose query heads are the 16 rows of its products) and AX_CPW = 2 kv heads of
//     values: scores once, online softmax in float32, two products with values (mma.sync m16n8k16).  With two kv heads the
//     eight warps are four such sets, a 16-key part of each 64-key tile each.
// Nothing is merged here: every (slice, part) leaves its unnormalised sums, maxima and sums of exponentials in scratch memory,
// and talk_merge_kernel, which reads them once, combines the parts, mixes the heads and applies the gate.
//
// Masking and the clearing of value rows behind the newest token as in attention_decode_tma.cuh.  Every mbarrier wait is
// bounded; a wait that gives up sets SS_ERR_WAIT_LIMIT.
#pragma once

#include "attention_mma.cuh"
#include "attention_tc5.cuh"

#define AX_WARPS 8
#define AX_THREADS (32 * (AX_WARPS + 1))
#define AX_CPW 2
#define AX_TABLE_MAX 512

struct AcrossArgs {
    const bf16* q;
    int64_t q_stride;
    const int32_t* block_tables;
    int max_blocks;
    const int32_t* q_start;
    const int32_t* seq_lens;
    int n_q, n_kv, page_size;
    int64_t num_pages;
    float scale;
    int n_slices, stages, nc, sets;  // nc: kv heads of values a block takes; sets: warp sets that share a tile's keys
    float* part_o;   // [request][slice * sets + set][n_kv (values)][n_q][D], unnormalised
    float* part_ml;  // [request][slice * sets + set][n_q][2]: maximum (in units of log2 e) and sum of exponentials
    int* err;
};

// keys of a tile: 16 per warp set with four sets, else 32
__host__ __device__ constexpr int across_tile_keys(int sets) { return sets == 4 ? 64 : 32; }
constexpr int across_stage_bytes(int D, int n_kv, int nc, int sets) { return across_tile_keys(sets) * (n_kv + nc) * D * 2; }
constexpr int across_smem_bytes(int D, int n_kv, int stage_bytes, int stages) {
    return 1024 + stages * stage_bytes + n_kv * 16 * (D + 8) * 2 + 256;
}

// BN: keys of a tile.  NK: keys of a tile a warp set takes.
template <int D, int BN, int NK>
__global__ void __launch_bounds__(AX_THREADS, 1)
attn_decode_across(const __grid_constant__ CUtensorMap map_kv, const AcrossArgs a) {
    pdl_launch_dependents();
    constexpr int KSTR = D + 8, HALVES = D / 64, HEAD = BN * D;  // elements of one head's rows in a tile
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const int G = a.n_kv, per = a.n_q / G, n_slices = a.n_slices, stages = a.stages;
    const int c0 = blockIdx.y * a.nc, nc = min(a.nc, G - c0);  // this block's kv heads of values
    const int stage_elems = (G + a.nc) * HEAD;
    bf16* ring = reinterpret_cast<bf16*>(base);
    bf16* Qs = ring + stages * stage_elems;  // [kv head][16][KSTR]
    uint64_t* full = reinterpret_cast<uint64_t*>(Qs + G * 16 * KSTR);
    uint64_t* empty = full + 4;
    volatile int* gave_up = reinterpret_cast<volatile int*>(empty + 4);
    __shared__ int32_t table_s[AX_TABLE_MAX];

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slice = blockIdx.x, r = blockIdx.z;
    const int row_q = a.q_start[r], seq_len = a.seq_lens[r], pos = seq_len - 1;
    const int tiles = seq_len > 0 ? (seq_len - 1) / BN + 1 : 0;
    const int each = (tiles + n_slices - 1) / n_slices;
    const int j_lo = slice * each, j_hi = min(tiles, j_lo + each) - 1, j_last = tiles - 1;
    const bool work = j_lo <= j_hi;
    // consumer warps: key head, pair of value heads, warp set
    const int pairs = (nc + AX_CPW - 1) / AX_CPW, slots = G * ((a.nc + AX_CPW - 1) / AX_CPW);
    const int set = warp / slots, in_set = warp - set * slots;
    const int ka = in_set % G, cp = in_set / G;
    const bool consumer = warp < AX_WARPS && set < a.sets && cp < pairs;
    const int active = a.sets * G * pairs;  // consumer warps that use a tile

    if (tid == 0) {
        for (int s = 0; s < stages; ++s) { fa::mbar_init(&full[s], 1); fa::mbar_init(&empty[s], active); }
        *gave_up = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    TableRef table;
    table.p = a.block_tables; table.base = 0; table.shift = -1;
    if (work)
        table = stage_table(table_s, a.block_tables + (int64_t)r * a.max_blocks, j_lo * BN, min(pos, j_hi * BN + BN - 1), a.page_size, AX_TABLE_MAX);
    __syncthreads();

    if (warp == AX_WARPS) {
        // ---------------- producer: a lane per box (page, half, head)
        if (work) {
            if (lane == 0) asm volatile("prefetch.tensormap [%0];" ::"l"(&map_kv) : "memory");
            const int rows = min(a.page_size, BN), boxes = BN / rows, total = boxes * HALVES * (G + nc);
            const int b_first = j_lo * BN / a.page_size, b_last = min(pos, j_hi * BN + BN - 1) / a.page_size;
            int64_t spare = table.p[b_first - table.base];  // a page of this request, for blocks that have none
            if (spare < 0 || spare >= a.num_pages) {
                if (lane == 0) atomicOr(a.err, SS_ERR_PAGE_RANGE);
                spare = 0;
            }
            const uint64_t once = fa::l2_evict_first_policy();
            bool waited = false, ok = true;
            for (int j = j_lo; j <= j_hi && ok; ++j) {
                const int i = j - j_lo, st = i % stages;
                if (i >= stages) ok = __all_sync(0xffffffffu, fa::mbar_wait(&empty[st], (i / stages - 1) & 1, gave_up));
                if (!ok) break;
                if (j == j_last && !waited) {
                    pdl_wait();  // the newest key and value are written by the kernel before this one
                    waited = true;
                }
                if (lane == 0) fa::mbar_expect_tx(&full[st], (G + nc) * HEAD * 2);
                __syncwarp();
                for (int b = lane; b < total; b += 32) {
                    const int h = b % HALVES, p = (b / HALVES) % boxes, head = b / (HALVES * boxes);
                    const int key = j * BN + p * rows, blk = key / a.page_size, off = key - blk * a.page_size;
                    int64_t page = (blk >= b_first && blk <= b_last) ? (int64_t)table.p[blk - table.base] : -1;
                    if (page >= a.num_pages) {
                        atomicOr(a.err, SS_ERR_PAGE_RANGE);
                        page = -1;
                    }
                    if (page < 0) page = spare;
                    bf16* dst = ring + st * stage_elems + head * HEAD + h * (BN * 64) + p * rows * 64;
                    const int z = head < G ? (int)((page * 2 + 0) * G + head) : (int)((page * 2 + 1) * G + c0 + head - G);
                    if (gridDim.y > 1) fa::tma_load_3d(dst, &map_kv, h * 64, off, z, &full[st]);  // the keys are read by several blocks
                    else fa::tma_load_3d_once(dst, &map_kv, h * 64, off, z, &full[st], once);
                }
            }
        }
        pdl_wait();
    } else {
        pdl_wait();
        const int part = slice * a.sets + set, n_parts = n_slices * a.sets;
        float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
        float o[AX_CPW][D / 8][4];
#pragma unroll
        for (int c = 0; c < AX_CPW; ++c)
#pragma unroll
            for (int d = 0; d < D / 8; ++d) o[c][d][0] = o[c][d][1] = o[c][d][2] = o[c][d][3] = 0.f;
        if (work) {
            // the queries: 16 rows per kv head, rows behind its heads are zero
            for (int c = tid; c < G * 16 * (D / 8); c += AX_WARPS * 32) {
                const int row = c / (D / 8), col = (c - row * (D / 8)) * 8, g = row >> 4, hr = row & 15;
                const bool ok = hr < per;
                cp_async16(Qs + row * KSTR + col, a.q + (int64_t)row_q * a.q_stride + (int64_t)(g * per + (ok ? hr : 0)) * D + col, ok);
            }
            cp_async_commit();
            cp_async_wait<0>();
            asm volatile("bar.sync 1, 256;" ::: "memory");  // the consumer warps
        }
        if (work && consumer) {
            const float scale_log2 = a.scale * 1.4426950408889634f;
            const int key_off = set * NK;
            const int v0 = cp * AX_CPW, n_v = min(AX_CPW, nc - v0);
            const bf16* Qa = Qs + ka * 16 * KSTR;
            // a row of a head in a tile: halves of 64 elements, BN rows of 128 bytes each, 16-byte chunks permuted by the row
            auto at = [](const bf16* tile, int row, int col) { return tile + (col >> 6) * (BN * 64) + row * 64 + ((((col >> 3) & 7) ^ (row & 7)) << 3); };
            for (int j = j_lo; j <= j_hi; ++j) {
                const int i = j - j_lo, st = i % stages;
                const bool ok = fa::mbar_wait(&full[st], (i / stages) & 1, gave_up);
                const bf16* Ks = ring + st * stage_elems + ka * HEAD;
                bf16* Vs = ring + st * stage_elems + (G + v0) * HEAD;
                const int key0 = j * BN + key_off;
                if (ok && key0 <= pos) {
                    if (j == j_last && pos < key0 + NK - 1) {
                        // value rows behind the newest token hold what the page's last owner left; their weights are zero,
                        // but 0 x inf is not: clear them (warps that share these values write the same zeros)
                        const int first = pos + 1 - j * BN, last = key_off + NK;
                        for (int c = lane; c < (last - first) * (D / 8) * n_v; c += 32) {
                            const int v = c / ((last - first) * (D / 8)), rest = c - v * ((last - first) * (D / 8));
                            *reinterpret_cast<uint4*>(const_cast<bf16*>(at(Vs + v * HEAD, first + rest / (D / 8), (rest % (D / 8)) * 8))) = make_uint4(0u, 0u, 0u, 0u);
                        }
                        __syncwarp();
                    }
                    float s[NK / 8][4];
#pragma unroll
                    for (int n = 0; n < NK / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
                    for (int ks = 0; ks < D / 16; ++ks) {
                        uint32_t qf[4];
                        ldmatrix_x4(qf, Qa + (lane & 15) * KSTR + ks * 16 + ((lane >> 4) << 3));
#pragma unroll
                        for (int n = 0; n < NK / 8; n += 2) {
                            uint32_t b[4];
                            ldmatrix_x4(b, at(Ks, key_off + n * 8 + (lane & 7) + ((lane >> 4) << 3), ks * 16 + (((lane >> 3) & 1) << 3)));
                            mma_bf16(s[n], qf, b[0], b[1]);
                            mma_bf16(s[n + 1], qf, b[2], b[3]);
                        }
                    }
                    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
                    for (int n = 0; n < NK / 8; ++n)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int key = key0 + n * 8 + ((lane & 3) << 1) + (e & 1);
                            const float v = key <= pos ? s[n][e] * scale_log2 : -INFINITY;
                            s[n][e] = v;
                            mx[e >> 1] = fmaxf(mx[e >> 1], v);
                        }
                    float alpha[2];
#pragma unroll
                    for (int h = 0; h < 2; ++h) {
                        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
                        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
                        mx[h] = fmaxf(m[h], mx[h]);  // finite: the tile's first key is seen
                        alpha[h] = fast_exp2(m[h] - mx[h]);
                        m[h] = mx[h];
                        l[h] *= alpha[h];
                    }
#pragma unroll
                    for (int n = 0; n < NK / 8; ++n)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            s[n][e] = fast_exp2(s[n][e] - m[e >> 1]);
                            l[e >> 1] += s[n][e];
                        }
                    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
                        for (int c = 0; c < AX_CPW; ++c)
#pragma unroll
                            for (int d = 0; d < D / 8; ++d) {
                                o[c][d][0] *= alpha[0]; o[c][d][1] *= alpha[0];
                                o[c][d][2] *= alpha[1]; o[c][d][3] *= alpha[1];
                            }
                    }
#pragma unroll
                    for (int kk = 0; kk < NK / 16; ++kk) {
                        const uint32_t p[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                               pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                        for (int c = 0; c < AX_CPW; ++c) {
                            if (c >= n_v) break;
#pragma unroll
                            for (int d = 0; d < D / 8; d += 2) {
                                uint32_t b[4];
                                ldmatrix_x4_trans(b, at(Vs + c * HEAD, key_off + kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), d * 8 + ((lane >> 4) << 3)));
                                mma_bf16(o[c][d], p, b[0], b[1]);
                                mma_bf16(o[c][d + 1], p, b[2], b[3]);
                            }
                        }
                    }
                }
                __syncwarp();
                if (lane == 0) {
                    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // before the next copy into this stage
                    fa::mbar_arrive(&empty[st]);
                }
            }
            // the part's results, for the rows that hold a head
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
                l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
                const int row = (lane >> 2) + h * 8;
                if (row >= per) continue;
                const int head = ka * per + row;
                if ((lane & 3) == 0 && c0 + v0 == 0)
                    *reinterpret_cast<float2*>(a.part_ml + (((int64_t)r * n_parts + part) * a.n_q + head) * 2) = make_float2(m[h], l[h]);
#pragma unroll
                for (int c = 0; c < AX_CPW; ++c) {
                    if (c >= n_v) break;
                    float* dst = a.part_o + ((((int64_t)r * n_parts + part) * G + c0 + v0 + c) * a.n_q + head) * D + ((lane & 3) << 1);
#pragma unroll
                    for (int d = 0; d < D / 8; ++d) *reinterpret_cast<float2*>(dst + d * 8) = make_float2(o[c][d][2 * h], o[c][d][2 * h + 1]);
                }
            }
        } else if (consumer && c0 == 0 && cp == 0) {  // an empty slice says so
            const int row = lane;
            if (row < per)
                *reinterpret_cast<float2*>(a.part_ml + (((int64_t)r * n_parts + part) * a.n_q + ka * per + row) * 2) = make_float2(-INFINITY, 0.f);
        }
    }
    if (*gave_up && lane == 0) atomicOr(a.err, SS_ERR_WAIT_LIMIT);
}

// ---------------------------------------------------------------- the parts' sums, the mixture of heads, the gate
//
// With w_p(g) = 2^(m_p(g) - max) / sum over the parts of head g, a_g,c = sum_p w_p(g) O_p(g, c):
//   out[r][h] = sigmoid(gate[r][h]) * sum_g table_t[g][h] a_g,c(h),   c(h) = h / per.
// A block takes AM_COLS columns of one kv head of values of one request.
#define AM_COLS 32
#define AM_THREADS 256
struct TalkMergeArgs {
    const float* part_o;
    const float* part_ml;
    const float* table_t;  // [g][h]
    const bf16* gate;      // rows gate_stride apart, or null
    int64_t gate_stride;
    bf16* out;
    const int32_t* q_start;
    const int32_t* seq_lens;
    int n_q, n_kv, n_parts;
};

template <int D>
__global__ void __launch_bounds__(AM_THREADS)
talk_merge_kernel(const TalkMergeArgs a) {
    extern __shared__ __align__(16) float am_smem[];
    float* A = am_smem;                    // [n_q][AM_COLS]
    float* W = A + a.n_q * AM_COLS;        // [n_q][n_parts]
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c = blockIdx.x / (D / AM_COLS), d0 = (blockIdx.x % (D / AM_COLS)) * AM_COLS, r = blockIdx.y;
    if (a.seq_lens[r] <= 0) return;
    const int per = a.n_q / a.n_kv;
    for (int g = warp; g < a.n_q; g += AM_THREADS / 32) {  // a warp per head: the weights of its parts
        float mx = -INFINITY, den = 0.f;
        for (int p = lane; p < a.n_parts; p += 32) mx = fmaxf(mx, a.part_ml[(((int64_t)r * a.n_parts + p) * a.n_q + g) * 2]);
        mx = warp_max(mx);
        for (int p = lane; p < a.n_parts; p += 32) {
            const float2 ml = *reinterpret_cast<const float2*>(a.part_ml + (((int64_t)r * a.n_parts + p) * a.n_q + g) * 2);
            const float e = ml.x == -INFINITY ? 0.f : exp2f(ml.x - mx);
            W[g * a.n_parts + p] = e;
            den = fmaf(e, ml.y, den);
        }
        den = warp_sum(den);
        const float inv = den > 0.f ? 1.f / den : 0.f;
        __syncwarp();
        for (int p = lane; p < a.n_parts; p += 32) W[g * a.n_parts + p] *= inv;
    }
    __syncthreads();
    const int64_t part_stride = (int64_t)a.n_kv * a.n_q * D;
    const float* o = a.part_o + ((int64_t)r * a.n_parts * a.n_kv + c) * a.n_q * D + d0;
    for (int i = tid; i < a.n_q * (AM_COLS / 4); i += AM_THREADS) {
        const int g = i / (AM_COLS / 4), d = (i % (AM_COLS / 4)) * 4;
        const float* src = o + (int64_t)g * D + d;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int p = 0; p < a.n_parts; ++p) {
            const float w = W[g * a.n_parts + p];
            if (w != 0.f) {  // (an empty part has written nothing)
                const float4 v = __ldcg(reinterpret_cast<const float4*>(src + p * part_stride));
                acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
            }
        }
        *reinterpret_cast<float4*>(A + g * AM_COLS + d) = acc;
    }
    __syncthreads();
    for (int i = tid; i < per * AM_COLS; i += AM_THREADS) {
        const int hr = i / AM_COLS, d = i % AM_COLS, h = c * per + hr;
        float v = 0.f;
#pragma unroll 4
        for (int g = 0; g < a.n_q; ++g) v = fmaf(__ldg(a.table_t + (int64_t)g * a.n_q + h), A[g * AM_COLS + d], v);
        const int64_t col = (int64_t)h * D + d0 + d, row = a.q_start[r];
        if (a.gate) v = gated<true>(v, to_float(a.gate[row * a.gate_stride + col]));
        a.out[row * a.n_q * D + col] = __float2bfloat16_rn(v);
    }
}
