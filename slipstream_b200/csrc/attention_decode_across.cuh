// Split-KV paged decode attention over the values of ALL kv heads, and the mixture of heads behind it: requests that bring
// ONE token, bfloat16, head size 64 or 128, 2 to 8 kv heads of at most 16 query heads, page sizes 8, 16, 32 and 64.
//
// Heads whose softmax weights are mixed before they meet the values (talking heads) need every query head's weights at the
// values of every kv head.  A block per pair of kv heads would read every key and value n_kv times.  Here a block takes a
// slice of a request's keys for all of its kv heads at once, so that every tile of keys and values is fetched once:
//   * a tile is BN keys: their K rows of all n_kv heads and their V rows of the block's `nc` heads (all of them up to four;
//     more than four are shared by blocks along grid.y), moved by TMA into a ring of stages by a producer warp: a box is the
//     rows of a page and a 64-element half for all heads at once, since a box costs the same however large it is (one box per
//     head took 2.4 us for a tile of 64 KB);
//   * a consumer warp has one kv head of keys and up to CPW kv heads of values, and a set of NK of a tile's keys (where there
//     are fewer kv heads than warps several sets share a tile).  Its products are turned over so that the few query heads of
//     a kv head are the narrow side: scores as keys x heads, outputs as head dims x heads (mma.sync m16n8k16; 7 heads fill 7
//     of 8 columns where they would fill 7 of 16 rows), the weights turned by movmatrix in between.
// Nothing is merged here: every (slice, set) leaves its unnormalised sums, maxima and sums of exponentials in scratch memory,
// and talk_merge_kernel, which reads them once, combines the parts, mixes the heads and applies the gate.
//
// Masking and the clearing of value rows behind the newest token as in attention_decode_tma.cuh.  Every mbarrier wait is
// bounded; a wait that gives up sets SS_ERR_WAIT_LIMIT.
#pragma once

#include "attention_mma.cuh"
#include "attention_tc5.cuh"

#define AX_WARPS 8
#define AX_THREADS (32 * (AX_WARPS + 1))
#define AX_TABLE_MAX 512

// How a layer's heads are laid out over a block.
struct AcrossLayout {
    int nh;      // columns of heads in steps of 8
    int nc;      // kv heads of values a block takes
    int cpw;     // kv heads of values a warp takes at most
    int sets;    // warp sets that share a tile's keys
    int bn, nk;  // keys of a tile, and of a set
    int stages;  // 0: the kernel does not take the layer
};

constexpr int across_stage_bytes(int D, int n_kv, const AcrossLayout& y) { return y.bn * (n_kv + y.nc) * D * 2; }
constexpr int across_smem_bytes(int D, int n_kv, const AcrossLayout& y) {
    return 1024 + y.stages * across_stage_bytes(D, n_kv, y) + n_kv * y.nh * 8 * (D + 8) * 2 + 256;
}

static AcrossLayout across_layout(int D, int n_q, int n_kv) {
    AcrossLayout y = {};
    if (n_kv < 2 || n_kv > 8 || n_q % n_kv || n_q / n_kv > 16) return y;
    y.nh = n_q / n_kv > 8 ? 2 : 1;
    y.cpw = y.nh == 1 ? 4 : 2;
    y.nc = n_kv <= 4 ? n_kv : y.cpw;
    y.sets = n_kv == 2 ? 4 : (y.nh == 1 && n_kv <= 4 ? 2 : 1);
    y.bn = n_kv == 2 ? 64 : 32;
    y.nk = y.bn / y.sets;
    for (int st = 4; st >= 2; --st) {
        y.stages = st;
        if (across_smem_bytes(D, n_kv, y) <= 220 * 1024) return y;
    }
    y.stages = 0;
    return y;
}

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
    int n_slices, stages, nc, sets;
    float* part_o;   // [request][slice * sets + set][kv head of values][kv head of keys][D][8 nh], unnormalised
    float* part_ml;  // [request][slice * sets + set][n_q][2]: maximum (in units of log2 e) and sum of exponentials
    int* err;
};

// Tiles a slice takes: an equal share of the request's, but at least 128 keys, since a part costs the combining kernel more
// than that (a request of 1,024 tokens fills 8 slices, whatever the launch has).
__device__ __forceinline__ int across_tiles_per_slice(int tiles, int n_slices, int tile_keys) {
    return max(128 / tile_keys, (tiles + n_slices - 1) / n_slices);
}

__device__ __forceinline__ uint32_t turn_8x8(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

template <int D, int BN, int NK, int NH, int CPW>
__global__ void __launch_bounds__(AX_THREADS, 1)
attn_decode_across(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const AcrossArgs a) {
    pdl_launch_dependents();
    constexpr int KSTR = D + 8, HALVES = D / 64, HEAD = BN * D;  // elements of one head's rows in a tile
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const int G = a.n_kv, per = a.n_q / G, n_slices = a.n_slices, stages = a.stages;
    const int c0 = blockIdx.y * a.nc, nc = min(a.nc, G - c0);  // this block's kv heads of values
    const int stage_elems = (G + a.nc) * HEAD;
    const int rows = min(a.page_size, BN), row_shift = __ffs(rows) - 1;  // keys of a box
    bf16* ring = reinterpret_cast<bf16*>(base);
    bf16* Qs = ring + stages * stage_elems;  // [kv head][8 NH][KSTR]
    uint64_t* full = reinterpret_cast<uint64_t*>(Qs + G * NH * 8 * KSTR);
    uint64_t* empty = full + 4;
    volatile int* gave_up = reinterpret_cast<volatile int*>(empty + 4);
    __shared__ int32_t table_s[AX_TABLE_MAX];

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int slice = blockIdx.x, r = blockIdx.z;
    const int row_q = a.q_start[r], seq_len = a.seq_lens[r], pos = seq_len - 1;
    const int tiles = seq_len > 0 ? (seq_len - 1) / BN + 1 : 0;
    const int each = across_tiles_per_slice(tiles, n_slices, BN);
    const int j_lo = slice * each, j_hi = min(tiles, j_lo + each) - 1, j_last = tiles - 1;
    const bool work = j_lo <= j_hi;
    // consumer warps: key head, run of value heads, warp set
    const int runs = (nc + CPW - 1) / CPW, slots = G * ((a.nc + CPW - 1) / CPW);
    const int set = warp / slots, in_set = warp - set * slots;
    const int ka = in_set % G, cp = in_set / G;
    const bool consumer = warp < AX_WARPS && set < a.sets && cp < runs;
    const int active = a.sets * G * runs;  // consumer warps that use a tile

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
        // ---------------- producer: a lane per box (page, half, keys or values)
        if (work) {
            if (lane == 0) asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
            if (lane == 0) asm volatile("prefetch.tensormap [%0];" ::"l"(&map_v) : "memory");
            const int boxes = BN / rows, total = boxes * HALVES * 2;
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
                if (lane == 0) fa::mbar_expect_tx(&full[st], stage_elems * 2);  // (a box may reach past the last head: what it brings is not read)
                __syncwarp();
                for (int b = lane; b < total; b += 32) {
                    const int h = b % HALVES, p = (b / HALVES) % boxes;
                    const bool keys = b < boxes * HALVES;
                    const int key = j * BN + p * rows, blk = key / a.page_size, off = key - blk * a.page_size;
                    int64_t page = (blk >= b_first && blk <= b_last) ? (int64_t)table.p[blk - table.base] : -1;
                    if (page >= a.num_pages) {
                        atomicOr(a.err, SS_ERR_PAGE_RANGE);
                        page = -1;
                    }
                    if (page < 0) page = spare;
                    const int heads = keys ? G : a.nc;
                    bf16* dst = ring + st * stage_elems + (keys ? 0 : G * HEAD) + (h * BN + p * rows) * heads * 64;
                    const CUtensorMap* map = keys ? &map_k : &map_v;
                    const int z = keys ? (int)((page * 2 + 0) * G) : (int)((page * 2 + 1) * G + c0);
                    if (gridDim.y > 1) fa::tma_load_3d(dst, map, h * 64, off, z, &full[st]);  // the keys are read by several blocks
                    else fa::tma_load_3d_once(dst, map, h * 64, off, z, &full[st], once);
                }
            }
        }
        pdl_wait();
    } else {
        pdl_wait();
        const int part = slice * a.sets + set, n_parts = n_slices * a.sets;
        if (work) {
            // the queries: 8 NH rows per kv head, rows behind its heads are zero
            for (int c = tid; c < G * NH * 8 * (D / 8); c += AX_WARPS * 32) {
                const int row = c / (D / 8), col = (c - row * (D / 8)) * 8, g = row / (NH * 8), hr = row % (NH * 8);
                const bool ok = hr < per;
                cp_async16(Qs + row * KSTR + col, a.q + (int64_t)row_q * a.q_stride + (int64_t)(g * per + (ok ? hr : 0)) * D + col, ok);
            }
            cp_async_commit();
            cp_async_wait<0>();
            asm volatile("bar.sync 1, 256;" ::: "memory");  // the consumer warps
        }
        if (work && consumer) {
            // a thread's heads of column tile t: 8 t + 2 (lane % 4) and the next; its keys lane / 4 and 8 further
            float m[NH][2], l[NH][2], o[CPW][D / 16][NH][4];
#pragma unroll
            for (int t = 0; t < NH; ++t) {
                m[t][0] = m[t][1] = -INFINITY;
                l[t][0] = l[t][1] = 0.f;
            }
#pragma unroll
            for (int c = 0; c < CPW; ++c)
#pragma unroll
                for (int d = 0; d < D / 16; ++d)
#pragma unroll
                    for (int t = 0; t < NH; ++t) o[c][d][t][0] = o[c][d][t][1] = o[c][d][t][2] = o[c][d][t][3] = 0.f;
            const float scale_log2 = a.scale * 1.4426950408889634f;
            const int key_off = set * NK;
            const int v0 = cp * CPW, n_v = min(CPW, nc - v0);
            const bf16* Qa = Qs + ka * NH * 8 * KSTR;
            // where a row of a tile lies: the box's rows of all heads (rows of 128 bytes, 16-byte chunks permuted by the row)
            // behind those of the boxes in front, the second 64 elements behind the whole tile's first
            auto row_at = [&](int row, int heads, int head) { return ((((row >> row_shift) * heads + head) << row_shift) + (row & (rows - 1))) * 64; };
            const int swz = lane & 7;  // (every row a lane addresses is its lane number mod 8)
            int k_row[NK / 16], v_row[NK / 16];
#pragma unroll
            for (int k = 0; k < NK / 16; ++k) {
                k_row[k] = row_at(key_off + k * 16 + (lane & 15), G, ka);
                v_row[k] = row_at(key_off + k * 16 + (lane & 7) + ((lane >> 4) << 3), a.nc, v0);
            }
            const int k_half = G * BN * 64, v_half = a.nc * BN * 64, v_head = rows * 64;
            auto col_at = [&](int col, int half_stride) { return (col >> 6) * half_stride + ((((col >> 3) & 7) ^ swz) << 3); };
            for (int j = j_lo; j <= j_hi; ++j) {
                const int i = j - j_lo, st = i % stages;
                const bool ok = fa::mbar_wait(&full[st], (i / stages) & 1, gave_up);
                const bf16* Ks = ring + st * stage_elems;
                bf16* Vs = ring + st * stage_elems + G * HEAD;
                const int key0 = j * BN + key_off;
                if (ok && key0 <= pos) {
                    if (j == j_last && pos < key0 + NK - 1) {
                        // value rows behind the newest token hold what the page's last owner left; their weights are zero,
                        // but 0 x inf is not: clear them (warps that share these values write the same zeros)
                        const int first = pos + 1 - j * BN, last = key_off + NK;
                        for (int c = lane; c < (last - first) * (D / 8) * n_v; c += 32) {
                            const int v = c / ((last - first) * (D / 8)), rest = c - v * ((last - first) * (D / 8));
                            const int col = (rest % (D / 8)) * 8;  // (a whole row: the order of its chunks does not matter)
                            *reinterpret_cast<uint4*>(Vs + row_at(first + rest / (D / 8), a.nc, v0 + v) + (col >> 6) * v_half + (col & 63)) = make_uint4(0u, 0u, 0u, 0u);
                        }
                        __syncwarp();
                    }
                    float s[NK / 16][NH][4];
                    {
                        float s2[NK / 16][NH][4];  // two chains of products: even and odd steps
#pragma unroll
                        for (int k = 0; k < NK / 16; ++k)
#pragma unroll
                            for (int t = 0; t < NH; ++t)
#pragma unroll
                                for (int e = 0; e < 4; ++e) s[k][t][e] = s2[k][t][e] = 0.f;
#pragma unroll
                        for (int ks = 0; ks < D / 16; ks += 2) {
                            uint32_t q[NH][4];
#pragma unroll
                            for (int t = 0; t < NH; ++t) ldmatrix_x4(q[t], Qa + (t * 8 + (lane & 7)) * KSTR + ks * 16 + ((lane >> 3) << 3));
#pragma unroll
                            for (int k = 0; k < NK / 16; ++k) {
                                uint32_t x[4], y[4];
                                ldmatrix_x4(x, Ks + k_row[k] + col_at(ks * 16 + ((lane >> 4) << 3), k_half));
                                ldmatrix_x4(y, Ks + k_row[k] + col_at((ks + 1) * 16 + ((lane >> 4) << 3), k_half));
#pragma unroll
                                for (int t = 0; t < NH; ++t) {
                                    mma_bf16(s[k][t], x, q[t][0], q[t][1]);
                                    mma_bf16(s2[k][t], y, q[t][2], q[t][3]);
                                }
                            }
                        }
#pragma unroll
                        for (int k = 0; k < NK / 16; ++k)
#pragma unroll
                            for (int t = 0; t < NH; ++t)
#pragma unroll
                                for (int e = 0; e < 4; ++e) {
                                    const int key = key0 + k * 16 + (lane >> 2) + (e >> 1) * 8;
                                    s[k][t][e] = key <= pos ? (s[k][t][e] + s2[k][t][e]) * scale_log2 : -INFINITY;
                                }
                    }
                    bool moved = false;
                    float alpha[NH][2];
#pragma unroll
                    for (int t = 0; t < NH; ++t)
#pragma unroll
                        for (int b = 0; b < 2; ++b) {
                            float mx = m[t][b];
#pragma unroll
                            for (int k = 0; k < NK / 16; ++k) mx = fmaxf(mx, fmaxf(s[k][t][b], s[k][t][2 + b]));
                            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 4));
                            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 8));
                            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));  // finite: the set's first key is seen
                            alpha[t][b] = fast_exp2(m[t][b] - mx);
                            moved |= mx != m[t][b];
                            m[t][b] = mx;
                            l[t][b] *= alpha[t][b];
                        }
                    uint32_t p[NK / 16][NH][2];  // the weights as the second product reads them: keys by pairs, heads
#pragma unroll
                    for (int k = 0; k < NK / 16; ++k)
#pragma unroll
                        for (int t = 0; t < NH; ++t) {
#pragma unroll
                            for (int e = 0; e < 4; ++e) {
                                s[k][t][e] = fast_exp2(s[k][t][e] - m[t][e & 1]);
                                l[t][e & 1] += s[k][t][e];
                            }
                            p[k][t][0] = turn_8x8(pack_bf16(s[k][t][0], s[k][t][1]));
                            p[k][t][1] = turn_8x8(pack_bf16(s[k][t][2], s[k][t][3]));
                        }
                    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                        for (int c = 0; c < CPW; ++c)
#pragma unroll
                            for (int d = 0; d < D / 16; ++d)
#pragma unroll
                                for (int t = 0; t < NH; ++t)
#pragma unroll
                                    for (int e = 0; e < 4; ++e) o[c][d][t][e] *= alpha[t][e & 1];
                    }
#pragma unroll
                    for (int c = 0; c < CPW; ++c) {
                        if (c >= n_v) break;
#pragma unroll
                        for (int k = 0; k < NK / 16; ++k)
#pragma unroll
                            for (int d = 0; d < D / 16; ++d) {
                                uint32_t v[4];
                                ldmatrix_x4_trans(v, Vs + v_row[k] + c * v_head + col_at(d * 16 + (((lane >> 3) & 1) << 3), v_half));
#pragma unroll
                                for (int t = 0; t < NH; ++t) mma_bf16(o[c][d][t], v, p[k][t][0], p[k][t][1]);
                            }
                    }
                }
                __syncwarp();
                if (lane == 0) {
                    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // before the next copy into this stage
                    fa::mbar_arrive(&empty[st]);
                }
            }
            // the part's results (the columns behind the kv head's last query head are not read)
#pragma unroll
            for (int t = 0; t < NH; ++t)
#pragma unroll
                for (int b = 0; b < 2; ++b) {
                    l[t][b] += __shfl_xor_sync(0xffffffffu, l[t][b], 4);
                    l[t][b] += __shfl_xor_sync(0xffffffffu, l[t][b], 8);
                    l[t][b] += __shfl_xor_sync(0xffffffffu, l[t][b], 16);
                    const int hr = t * 8 + (lane & 3) * 2 + b;
                    if (lane < 4 && hr < per && c0 + v0 == 0)
                        *reinterpret_cast<float2*>(a.part_ml + (((int64_t)r * n_parts + part) * a.n_q + ka * per + hr) * 2) = make_float2(m[t][b], l[t][b]);
                }
#pragma unroll
            for (int c = 0; c < CPW; ++c) {
                if (c >= n_v) break;
                float* dst = a.part_o + ((((int64_t)r * n_parts + part) * G + c0 + v0 + c) * G + ka) * D * (NH * 8) + (lane & 3) * 2;
#pragma unroll
                for (int d = 0; d < D / 16; ++d)
#pragma unroll
                    for (int t = 0; t < NH; ++t)
#pragma unroll
                        for (int e = 0; e < 2; ++e)
                            *reinterpret_cast<float2*>(dst + (d * 16 + (lane >> 2) + e * 8) * (NH * 8) + t * 8) = make_float2(o[c][d][t][2 * e], o[c][d][t][2 * e + 1]);
            }
        } else if (!work && consumer && c0 == 0 && cp == 0 && lane < per) {  // an empty slice says so
            *reinterpret_cast<float2*>(a.part_ml + (((int64_t)r * n_parts + part) * a.n_q + ka * per + lane) * 2) = make_float2(-INFINITY, 0.f);
        }
    }
    if (*gave_up && lane == 0) atomicOr(a.err, SS_ERR_WAIT_LIMIT);
}

// ---------------------------------------------------------------- the parts' sums, the mixture of heads, the gate
//
// With w_p(g) = 2^(m_p(g) - max) / sum over the parts of head g, a_g,c = sum_p w_p(g) O_p(g, c):
//   out[r][h] = sigmoid(gate[r][h]) * sum_g table_t[g][h] a_g,c(h),   c(h) = h / per.
// A block takes AM_COLS head dims of one kv head of values of one request.
#define AM_COLS 32
#define AM_THREADS 512
struct TalkMergeArgs {
    const float* part_o;
    const float* part_ml;
    const float* table_t;  // [g][h]
    const bf16* gate;      // rows gate_stride apart, or null
    int64_t gate_stride;
    bf16* out;
    const int32_t* q_start;
    const int32_t* seq_lens;
    int n_q, n_kv, nh, n_parts, n_slices, tile_keys, splits;  // splits: threads that share the parts of an element
};

// float4 items (four heads of one head dim) of a block's columns, and how many threads share each
constexpr int talk_merge_items(int n_kv, int nh) { return n_kv * AM_COLS * nh * 2; }
constexpr int talk_merge_splits(int n_kv, int nh) { return talk_merge_items(n_kv, nh) >= AM_THREADS ? 1 : AM_THREADS / talk_merge_items(n_kv, nh); }

constexpr int talk_merge_smem(int n_q, int n_kv, int nh, int n_parts) {
    const int slots = n_kv * nh * 8, splits = talk_merge_splits(n_kv, nh);
    return (n_parts * slots + splits * slots * (AM_COLS + 1) + n_q * (n_q / n_kv)) * 4;
}

template <int D, int NH>
__global__ void __launch_bounds__(AM_THREADS, 2)
talk_merge_kernel(const TalkMergeArgs a) {
    extern __shared__ __align__(16) float am_smem[];
    constexpr int wide = NH * 8;
    const int slots = a.n_kv * wide;                 // heads with the padding of every kv head
    float* W = am_smem;                              // [n_parts][slots]: weights of the parts
    float* A = W + a.n_parts * slots;                // [splits][slots][AM_COLS + 1]
    float* T = A + a.splits * slots * (AM_COLS + 1); // [n_q][per]: the mixtures of this kv head's query heads
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c = blockIdx.x / (D / AM_COLS), d0 = (blockIdx.x % (D / AM_COLS)) * AM_COLS, r = blockIdx.y;
    const int seq_len = a.seq_lens[r], row = a.q_start[r];
    const int per = a.n_q / a.n_kv;
    // the parts that hold keys: those of the first slices (as the kernel in front cut them)
    const int tiles = seq_len > 0 ? (seq_len - 1) / a.tile_keys + 1 : 0, each = across_tiles_per_slice(tiles, a.n_slices, a.tile_keys);
    const int parts = (tiles + each - 1) / each * (a.n_parts / a.n_slices);
    for (int g = warp; g < a.n_q; g += AM_THREADS / 32)  // constants of the layer: before the kernel in front is complete
        if (lane < per) T[g * per + lane] = a.table_t[g * a.n_q + c * per + lane];
    pdl_wait();
    if (seq_len <= 0) return;
    float gate = 0.f;  // of this thread's first output
    if (a.gate && tid < per * AM_COLS) gate = to_float(a.gate[row * a.gate_stride + (int64_t)(c * per + tid / AM_COLS) * D + d0 + tid % AM_COLS]);
    // sixteen lanes per head: the weights of its parts
    const int l16 = lane & 15;
    for (int s = tid >> 4; s < (slots + 1) / 2 * 2; s += AM_THREADS / 16) {
        const int hr = s % wide, g = s / wide * per + hr;
        const bool on = s < slots && hr < per;
        const float2* ml = reinterpret_cast<const float2*>(a.part_ml) + r * a.n_parts * a.n_q + g;
        float mx = -INFINITY, den = 0.f;
        float2 v[4];
        for (int p0 = 0; p0 < parts; p0 += 64) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int p = p0 + l16 + 16 * i;
                v[i] = on && p < parts ? __ldcg(ml + p * a.n_q) : make_float2(-INFINITY, 0.f);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) mx = fmaxf(mx, v[i].x);
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        for (int p0 = 0; p0 < parts; p0 += 64) {
            if (parts > 64) {  // (up to 64 parts are still in registers)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int p = p0 + l16 + 16 * i;
                    v[i] = on && p < parts ? __ldcg(ml + p * a.n_q) : make_float2(-INFINITY, 0.f);
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int p = p0 + l16 + 16 * i;
                const float e = v[i].x == -INFINITY ? 0.f : exp2f(v[i].x - mx);
                den = fmaf(e, v[i].y, den);
                if (s < slots && p < parts) W[p * slots + s] = e;
            }
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) den += __shfl_xor_sync(0xffffffffu, den, o);
        const float inv = den > 0.f ? 1.f / den : 0.f;
        if (s < slots)
            for (int p = l16; p < parts; p += 16) W[p * slots + s] *= inv;
    }
    __syncthreads();
    const int64_t head_stride = (int64_t)D * wide, part_stride = (int64_t)a.n_kv * a.n_kv * head_stride;
    const float* o = a.part_o + (int64_t)r * a.n_parts * part_stride + (int64_t)c * a.n_kv * head_stride + (int64_t)d0 * wide;
    constexpr int run4 = wide / 4, unit = AM_COLS * run4;  // float4 items of a kv head of keys
    for (int u = tid / unit; u < a.n_kv * a.splits; u += AM_THREADS / unit) {
        const int sp = u / a.n_kv, ka = u - sp * a.n_kv, at = tid % unit;
        const int d = at / run4, s0 = ka * wide + (at % run4) * 4;
        const float* src = o + ka * head_stride + at * 4;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int p = sp; p < parts; p += a.splits) {
            const float4 w = *reinterpret_cast<const float4*>(W + p * slots + s0);
            const float4 v = __ldcg(reinterpret_cast<const float4*>(src + p * part_stride));
            acc.x = fmaf(w.x, v.x, acc.x); acc.y = fmaf(w.y, v.y, acc.y); acc.z = fmaf(w.z, v.z, acc.z); acc.w = fmaf(w.w, v.w, acc.w);
        }
        float* dst = A + (sp * slots + s0) * (AM_COLS + 1) + d;
        dst[0] = acc.x;
        dst[AM_COLS + 1] = acc.y;
        dst[2 * (AM_COLS + 1)] = acc.z;
        dst[3 * (AM_COLS + 1)] = acc.w;
    }
    __syncthreads();
    for (int i = tid; i < per * AM_COLS; i += AM_THREADS) {
        const int hr = i / AM_COLS, d = i % AM_COLS;
        float v = 0.f;
        for (int ka = 0; ka < a.n_kv; ++ka)
            for (int sp = 0; sp < a.splits; ++sp) {
                const float* x = A + (sp * slots + ka * wide) * (AM_COLS + 1) + d;
                const float* t = T + ka * per * per + hr;
#pragma unroll 8
                for (int k = 0; k < per; ++k) v = fmaf(t[k * per], x[k * (AM_COLS + 1)], v);
            }
        const int64_t col = (int64_t)(c * per + hr) * D + d0 + d;
        if (a.gate) v = gated<true>(v, i == tid ? gate : to_float(a.gate[row * a.gate_stride + col]));
        a.out[(int64_t)row * a.n_q * D + col] = __float2bfloat16_rn(v);
    }
}
