// Attention library for one head size: compiled with -DHEAD_DIM=<multiple of 16>,
// once for each head size a loaded model uses.
#include "attention_simt.cuh"

#ifndef HEAD_DIM
#error "compile with -DHEAD_DIM=<head size>"
#endif
static_assert(HEAD_DIM % 16 == 0 && HEAD_DIM >= 16 && HEAD_DIM <= 256,
              "head sizes are multiples of 16 up to 256");

extern "C" int ss_attn_head_dim() { return HEAD_DIM; }

extern "C" int ss_attn_simt(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                            const void* kv, const int32_t* block_tables, int max_blocks,
                            const int32_t* tile_req, const int32_t* tile_q0, int n_tiles,
                            const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv,
                            int page_size, int64_t num_pages, float scale, int window, int dtype,
                            const void* gate, int* err, cudaStream_t stream, float softcap, const float* sinks, int keep, int across) {
    if (n_tiles <= 0) return 0;
    if (keep < 0 || (keep > 0 && window <= 0) || (across && gate)) return (int)cudaErrorInvalidValue;
    if (dtype == SS_BF16)
        return launch_attn_simt<bf16, HEAD_DIM>(q, q_stride, out, out_stride, kv, block_tables, max_blocks,
                                                tile_req, tile_q0, n_tiles, q_start, seq_lens, n_q, n_kv,
                                                page_size, num_pages, scale, window, gate, err, stream, softcap, sinks, keep, across);
    return launch_attn_simt<float, HEAD_DIM>(q, q_stride, out, out_stride, kv, block_tables, max_blocks,
                                             tile_req, tile_q0, n_tiles, q_start, seq_lens, n_q, n_kv,
                                             page_size, num_pages, scale, window, gate, err, stream, softcap, sinks, keep, across);
}

#include "attention_mma.cuh"

// What the kernels that combine a differential head's two maps ask of a call: an even number of query heads per kv
// head, values of at most the head size in runs of 8, and an output whose rows they can write 16 bytes at a time.
static bool diff_pair_fits(const DiffPair& d, int n_q, int n_kv, int64_t out_stride, const void* out) {
    return !d.on || ((n_q / n_kv) % 2 == 0 && d.dim > 0 && d.dim <= HEAD_DIM && d.dim % 8 == 0 && out_stride % 8 == 0 &&
                     ((uintptr_t)out & 15) == 0);
}

// Most slices a decode call may ask for: the last block of a head block lines up one weight per (head, slice) in
// shared memory, and the launchers' policies never ask for more.
#define SS_DECODE_MAX_SLICES 64

// Prompt portions and mixed batches, bfloat16.  Tiles: 64 rows of (token, head of the group) pairs of one
// request, listed by the host as (request, first row); the grid's second axis is the kv head.
extern "C" int ss_attn_prefill_mma(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                                   const void* kv, const int32_t* block_tables, int max_blocks,
                                   const int32_t* tile_req, const int32_t* tile_row0, int n_tiles,
                                   const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv,
                                   int page_size, int64_t num_pages, float scale, int window, const void* gate, int* err,
                                   cudaStream_t stream, float softcap, const float* sinks, int keep, int out_f32, int diff_on,
                                   float diff_lam, float diff_mult, float diff_eps, int diff_dim, int across) {
    if (n_tiles <= 0) return 0;
    const DiffPair diff = {diff_on, diff_lam, diff_mult, diff_eps, diff_dim};
    if (keep < 0 || (keep > 0 && window <= 0) || !diff_pair_fits(diff, n_q, n_kv, out_stride, out) || (diff_on && (gate || out_f32)) ||
        (out_f32 && gate) || (across && (diff_on || gate)))
        return (int)cudaErrorInvalidValue;
    constexpr int smem = mma_smem_bytes<HEAD_DIM>();
    static SsPerDevice opted;
    if (int rc_smem = ss_opt_in_smem(attn_prefill_mma<HEAD_DIM>, smem, opted)) return rc_smem;
    dim3 grid(n_tiles, across ? n_kv * n_kv : n_kv);
    ss_launch(attn_prefill_mma<HEAD_DIM>, dim3(grid), dim3(MMA_THREADS), smem, stream, 
        (const bf16*)q, q_stride, (bf16*)out, out_stride, (const bf16*)kv, block_tables, max_blocks, tile_req,
        tile_row0, q_start, seq_lens, n_q, n_kv, page_size, num_pages, scale, window, err, (const bf16*)gate, softcap, sinks, keep, out_f32, diff, across);
    return SS_LAUNCH_CHECK();
}

// Requests that bring one token each, bfloat16, split over the keys into n_slices.  part_o
// ([requests][n_q][n_slices][D] float32), part_lse ([requests][n_q][n_slices] float32) and counters (one int
// per request and block of 16 heads of a kv group; zero before the first call, left zero by every call) are
// scratch memory of the caller; they are not touched when n_slices is at most 8.  sinks (here and in the two entry
// points above; float32, one per query head, or null): one more term exp(sinks[h]) in the softmax's denominator.  fused: q points at rows
// [q heads | k heads | v heads] as projected; the kernel rotates queries and the newest key by the request's
// last position (inv_freq: float32 [rot_dim / 2]) and writes the newest key and value to their page.  keep (here and in
// the other entry points): with a window, the request's first keys stay visible.  out_f32: out is float32.
extern "C" int ss_attn_decode_mma(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                                  const void* kv, const int32_t* block_tables, int max_blocks, int n_requests,
                                  const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv,
                                  int page_size, int64_t num_pages, float scale, int window, int n_slices,
                                  const float* inv_freq, int rot_dim, int fused, float* part_o, float* part_lse, int* counters,
                                  const void* gate, int* err, cudaStream_t stream, float softcap, const float* sinks, int keep,
                                  int out_f32, int across) {
    if (keep < 0 || (keep > 0 && window <= 0) || (out_f32 && gate) || (across && (fused || gate))) return (int)cudaErrorInvalidValue;
    if (n_requests <= 0) return 0;
    const int cluster = n_slices >= 2 && n_slices <= 8;  // the slices are combined through shared memory
    if (fused && (rot_dim < 0 || rot_dim > HEAD_DIM || rot_dim % 2 || (rot_dim > 0 && !inv_freq))) return (int)cudaErrorInvalidValue;
    if (n_slices < 1 || n_slices > SS_DECODE_MAX_SLICES) return (int)cudaErrorInvalidValue;
    if (n_slices > 1 && !cluster && (!part_o || !part_lse || !counters)) return (int)cudaErrorInvalidValue;
    constexpr int smem = mma_smem_bytes<HEAD_DIM>(16, DECODE_STAGES);
    static SsPerDevice opted;
    if (int rc_smem = ss_opt_in_smem(attn_decode_mma<HEAD_DIM>, smem, opted)) return rc_smem;
    const int G = n_q / n_kv;
    dim3 grid(n_requests, (across ? n_kv * n_kv : n_kv) * ((G + 15) / 16), n_slices);
    if (cluster)
        ss_launch_cluster(attn_decode_mma<HEAD_DIM>, dim3(grid), dim3(MMA_THREADS), smem, stream, n_slices,
            (const bf16*)q, q_stride, (bf16*)out, out_stride, (const bf16*)kv, block_tables, max_blocks, q_start,
            seq_lens, n_q, n_kv, page_size, num_pages, scale, window, n_slices, 1, inv_freq, rot_dim, fused, part_o, part_lse, counters, err, (const bf16*)gate, softcap, sinks, keep, out_f32, across);
    else
        ss_launch(attn_decode_mma<HEAD_DIM>, dim3(grid), dim3(MMA_THREADS), smem, stream,
            (const bf16*)q, q_stride, (bf16*)out, out_stride, (const bf16*)kv, block_tables, max_blocks, q_start,
            seq_lens, n_q, n_kv, page_size, num_pages, scale, window, n_slices, 0, inv_freq, rot_dim, fused, part_o, part_lse, counters, err, (const bf16*)gate, softcap, sinks, keep, out_f32, across);
    return SS_LAUNCH_CHECK();
}

// ---------------------------------------------------------------- tcgen05 prefill attention (head size 64 or 128)
#if HEAD_DIM == 64 || HEAD_DIM == 128
#include "attention_tc5.cuh"

extern "C" int ss_attn_prefill_tc5_supported() { return 1; }

// q: first query head of row 0 of the stacked [N, q_stride] projection output (n_q heads of HEAD_DIM);
// kv: this layer's pages [num_pages][2][n_kv][page_size][HEAD_DIM].  Tiles: (request, first token) of
// 128 / (n_q / n_kv) consecutive query tokens of one request.  page_size must be a multiple of 8 that divides 64.
extern "C" int ss_attn_prefill_tc5(const void* q, int64_t q_stride, int n_tokens, void* out, int64_t out_stride,
                                   const void* kv, const int32_t* block_tables, int max_blocks,
                                   const int32_t* tile_req, const int32_t* tile_tok0, int n_tiles,
                                   const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv, int page_size,
                                   int64_t num_pages, float scale, int splits, int span, int* err, cudaStream_t stream,
                                   float softcap, const float* sinks, int keep, int out_f32, int diff_on, float diff_lam,
                                   float diff_mult, float diff_eps, int diff_dim, int across) {
    if (n_tiles <= 0) return 0;
    const DiffPair diff = {diff_on, diff_lam, diff_mult, diff_eps, diff_dim};
    if (keep < 0 || (keep > 0 && span <= 0) || !diff_pair_fits(diff, n_q, n_kv, out_stride, out) || (diff_on && (splits != 1 || out_f32 || across)) ||
        (out_f32 && (out_stride % 4 || ((uintptr_t)out & 15))))
        return (int)cudaErrorInvalidValue;
    const int G = n_q / n_kv;
    if (G < 1 || G > 128 || page_size % 8 != 0 || 64 % page_size != 0 || q_stride % 8 != 0) return -3003;
    if (splits != 1 && splits != 2 && splits != 4 && splits != 8) return -3004;
    const int TOK = 128 / G, n_u = across ? n_kv * n_kv : n_kv;
    CUtensorMap map_q, map_kv;
    int rc = fa::make_map3(&map_q, q, HEAD_DIM, (uint64_t)n_q, (uint64_t)n_tokens, (uint64_t)HEAD_DIM * 2,
                           (uint64_t)q_stride * 2, 64, (uint32_t)G, (uint32_t)TOK);
    if (rc) return rc;
    rc = fa::make_map3(&map_kv, kv, HEAD_DIM, (uint64_t)page_size, (uint64_t)num_pages * 2 * n_kv, (uint64_t)HEAD_DIM * 2,
                       (uint64_t)page_size * HEAD_DIM * 2, 64, (uint32_t)page_size, 1);
    if (rc) return rc;
    fa::Args a;
    a.out = (bf16*)out; a.out_stride = out_stride; a.block_tables = block_tables; a.max_blocks = max_blocks;
    a.tile_req = tile_req; a.tile_tok0 = tile_tok0; a.q_start = q_start; a.seq_lens = seq_lens;
    a.n_q = n_q; a.n_kv = n_kv; a.page_size = page_size; a.num_pages = num_pages; a.scale = scale; a.err = err;
    a.span = span; a.softcap = softcap; a.sinks = sinks; a.keep = keep; a.out_f32 = out_f32; a.across = across; a.diff = diff;
    constexpr int smem = fa::smem_bytes<HEAD_DIM>();
    static SsPerDevice opted;
    if (int rc_smem = ss_opt_in_smem(fa::attn_prefill_tc5<HEAD_DIM>, smem, opted)) return rc_smem;
    // splits > 1: the key tiles of every query tile are shared by a thread-block cluster of that many blocks
    if (splits > 1)
        ss_launch_cluster(fa::attn_prefill_tc5<HEAD_DIM>, dim3(n_tiles * n_u, 1, splits), dim3(FA_THREADS), smem, stream, splits, map_q, map_kv, a);
    else
        ss_launch(fa::attn_prefill_tc5<HEAD_DIM>, dim3(n_tiles * n_u), dim3(FA_THREADS), smem, stream, map_q, map_kv, a);
    return SS_LAUNCH_CHECK();
}

#include "attention_decode_tma.cuh"

template <int NS, int FORM>
static int launch_decode_tma(const CUtensorMap& map_kv, const DecodeTmaArgs& a, dim3 grid, int cluster, int smem,
                             cudaStream_t stream) {
    // the most a launch can ask for: 16 heads in a cluster of 7 are 3 x 7 records; the records a block receives from
    // its cluster are sized by the heads it really has
    static SsPerDevice opted;
    if (int rc_smem = ss_opt_in_smem(attn_decode_tma<HEAD_DIM, NS, FORM>, decode_tma_smem_bytes<HEAD_DIM, NS>(24, 8), opted))
        return rc_smem;
    if (cluster > 1)
        ss_launch_cluster(attn_decode_tma<HEAD_DIM, NS, FORM>, dim3(grid), dim3(DT_THREADS), smem, stream, cluster, map_kv, a);
    else
        ss_launch(attn_decode_tma<HEAD_DIM, NS, FORM>, dim3(grid), dim3(DT_THREADS), smem, stream, map_kv, a);
    return SS_LAUNCH_CHECK();
}

// The decode kernel with TMA-fed tiles: arguments as ss_attn_decode_mma; page_size 8, 16, 32 or 64.  stages: 2 or 3
// tiles of keys and values in the ring of a block (see the kernel).
extern "C" int ss_attn_decode_tma(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                                  void* kv, const int32_t* block_tables, int max_blocks, int n_requests,
                                  const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv,
                                  int page_size, int64_t num_pages, float scale, int window, int n_slices,
                                  const float* inv_freq, int rot_dim, int fused, float* part_o,
                                  float* part_lse, int* counters, int stages, const void* gate, int* err, cudaStream_t stream,
                                  float softcap, const float* sinks, int keep, int out_f32, int across) {
    if (n_requests <= 0) return 0;
    if (keep < 0 || (keep > 0 && window <= 0) || (out_f32 && gate) || (across && (fused || gate))) return (int)cudaErrorInvalidValue;
    if (page_size % 8 != 0 || 64 % page_size != 0) return -3003;
    // up to 8 slices: one cluster; a multiple of 8 beyond: clusters of 8 whose results meet in scratch memory;
    // any other count: single blocks and scratch memory
    const int cluster = n_slices <= 8 ? n_slices : (n_slices % 8 == 0 ? 8 : 1);
    if (n_slices < 1 || n_slices > SS_DECODE_MAX_SLICES || (stages != 2 && stages != 3)) return (int)cudaErrorInvalidValue;
    if (n_slices > 8 && (!part_o || !part_lse || !counters)) return (int)cudaErrorInvalidValue;
    if (fused && (rot_dim < 0 || rot_dim > HEAD_DIM || rot_dim % 2 || (rot_dim > 0 && !inv_freq))) return (int)cudaErrorInvalidValue;
    CUtensorMap map_kv;
    int rc = fa::make_map3(&map_kv, kv, HEAD_DIM, (uint64_t)page_size, (uint64_t)num_pages * 2 * n_kv, (uint64_t)HEAD_DIM * 2,
                           (uint64_t)page_size * HEAD_DIM * 2, 64, (uint32_t)page_size, 1);
    if (rc) return rc;
    DecodeTmaArgs a;
    a.q = (const bf16*)q; a.q_stride = q_stride; a.out = (bf16*)out; a.out_stride = out_stride; a.kv = (bf16*)kv;
    a.block_tables = block_tables; a.max_blocks = max_blocks; a.q_start = q_start; a.seq_lens = seq_lens;
    a.n_q = n_q; a.n_kv = n_kv; a.page_size = page_size; a.num_pages = num_pages; a.scale = scale; a.softcap = softcap; a.window = window;
    a.n_slices = n_slices; a.cluster = cluster; a.inv_freq = inv_freq; a.rot_dim = rot_dim; a.fused = fused;
    a.part_o = part_o; a.part_lse = part_lse; a.counters = counters; a.err = err; a.gate = (const bf16*)gate;
    a.sinks = sinks; a.keep = keep; a.out_f32 = out_f32; a.across = across;
    const int G = n_q / n_kv;
    dim3 grid(n_requests, (across ? n_kv * n_kv : n_kv) * ((G + 15) / 16), n_slices);
    // the usual decode step (rotation inside, no window, one cluster, a rotary size in steps of 16) has kernels of its own
    const bool usual = fused && window == 0 && gate == nullptr && sinks == nullptr && !out_f32 && softcap <= 0.f && cluster == n_slices && cluster > 1 && rot_dim > 0 && rot_dim % 16 == 0;
    const int smem3 = decode_tma_smem_bytes<HEAD_DIM, 3>(G < 16 ? G : 16, cluster);
    const int smem2 = decode_tma_smem_bytes<HEAD_DIM, 2>(G < 16 ? G : 16, cluster);
    if (stages == 3 && usual) return launch_decode_tma<3, 1>(map_kv, a, grid, cluster, smem3, stream);
    if (stages == 3) return launch_decode_tma<3, 0>(map_kv, a, grid, cluster, smem3, stream);
    if (usual) return launch_decode_tma<2, 1>(map_kv, a, grid, cluster, smem2, stream);
    return launch_decode_tma<2, 0>(map_kv, a, grid, cluster, smem2, stream);
}

#include "attention_decode_across.cuh"

// What a layer needs of ss_attn_decode_across's scratch: parts per slice (the return value; 0 where the kernel does not take
// the layer) and columns of heads per kv head.
extern "C" int ss_attn_decode_across_sets(int n_q, int n_kv, int page_size, int* head_cols) {
    if (page_size % 8 != 0 || 64 % page_size != 0) return 0;
    const AcrossLayout y = across_layout(HEAD_DIM, n_q, n_kv);
    if (head_cols) *head_cols = y.nh * 8;
    return y.stages ? y.sets : 0;
}

template <int BN, int NK, int NH, int CPW>
static int launch_across(const CUtensorMap& map_k, const CUtensorMap& map_v, const AcrossArgs& a, dim3 grid, int smem, cudaStream_t stream) {
    static SsPerDevice opted;
    if (int rc = ss_opt_in_smem(attn_decode_across<HEAD_DIM, BN, NK, NH, CPW>, 220 * 1024, opted)) return rc;
    ss_launch(attn_decode_across<HEAD_DIM, BN, NK, NH, CPW>, grid, dim3(AX_THREADS), smem, stream, map_k, map_v, a);
    return SS_LAUNCH_CHECK();
}

// A decode step with talking heads.  q: rotated or normed queries, n_q heads of HEAD_DIM a row; part_o (float32
// [requests][parts][n_kv][n_kv][HEAD_DIM][head columns]) and part_ml ([requests][parts][n_q][2]) scratch of the caller, parts =
// n_slices * sets; table_t, gate and out as ss_talk_heads (bfloat16).  Two launches.
extern "C" int ss_attn_decode_across(const void* q, int64_t q_stride, void* out, const void* kv, const int32_t* block_tables, int max_blocks,
                                     int n_requests, const int32_t* q_start, const int32_t* seq_lens, int n_q, int n_kv, int page_size,
                                     int64_t num_pages, float scale, int n_slices, float* part_o, float* part_ml, const float* table_t,
                                     const void* gate, int64_t gate_stride, int* err, cudaStream_t stream) {
    if (n_requests <= 0) return 0;
    if (page_size % 8 != 0 || 64 % page_size != 0 || n_slices < 1 || n_slices > SS_DECODE_MAX_SLICES || q_stride % 8) return (int)cudaErrorInvalidValue;
    const AcrossLayout y = across_layout(HEAD_DIM, n_q, n_kv);
    if (!y.stages) return (int)cudaErrorInvalidValue;
    CUtensorMap map_k, map_v;
    int rc = 0;
    for (int v = 0; v < 2 && !rc; ++v)
        rc = fa::make_map3(v ? &map_v : &map_k, kv, HEAD_DIM, (uint64_t)page_size, (uint64_t)num_pages * 2 * n_kv, (uint64_t)HEAD_DIM * 2,
                           (uint64_t)page_size * HEAD_DIM * 2, 64, (uint32_t)(page_size < y.bn ? page_size : y.bn), (uint32_t)(v ? y.nc : n_kv));
    if (rc) return rc;
    AcrossArgs a;
    a.q = (const bf16*)q; a.q_stride = q_stride; a.block_tables = block_tables; a.max_blocks = max_blocks; a.q_start = q_start;
    a.seq_lens = seq_lens; a.n_q = n_q; a.n_kv = n_kv; a.page_size = page_size; a.num_pages = num_pages; a.scale = scale;
    a.n_slices = n_slices; a.stages = y.stages; a.nc = y.nc; a.sets = y.sets; a.part_o = part_o; a.part_ml = part_ml; a.err = err;
    const int smem = across_smem_bytes(HEAD_DIM, n_kv, y);
    const dim3 grid(n_slices, (n_kv + y.nc - 1) / y.nc, n_requests);
    if (y.nh == 1) {
        if (y.bn == 64) rc = launch_across<64, 16, 1, 4>(map_k, map_v, a, grid, smem, stream);
        else if (y.nk == 16) rc = launch_across<32, 16, 1, 4>(map_k, map_v, a, grid, smem, stream);
        else rc = launch_across<32, 32, 1, 4>(map_k, map_v, a, grid, smem, stream);
    } else {
        rc = y.bn == 64 ? launch_across<64, 16, 2, 2>(map_k, map_v, a, grid, smem, stream) : launch_across<32, 32, 2, 2>(map_k, map_v, a, grid, smem, stream);
    }
    if (rc) return rc;
    TalkMergeArgs t;
    t.part_o = part_o; t.part_ml = part_ml; t.table_t = table_t; t.gate = (const bf16*)gate; t.gate_stride = gate_stride; t.out = (bf16*)out;
    t.q_start = q_start; t.seq_lens = seq_lens; t.n_q = n_q; t.n_kv = n_kv; t.nh = y.nh; t.n_parts = n_slices * y.sets;
    t.n_slices = n_slices; t.tile_keys = y.bn; t.splits = talk_merge_splits(n_kv, y.nh);
    const int merge_smem = talk_merge_smem(n_q, n_kv, y.nh, t.n_parts);
    const dim3 merge_grid(n_kv * (HEAD_DIM / AM_COLS), n_requests);
    if (y.nh == 1) {
        static SsPerDevice opted;
        if (int rc_smem = ss_opt_in_smem(talk_merge_kernel<HEAD_DIM, 1>, 100 * 1024, opted)) return rc_smem;
        ss_launch(talk_merge_kernel<HEAD_DIM, 1>, merge_grid, dim3(AM_THREADS), merge_smem, stream, t);
    } else {
        static SsPerDevice opted;
        if (int rc_smem = ss_opt_in_smem(talk_merge_kernel<HEAD_DIM, 2>, 100 * 1024, opted)) return rc_smem;
        ss_launch(talk_merge_kernel<HEAD_DIM, 2>, merge_grid, dim3(AM_THREADS), merge_smem, stream, t);
    }
    return SS_LAUNCH_CHECK();
}
#else
extern "C" int ss_attn_prefill_tc5_supported() { return 0; }
#endif

// ---------------------------------------------------------------- the entry point that allocates nothing
#include "no_alloc.h"
static_assert(SS_NOALLOC_MAX_SLICES == SS_DECODE_MAX_SLICES, "both entry points take the same slice counts");

// Scratch of ss_attn_decode_noalloc.  In host code this name is only a handle for
// cudaGetSymbolAddress, never a device address.
static __device__ __align__(256) float ss_noalloc_scratch[SS_NOALLOC_SCRATCH_FLOATS];

#define SS_NOALLOC_MAX_DEVICES 64
static float* ss_noalloc_ptr[SS_NOALLOC_MAX_DEVICES];  // device address of the array, per device

// One counter per (request, block of 16 heads of a kv group): the slice that finishes last combines the
// others.  Zero when the library is loaded; every call leaves them zero.
static __device__ __align__(256) int ss_noalloc_counters[SS_NOALLOC_COUNTERS];
static int* ss_noalloc_counter_ptr[SS_NOALLOC_MAX_DEVICES];

extern "C" int64_t ss_attn_decode_noalloc_floats(int n_requests, int n_q, int n_slices) {
    return (int64_t)n_requests * n_q * n_slices * (HEAD_DIM + 1);
}

extern "C" const char* ss_attn_decode_noalloc_message(int code) {
    switch (code) {
        case 0: return "ok";
        case SS_NOALLOC_TOO_LARGE:
            return "the call needs more than the 8 MiB of built-in scratch (n_requests * n_q * n_slices * "
                   "(head size + 1) floats): use fewer slices or requests, or ss_attn_decode_mma with scratch of your own";
        case SS_NOALLOC_BAD_ARGUMENT:
            return "a count is not positive, n_q is not a multiple of n_kv, or n_slices is above 64";
        case SS_NOALLOC_SETUP_FAILED: return "could not look up the scratch array on the current device";
        default: return code > 0 ? cudaGetErrorString((cudaError_t)code) : "unknown code";
    }
}

extern "C" int ss_attn_decode_noalloc(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                                      const void* kv, const int32_t* block_tables, int max_blocks,
                                      int n_requests, const int32_t* q_start, const int32_t* seq_lens, int n_q,
                                      int n_kv, int page_size, int64_t num_pages, float scale, int window,
                                      int n_slices, int* err, cudaStream_t stream) {
    if (n_requests <= 0 || n_q <= 0 || n_kv <= 0 || n_slices < 1 || n_slices > SS_NOALLOC_MAX_SLICES ||
        n_q % n_kv != 0 || page_size <= 0)
        return SS_NOALLOC_BAD_ARGUMENT;
    const int64_t floats = ss_attn_decode_noalloc_floats(n_requests, n_q, n_slices);
    if (floats > (int64_t)SS_NOALLOC_SCRATCH_FLOATS) return SS_NOALLOC_TOO_LARGE;
    if ((int64_t)n_requests * n_kv * ((n_q / n_kv + 15) / 16) > (int64_t)SS_NOALLOC_COUNTERS) return SS_NOALLOC_TOO_LARGE;

    // set-up, once per device, with that device current
    int device = -1;
    if (cudaGetDevice(&device) != cudaSuccess || device < 0 || device >= SS_NOALLOC_MAX_DEVICES)
        return SS_NOALLOC_SETUP_FAILED;
    float* scratch = ss_noalloc_ptr[device];
    if (scratch == nullptr) {
        if (cudaGetSymbolAddress((void**)&scratch, ss_noalloc_scratch) != cudaSuccess || scratch == nullptr)
            return SS_NOALLOC_SETUP_FAILED;
        ss_noalloc_ptr[device] = scratch;
    }
    int* counters = ss_noalloc_counter_ptr[device];
    if (counters == nullptr) {
        if (cudaGetSymbolAddress((void**)&counters, ss_noalloc_counters) != cudaSuccess || counters == nullptr)
            return SS_NOALLOC_SETUP_FAILED;
        ss_noalloc_counter_ptr[device] = counters;
    }
    float* part_o = scratch;
    float* part_lse = scratch + (int64_t)n_requests * n_q * n_slices * HEAD_DIM;

    constexpr int smem = mma_smem_bytes<HEAD_DIM>(16, DECODE_STAGES);
    static SsPerDevice opted;
    if (int rc_smem = ss_opt_in_smem(attn_decode_mma<HEAD_DIM>, smem, opted)) return rc_smem;
    const int G = n_q / n_kv;
    dim3 grid(n_requests, n_kv * ((G + 15) / 16), n_slices);
    ss_launch(attn_decode_mma<HEAD_DIM>, dim3(grid), dim3(MMA_THREADS), smem, stream, 
        (const bf16*)q, q_stride, (bf16*)out, out_stride, (const bf16*)kv, block_tables, max_blocks, q_start,
        seq_lens, n_q, n_kv, page_size, num_pages, scale, window, n_slices, 0, (const float*)nullptr, 0, 0, part_o, part_lse, counters, err, (const bf16*)nullptr, 0.f, (const float*)nullptr, 0, 0, 0);
    return SS_LAUNCH_CHECK();
}

extern "C" void ss_set_pdl(int on) { ss_pdl_flag() = on; }
