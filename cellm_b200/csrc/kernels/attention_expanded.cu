// Attention of prompt portions over a latent cache in its expanded form, on the 5th-generation tensor cores (tcgen05).
//
// A latent mixer caches one compressed row [latent (rank) | shared rotated key part (rot_dim)] per token. A head's key is
// [K_h c | rotated part], its value V_h c. Single tokens attend to the rows themselves (attention_latent.cu: rank + rot_dim
// multiply-adds a key and head for the score, rank for the value). For a portion of many tokens it is cheaper to make the
// heads' keys and values first, once for all of the portion's tokens, by one product over the rows that the portion can
// see: dim + rot_dim and vdim multiply-adds a pair are left.
//
//   latent_rows    the rows that the step's requests can see, copied out of their pages into one dense matrix, request after
//                  request (with a window: from the first row that the request's first new token can see)
//   (a product)    kv = rows[:, :rank] . [K; V]^T: all heads' unrotated keys, then all heads' values, [rows, heads * (dim + vdim)]
//   attention      flash attention of every head over its own keys and values:
//
// One CTA takes two tiles of 128 tokens of one head and walks the request's keys in blocks of 128:
//   warp 0      TMA: the two Q tiles once, then per block the key and value tiles, in chunks of 64 columns (128 keys x 128
//               bytes, 128-byte swizzle) through one ring of 16-KB slots: a block's key chunks (unrotated, rotated), then
//               its value chunks, then the next block's;
//   warp 1      MMA: per tile S = Q.K^T (M 128, N 128, K = dim, then rot_dim) and O += P.V (M 128, N up to 64 a chunk, K
//               128). P takes the place of the scores in tensor memory, so a tile's next scores are issued behind its P.V;
//               while one tile's softmax runs, the tensor cores work on the other tile;
//   warps 2..5  softmax of the first tile, warps 6..9 of the second, one row per thread, as in attention_tc.cu: scores into
//               registers, mask, running maximum and sum in 32-bit, P = 2^(s*c - m) rounded to bfloat16 into tensor memory;
//               the output accumulator is rescaled only when a row's maximum has grown by more than 2^8.
// Sinks (one more term in a row's denominator) and the output gate (sigmoid of one number per token and head) enter in the
// epilogue. Every wait on an mbarrier is bounded: a role that gives up sets CELLM_DEV_WAIT_TIMEOUT and an abort flag; the
// CTA frees its tensor memory and returns.
#include "tcgen05_attn.cuh"

namespace {

constexpr int TM = 128;              // rows (tokens) of a tile
constexpr int TN = 128;              // keys of a block
constexpr int CHUNK = TN * 128;      // bytes of a chunk: 128 rows of 64 bfloat16
constexpr int MAX_SLOTS = 12;
constexpr int MAX_Q_CHUNKS = 4;      // of a tile: ceil(dim / 64) + ceil(rot_dim / 64)
constexpr int O_COL = 256;           // tensor memory: scores (and P) of tile t in columns t * 128, its output in 256 + t * 128
constexpr int TMEM_ALL = 512;
constexpr int THREADS = 320;         // warp 0 TMA, warp 1 MMA, warps 2..5 softmax of tile 0, warps 6..9 of tile 1
constexpr int SMEM_LIMIT = 227 * 1024;

struct Control {
    uint64_t q_full, slot_full[MAX_SLOTS], slot_empty[MAX_SLOTS];
    uint64_t s_full[2], p_full[2], pv_done[2];
    uint32_t tmem_base;
    int abort_flag;
};

// The dense rows of request b begin at row `at` with its key `first`.
__device__ __forceinline__ int first_row_key(int ctx, int window) { return window > 0 ? max(0, ctx - window + 1) : 0; }

// ---- the rows out of their pages: 16-byte pieces ---------------------------------------------------------------------
__global__ void latent_rows_kernel(uint4* __restrict__ rows, const uint4* pool, const int* __restrict__ cu_seqlens,
                                   const int* __restrict__ ctx_lens, const int* __restrict__ block_table, int bt_stride, int B, int num_pages,
                                   int page_size, int window, int kw8, int* __restrict__ err) {
    pdl_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    int r = blockIdx.x * (blockDim.x >> 5) + warp, b = 0, key = 0;
    for (; b < B; ++b) {
        const int ctx = ctx_lens[b], n = cu_seqlens[b + 1] - cu_seqlens[b], first = first_row_key(ctx, window);
        const int len = n > 0 ? ctx + n - first : 0;
        if (r < len) { key = first + r; break; }
        r -= len;
    }
    pdl_wait();
    if (b >= B) return;
    const int page = block_table[(size_t)b * bt_stride + key / page_size];
    const size_t dst = (size_t)(blockIdx.x * (blockDim.x >> 5) + warp) * kw8;
    if (page < 0 || page >= num_pages) {
        if (lane == 0) atomicOr(err, CELLM_DEV_BAD_PAGE);
        for (int i = lane; i < kw8; i += 32) rows[dst + i] = make_uint4(0, 0, 0, 0);
        return;
    }
    const size_t src = ((size_t)page * page_size + key % page_size) * kw8;
    for (int i = lane; i < kw8; i += 32) rows[dst + i] = pool[src + i];
}

struct Shape {
    int dim, rot, vdim, heads;
    int kc_plain, kc_rot, vc;        // chunks of a key's unrotated and rotated parts and of a value
    int rank;                        // column of the rotated part in a row
    int slots;                       // of the ring
};

__global__ void __launch_bounds__(384, 1)
attention_expanded_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_q_rot,
                          const __grid_constant__ CUtensorMap map_kv, const __grid_constant__ CUtensorMap map_rows,
                          __nv_bfloat16* __restrict__ out, const int* __restrict__ cu_seqlens, const int* __restrict__ ctx_lens, int B,
                          Shape sh, float scale_log2e, int window, const float* __restrict__ sinks, const float* gate, int* __restrict__ err) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    const int kc = sh.kc_plain + sh.kc_rot;
    uint8_t* q_s = smem_raw;                                          // [2][kc] chunks
    uint8_t* ring = smem_raw + 2 * kc * CHUNK;                        // [slots] chunks
    Control& sm = *reinterpret_cast<Control*>(ring + sh.slots * CHUNK);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y;
    if (smem_u32(smem_raw) & 1023u) {            // the swizzled tiles need 1024-byte alignment
        if (threadIdx.x == 0) atomicOr(err, CELLM_DEV_BAD_LAYOUT);
        return;
    }
    if (threadIdx.x == 0) {
        mbar_init(&sm.q_full, 1);
        for (int i = 0; i < sh.slots; ++i) { mbar_init(&sm.slot_full[i], 1); mbar_init(&sm.slot_empty[i], 1); }
        for (int t = 0; t < 2; ++t) { mbar_init(&sm.s_full[t], 1); mbar_init(&sm.p_full[t], 128); mbar_init(&sm.pv_done[t], 1); }
        sm.abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_kv) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_rows) : "memory");
    }
    if (warp == 1) tmem_alloc(&sm.tmem_base, TMEM_ALL);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_trigger();
    pdl_wait();
    const uint32_t tmem = sm.tmem_base;
    volatile int* abort_flag = &sm.abort_flag;

    // which request this pair of tiles belongs to (from the last to the first: longest first), and where its dense rows begin
    const int item = (int)gridDim.x - 1 - (int)blockIdx.x;
    int b = 0, base = 0, row0 = 0;
    for (; b < B; ++b) {
        const int n = cu_seqlens[b + 1] - cu_seqlens[b], nt = (n + 2 * TM - 1) / (2 * TM);
        if (item < base + nt) break;
        base += nt;
        if (n > 0) row0 += ctx_lens[b] + n - first_row_key(ctx_lens[b], window);
    }
    const bool live = b < B;
    int t_base = 0, q_len = 0, ctx = 0, kb0 = 0, nblk = 0;
    int tok0[2] = {0, 0}, lo_blk[2] = {0, 0}, hi_blk[2] = {0, 0};
    if (live) {
        t_base = cu_seqlens[b];
        q_len = cu_seqlens[b + 1] - t_base;
        ctx = ctx_lens[b];
        row0 -= first_row_key(ctx, window);                           // the dense row of key j is row0 + j
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            tok0[t] = (item - base) * 2 * TM + t * TM;
            if (tok0[t] < q_len) {
                const int tok1 = min(tok0[t] + TM, q_len) - 1;
                lo_blk[t] = (window > 0 ? max(0, ctx + tok0[t] - window + 1) : 0) / TN;
                hi_blk[t] = (ctx + tok1) / TN + 1;
            }
        }
        // tile 1 holds later tokens: its blocks start and end no earlier than tile 0's
        kb0 = lo_blk[0];
        nblk = (hi_blk[1] > 0 ? hi_blk[1] : hi_blk[0]) - kb0;
    }
    auto active = [&](int t, int j) { return kb0 + j >= (t ? lo_blk[1] : lo_blk[0]) && kb0 + j < (t ? hi_blk[1] : hi_blk[0]); };
    const int per_block = kc + sh.vc;                                 // chunks of a block

    if (warp == 0) {
        if (live && lane == 0) {
            const int tiles = hi_blk[1] > 0 ? 2 : 1, qw = sh.dim + sh.rot;
            mbar_expect_tx(&sm.q_full, (uint32_t)(tiles * kc * CHUNK));
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                if (t >= tiles) break;
                for (int c = 0; c < sh.kc_plain; ++c) tma_load_2d(q_s + (t * kc + c) * CHUNK, &map_q, head * qw + c * 64, t_base + tok0[t], &sm.q_full);
                for (int c = 0; c < sh.kc_rot; ++c)
                    tma_load_2d(q_s + (t * kc + sh.kc_plain + c) * CHUNK, &map_q_rot, head * sh.rot + c * 64, t_base + tok0[t], &sm.q_full);
            }
            bool ok = true;
            int slot = 0;
            uint32_t phase = 0;
            for (int j = 0; ok && j < nblk; ++j) {
                const int row = row0 + (kb0 + j) * TN;                // may lie before the first row: those keys are masked
                for (int c = 0; c < per_block; ++c) {
                    ok = mbar_wait(&sm.slot_empty[slot], phase ^ 1u, abort_flag);
                    if (!ok) break;
                    mbar_expect_tx(&sm.slot_full[slot], CHUNK);
                    uint8_t* dst = ring + slot * CHUNK;
                    if (c < sh.kc_plain) tma_load_2d(dst, &map_kv, head * sh.dim + c * 64, row, &sm.slot_full[slot]);
                    else if (c < kc) tma_load_2d(dst, &map_rows, sh.rank + (c - sh.kc_plain) * 64, row, &sm.slot_full[slot]);
                    else tma_load_2d(dst, &map_kv, sh.heads * sh.dim + head * sh.vdim + (c - kc) * 64, row, &sm.slot_full[slot]);
                    if (++slot == sh.slots) { slot = 0; phase ^= 1u; }
                }
            }
            if (!ok) { *abort_flag = 1; atomicOr(err, CELLM_DEV_WAIT_TIMEOUT); }
        }
    } else if (warp == 1) {
        if (live && lane == 0) {
            const uint32_t idesc_s = umma_idesc(TM, TN, false);       // S[128 x 128] = Q (K-major) . K^T (K-major)
            const uint32_t idesc_v0 = umma_idesc(TM, min(sh.vdim, 64), true), idesc_v1 = umma_idesc(TM, max(sh.vdim - 64, 16), true);
            const uint64_t dq0 = umma_desc(smem_u32(q_s)), dr0 = umma_desc(smem_u32(ring));
            bool started[2] = {false, false};                         // a tile's output accumulator holds something
            uint32_t p_phase[2] = {0, 0};
            bool ok = mbar_wait(&sm.q_full, 0, abort_flag);
            // The chunks go through the ring in order: a cursor is a slot and its fill's parity.
            struct Cursor { int slot; uint32_t phase; };
            auto advance = [&](Cursor c, int n) { c.slot += n; if (c.slot >= sh.slots) { c.slot -= sh.slots; c.phase ^= 1u; } return c; };
            auto wait_chunks = [&](Cursor c, int n) -> bool {
                for (int i = 0; i < n; ++i, c = advance(c, 1))
                    if (!mbar_wait(&sm.slot_full[c.slot], c.phase, abort_flag)) return false;
                return true;
            };
            auto release_chunks = [&](Cursor c, int n) {
                for (int i = 0; i < n; ++i, c = advance(c, 1)) umma_commit(&sm.slot_empty[c.slot]);
            };
            // scores of a block whose key chunks begin at c, for tile t. They take the place of the tile's P, which the P.V
            // issued before them reads: one thread's products run in the order in which it issues them.
            auto issue_s = [&](int t, Cursor c) {
                uint64_t dq = dq0 + (uint64_t)(t * kc * (CHUNK / 16));
                uint32_t acc = 0u;
                for (int part = 0; part < 2; ++part) {
                    int steps = (part ? sh.rot : sh.dim) / 16;
                    while (steps > 0) {
                        const uint64_t dk = dr0 + (uint64_t)(c.slot * (CHUNK / 16));
#pragma unroll
                        for (int ks = 0; ks < 4; ++ks) {
                            if (ks < steps) umma_bf16(tmem + (uint32_t)(t * TN), dq + (uint64_t)(ks * 2), dk + (uint64_t)(ks * 2), idesc_s, acc);
                            acc = 1u;
                        }
                        steps -= 4;
                        dq += (uint64_t)(CHUNK / 16);
                        c = advance(c, 1);
                    }
                }
                umma_commit(&sm.s_full[t]);
            };
            auto issue_pv = [&](int t, Cursor c) -> bool {
                if (!mbar_wait(&sm.p_full[t], p_phase[t], abort_flag)) return false;
                p_phase[t] ^= 1u;
                tc_fence_after();
                for (int v = 0; v < sh.vc; ++v, c = advance(c, 1)) {
                    const uint64_t dv = dr0 + (uint64_t)(c.slot * (CHUNK / 16));
#pragma unroll
                    for (int ks = 0; ks < TN / 16; ++ks)               // 16 keys = 8 columns of P = 16 rows of V
                        umma_bf16_ts(tmem + (uint32_t)(O_COL + t * TN + v * 64), tmem + (uint32_t)(t * TN + ks * 8), dv + (uint64_t)(ks * 16 * 128 / 16),
                                     v ? idesc_v1 : idesc_v0, started[t] || ks != 0 ? 1u : 0u);
                }
                started[t] = true;
                return true;
            };
            Cursor keys{0, 0u};
            if (ok && nblk > 0) {
                ok = wait_chunks(keys, kc);
                if (ok) {
                    tc_fence_after();
#pragma unroll
                    for (int t = 0; t < 2; ++t)
                        if (active(t, 0)) issue_s(t, keys);
                    release_chunks(keys, kc);
                }
            }
            for (int j = 0; ok && j < nblk; ++j) {
                const Cursor vals = advance(keys, kc), next = advance(vals, sh.vc);
                const bool more = j + 1 < nblk;
                ok = wait_chunks(vals, sh.vc) && (!more || wait_chunks(next, kc));
                if (!ok) break;
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    if (ok && active(t, j)) ok = issue_pv(t, vals);
                    if (ok && active(t, j) && !active(t, j + 1)) umma_commit(&sm.pv_done[t]);       // the tile's last
                    if (t == 1 && ok) release_chunks(vals, sh.vc);
                    if (ok && more && active(t, j + 1)) { tc_fence_after(); issue_s(t, next); }
                }
                if (ok && more) release_chunks(next, kc);
                keys = next;
            }
            if (!ok) { *abort_flag = 1; atomicOr(err, CELLM_DEV_WAIT_TIMEOUT); }
        }
    } else if (live && (warp >= 6 ? hi_blk[1] : hi_blk[0]) > 0) {
        const int t = (warp - 2) >> 2;                                // which tile
        const int lo_t = t ? lo_blk[1] : lo_blk[0], hi_t = t ? hi_blk[1] : hi_blk[0];
        const int qt = warp & 3;                                      // quarter of the tile's rows = of tensor memory's lanes
        const int tok = (t ? tok0[1] : tok0[0]) + qt * 32 + lane;                     // token within the portion
        const bool row_ok = tok < q_len;
        const int pos = row_ok ? ctx + tok : -1;
        const int lo = window > 0 ? pos - window + 1 : 0;
        const uint32_t lane_base = tmem + ((uint32_t)(qt * 32) << 16);
        const uint32_t s_col = (uint32_t)(t * TN), o_col = (uint32_t)(O_COL + t * TN);
        const int n_blocks = hi_t - lo_t;
        const int o_cols = (sh.vdim + 31) / 32 * 32;
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        for (int it = 0; it < n_blocks; ++it) {
            // the scores are there; the tile's P.V before them is done too (they were issued after it)
            ok = mbar_wait(&sm.s_full[t], (uint32_t)it & 1u, abort_flag);
            if (!ok) break;
            tc_fence_after();
            uint32_t s[TN];
#pragma unroll
            for (int c = 0; c < TN / 32; ++c) tmem_ld32_nowait(lane_base + s_col + (uint32_t)(c * 32), s + c * 32);
            tmem_ld_wait();
            const int jbase = (lo_t + it) * TN;
            const bool open_block = row_ok && jbase + TN - 1 <= pos && jbase >= lo;
            if (!open_block) {
#pragma unroll
                for (int i = 0; i < TN; ++i) {
                    const int key = jbase + i;
                    if (!(key <= pos && key >= lo)) s[i] = 0xff800000u;            // -inf
                }
            }
            float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
            for (int i = 0; i < TN; i += 4) {
                mx0 = fmaxf(mx0, __uint_as_float(s[i]));     mx1 = fmaxf(mx1, __uint_as_float(s[i + 1]));
                mx2 = fmaxf(mx2, __uint_as_float(s[i + 2])); mx3 = fmaxf(mx3, __uint_as_float(s[i + 3]));
            }
            const float m_new = fmaxf(m, fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3)) * scale_log2e);
            const bool want = m_new > m + RESCALE_STEP || (m == -INFINITY && m_new != -INFINITY);
            if (__any_sync(0xffffffffu, want)) {
                if (it > 0) {
                    const float corr = want ? (m == -INFINITY ? 0.f : fast_exp2(m - m_new)) : 1.0f;
#pragma unroll 1
                    for (int c = 0; c < o_cols; c += 32) {
                        uint32_t o[32];
                        tmem_ld32(lane_base + o_col + (uint32_t)c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                        tmem_st32(lane_base + o_col + (uint32_t)c, o);
                    }
                    if (want) l *= corr;
                }
                if (want) m = m_new;
            }
            // P = 2^(s*c - m) in place (-inf gives 0), then rounded to bfloat16 pairs (in place again)
            const float neg_use = m == -INFINITY ? 0.f : -m;
#pragma unroll
            for (int i = 0; i < TN; ++i) s[i] = __float_as_uint(fast_exp2(fmaf(__uint_as_float(s[i]), scale_log2e, neg_use)));
            float sum0 = 0.f, sum1 = 0.f, sum2 = 0.f, sum3 = 0.f;
#pragma unroll
            for (int i = 0; i < TN / 2; i += 2) {
                const float a0 = __uint_as_float(s[2 * i]), a1 = __uint_as_float(s[2 * i + 1]);
                const float a2 = __uint_as_float(s[2 * i + 2]), a3 = __uint_as_float(s[2 * i + 3]);
                sum0 += a0; sum1 += a1; sum2 += a2; sum3 += a3;
                s[i] = pack_bf16(a0, a1);
                s[i + 1] = pack_bf16(a2, a3);
            }
            l += (sum0 + sum1) + (sum2 + sum3);
#pragma unroll
            for (int c = 0; c < TN / 64; ++c) tmem_st32_nowait(lane_base + s_col + (uint32_t)(c * 32), s + c * 32);
            tmem_st_wait();
            tc_fence_before();
            mbar_arrive(&sm.p_full[t]);
        }
        if (ok && n_blocks > 0) ok = mbar_wait(&sm.pv_done[t], 0, abort_flag);
        if (!ok && lane == 0) { *abort_flag = 1; atomicOr(err, CELLM_DEV_WAIT_TIMEOUT); }
        if (ok) {
            tc_fence_after();
            if (sinks && row_ok) l += exp2f(sinks[head] * 1.4426950408889634f - (m == -INFINITY ? 0.f : m));
            float inv = l > 0.f ? 1.0f / l : 0.f;
            if (gate && row_ok) inv *= 1.f / (1.f + __expf(-gate[(size_t)(t_base + tok) * sh.heads + head]));
            __nv_bfloat16* dst = out + ((size_t)(t_base + tok) * sh.heads + head) * sh.vdim;
#pragma unroll 1
            for (int c = 0; c < o_cols; c += 32) {
                uint32_t o[32];
                tmem_ld32(lane_base + o_col + (uint32_t)c, o);
                if (row_ok) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (c + i * 8 < sh.vdim) {
                            uint32_t w4[4];
#pragma unroll
                            for (int k = 0; k < 4; ++k)
                                w4[k] = pack_bf16(__uint_as_float(o[8 * i + 2 * k]) * inv, __uint_as_float(o[8 * i + 2 * k + 1]) * inv);
                            *reinterpret_cast<uint4*>(dst + c + i * 8) = make_uint4(w4[0], w4[1], w4[2], w4[3]);
                        }
                    }
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, TMEM_ALL);
}

// The kernel's shape for a mixer's sizes, or false if it does not take them.
bool shape_of(int heads, int dim, int rot, int vdim, int rank, Shape* out) {
    if (heads < 1 || dim < 16 || (dim & 15) || rot < 0 || (rot & 15) || vdim < 16 || (vdim & 15) || vdim > 128 || rank < 8 || (rank & 7)) return false;
    Shape s{dim, rot, vdim, heads, (dim + 63) / 64, (rot + 63) / 64, (vdim + 63) / 64, rank, 0};
    const int kc = s.kc_plain + s.kc_rot;
    if (kc > MAX_Q_CHUNKS) return false;
    const int room = (SMEM_LIMIT - (int)sizeof(Control) - 2 * kc * CHUNK) / CHUNK;
    s.slots = room < MAX_SLOTS ? room : MAX_SLOTS;
    if (s.slots < kc + s.vc) return false;      // a block's values and the next block's keys are held at once
    *out = s;
    return true;
}

}  // namespace

// 1 if the kernel takes a mixer of these sizes.
CELLM_API int cellm_attention_expanded_supports(int heads, int dim, int rot_dim, int vdim, int rank) {
    Shape s;
    return shape_of(heads, dim, rot_dim, vdim, rank, &s) ? 1 : 0;
}

// rows [n_rows, kw] bfloat16: for every request of the step with new tokens its rows ctx + tokens, of which with a window only
// those from max(0, ctx - window + 1) on, request after request. pool: one layer's rows [pages][page_size][kw], kw a
// multiple of 8.
CELLM_API int cellm_latent_rows(void* rows, const void* pool, const int* cu_seqlens, const int* ctx_lens, const int* block_table, int bt_stride,
                                int B, int n_rows, int num_pages, int page_size, int window, int kw, int* err, cudaStream_t stream) {
    if (B <= 0 || n_rows <= 0) return CELLM_OK;
    if (kw <= 0 || (kw & 7) || page_size <= 0 || window < 0) return CELLM_ERR_SIZE;
    if (((uintptr_t)rows | (uintptr_t)pool) & 15) return CELLM_ERR_ALIGN;
    CELLM_RUN(latent_rows_kernel, (unsigned)((n_rows + 7) / 8), 256, 0, stream, (uint4*)rows, (const uint4*)pool, cu_seqlens, ctx_lens, block_table,
              bt_stride, B, num_pages, page_size, window, kw / 8, err);
    return CELLM_OK;
}

// out [T, heads * vdim]; q [T, q_ld], heads of dim + rot_dim (the unrotated parts are read), q_rot [T, heads * rot_dim] (turned);
// rows [n_rows, kw] as cellm_latent_rows leaves them (read from column rank on), kv [n_rows, heads * dim + heads * vdim]. n_tiles:
// the sum over the requests of ceil(tokens / 256). sinks [heads], gate [T, heads]: 32-bit or null.
CELLM_API int cellm_attention_expanded(void* out, const void* q, long long q_ld, const void* q_rot, const void* rows, const void* kv,
                                       const int* cu_seqlens, const int* ctx_lens, int B, int T, int n_tiles, int n_rows, int heads, int dim,
                                       int rot_dim, int vdim, int rank, float scale, int window, const float* sinks, const float* gate, int* err,
                                       cudaStream_t stream) {
    if (T <= 0 || B <= 0 || n_tiles <= 0) return CELLM_OK;
    Shape sh;
    if (!shape_of(heads, dim, rot_dim, vdim, rank, &sh) || !(scale > 0.f) || window < 0 || n_rows <= 0) return CELLM_ERR_SIZE;
    const int qw = dim + rot_dim, kw = rank + rot_dim, n = heads * (dim + vdim);
    if (q_ld < (long long)heads * qw || (q_ld & 7) || (kw & 7)) return CELLM_ERR_SIZE;
    if (((uintptr_t)out | (uintptr_t)q | (uintptr_t)q_rot | (uintptr_t)rows | (uintptr_t)kv) & 15) return CELLM_ERR_ALIGN;
    if (rot_dim && !q_rot) return CELLM_ERR_ARG;
    CUtensorMap mq, mr, mkv, mrows;
    if (!tensor_map(&mq, q, T, (uint64_t)heads * qw, (uint64_t)q_ld * 2, TM) || !tensor_map(&mkv, kv, n_rows, n, (uint64_t)n * 2, TN) ||
        !tensor_map(&mrows, rows, n_rows, kw, (uint64_t)kw * 2, TN))
        return CELLM_ERR_ARG;
    mr = mq;
    if (rot_dim && !tensor_map(&mr, q_rot, T, (uint64_t)heads * rot_dim, (uint64_t)heads * rot_dim * 2, TM)) return CELLM_ERR_ARG;
    const size_t smem = (size_t)(2 * (sh.kc_plain + sh.kc_rot) + sh.slots) * CHUNK + sizeof(Control);
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_expanded_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_LIMIT);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    CELLM_RUN(attention_expanded_kernel, dim3((unsigned)n_tiles, (unsigned)heads), THREADS, smem, stream, mq, mr, mkv, mrows, (__nv_bfloat16*)out,
              cu_seqlens, ctx_lens, B, sh, scale * 1.4426950408889634f, window, sinks, gate, err);
    return CELLM_OK;
}
