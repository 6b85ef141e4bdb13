// The scalar-decay recurrence of long prompt portions, in chunks of 64 tokens on the tensor cores (mma.sync m16n8k16):
//
//   S_t = d_t S_(t-1) + w_t k_t v_t^T,   o_t = S_t^T q_t      (d_t, w_t one number per head and token; S [dim, vd] per head)
//
// With c_t the sum of ln d over a chunk's tokens up to t and S the state before the chunk,
//
//   o_t = e^(c_t) S^T q_t + sum over s <= t of e^(c_t - c_s) w_s (q_t . k_s) v_s
//   S behind the chunk = e^(c_last) S + sum over s of e^(c_last - c_s) w_s k_s v_s^T
//
// so that only the state's passage from chunk to chunk is sequential. Three kernels:
//
//   decay_chunk_states   every chunk's own contribution to the state (the last sum), all chunks and heads at once
//   decay_chunk_pass     the states before every chunk, a thread four entries of S, from the request's slot and back to it
//   decay_chunk_outputs  the read-outs
//
// Decays, their sums and exponentials, the state and all accumulators are 32-bit. A tensor-core operand x enters as two
// bfloat16 numbers, hi = bf16(x) and lo = bf16(x - hi), and a product as hi hi + hi lo + lo hi: about 16 bits of every
// factor, in products whose 32-bit sums do not feed back into the operands' rounding. Heads whose q and k are shared (a
// group) are taken several to a CTA, with q, k and their products formed once.
//
// Portions of a step shorter than `min_len` are left alone (the walk of recurrent.cu takes them).
#include <algorithm>

#include "mma_tiles.cuh"

namespace {

constexpr int CL = 64;          // tokens a chunk
constexpr int THREADS = 256;

struct ChunkArgs {
    const float *q, *k, *v, *logd, *write;
    long long ld_q, ld_k, ld_v, ld_d, ld_w;
    const int* cu_seqlens;
    const int* slot_ids;
    int B, min_len, heads, groups, dim, vd, hpc;      // hpc: heads a CTA (of one group)
    int pitch;              // vd rounded up to a multiple of 8: a row's width in ws
    float* ws;              // [chunk][head][dim][pitch]: a chunk's own contribution; then, in the same bytes, the state before it
                            // in packs of eight values, [8 hi | 8 lo] bfloat16
    float* tot;             // [chunk][head]: c_last
};

// Which portion the chunk with this index lies in: its first token and how many it has (0: none).
__device__ __forceinline__ int find_chunk(const ChunkArgs& a, int chunk, int& t0) {
    for (int b = 0; b < a.B; ++b) {
        const int start = a.cu_seqlens[b], len = a.cu_seqlens[b + 1] - start;
        if (len < a.min_len) continue;
        const int n = (len + CL - 1) / CL;
        if (chunk < n) { t0 = start + chunk * CL; return min(CL, len - chunk * CL); }
        chunk -= n;
    }
    return 0;
}

// Eight values of a 32-bit row of `width` values from column c0 on (zeros behind the width).
__device__ __forceinline__ void load8(float (&x)[8], const float* row, int c0, int width, bool ok, bool vec) {
    if (ok && vec && c0 < width) {
        const float4 a = *reinterpret_cast<const float4*>(row + c0), b = *reinterpret_cast<const float4*>(row + c0 + 4);
        x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w; x[4] = b.x; x[5] = b.y; x[6] = b.z; x[7] = b.w;
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = (ok && c0 + e < width) ? row[c0 + e] : 0.f;
    }
}
__device__ __forceinline__ bool rows_of_packs(const float* src, long long ld, int width) {
    return (width & 7) == 0 && (ld & 3) == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0;
}
// The two bfloat16 numbers of eight values.
__device__ __forceinline__ void split8(const float (&x)[8], uint4& hi, uint4& lo) {
    uint32_t h[4], l[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const __nv_bfloat162 p = __floats2bfloat162_rn(x[2 * e], x[2 * e + 1]);
        h[e] = *reinterpret_cast<const uint32_t*>(&p);
        const float2 back = __bfloat1622float2(p);
        l[e] = pack_bf16(x[2 * e] - back.x, x[2 * e + 1] - back.y);
    }
    hi = make_uint4(h[0], h[1], h[2], h[3]);
    lo = make_uint4(l[0], l[1], l[2], l[3]);
}

// Rows of a tile [CL][W] (W bfloat16 wide, permuted as mma_tiles.cuh says) from 32-bit rows of `width` values at pitch ld,
// times scale[row], as hi and lo; zeros behind the width and behind `len` rows.
template <int W>
__device__ __forceinline__ void split_rows(uint8_t* hi, uint8_t* lo, const float* src, long long ld, int width, int len, const float* scale) {
    constexpr int CH = W / 8;
    const bool vec = rows_of_packs(src, ld, width);
#pragma unroll 2
    for (int i = threadIdx.x; i < CL * CH; i += THREADS) {
        const int row = i / CH, chunk = i % CH;
        float x[8];
        load8(x, src + (size_t)row * ld, chunk * 8, width, row < len, vec);
        if (scale) {
            const float f = scale[row];
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= f;
        }
        const int off = tile_offset<W>(row, chunk);
        split8(x, *reinterpret_cast<uint4*>(hi + off), *reinterpret_cast<uint4*>(lo + off));
    }
}

// c_t of a head's chunk into cum[CL] (rows behind `len` repeat the last) by the first warp, and the writing factors.
__device__ __forceinline__ void chunk_sums(const ChunkArgs& a, int t0, int len, int h, float* cum, float* wr) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x, r = 2 * lane;
        const float d0 = r < len ? a.logd[(size_t)(t0 + r) * a.ld_d + h] : 0.f, d1 = r + 1 < len ? a.logd[(size_t)(t0 + r + 1) * a.ld_d + h] : 0.f;
        float s = d0 + d1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        cum[r] = s - d1;
        cum[r + 1] = s;
    } else if (threadIdx.x < 32 + CL) {
        const int r = threadIdx.x - 32;
        wr[r] = r < len ? (a.write ? a.write[(size_t)(t0 + r) * a.ld_w + h] : 1.f) : 0.f;
    }
}

__device__ __forceinline__ void mma3(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    mma_bf16(c, ah, bh0, bh1);
    mma_bf16(c, ah, bl0, bl1);
    mma_bf16(c, al, bh0, bh1);
}

template <int NP, int VP>
__global__ void __launch_bounds__(THREADS)
decay_chunk_states_kernel(const ChunkArgs a) {
    extern __shared__ __align__(128) uint8_t dc_smem[];
    uint8_t* k_h = dc_smem;
    uint8_t* k_l = k_h + CL * NP * 2;
    uint8_t* v_h = k_l + CL * NP * 2;
    uint8_t* v_l = v_h + CL * VP * 2;
    __shared__ float cum[CL], wr[CL], fac[CL];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    pdl_trigger();
    pdl_wait();
    int t0 = 0;
    const int len = find_chunk(a, blockIdx.x, t0);
    if (len == 0) return;
    const int h0 = blockIdx.y * a.hpc, g = h0 / (a.heads / a.groups);
    split_rows<NP>(k_h, k_l, a.k + (size_t)t0 * a.ld_k + (size_t)g * a.dim, a.ld_k, a.dim, len, nullptr);
    constexpr int MT = NP / 16, SHARES = 8 / MT;           // warps of a row tile share its column pairs
    const int mt = warp % MT, share = warp / MT;
    __syncthreads();
    uint32_t ah[CL / 16][4], al[CL / 16][4];               // the keys serve every head of the CTA
#pragma unroll
    for (int kk = 0; kk < CL / 16; ++kk) {
        const int ar = kk * 16 + (lane & 7) + ((lane >> 4) << 3), ac = mt * 2 + ((lane >> 3) & 1);        // k's rows are the product's columns
        ldmatrix_x4_trans(ah[kk], k_h + tile_offset<NP>(ar, ac));
        ldmatrix_x4_trans(al[kk], k_l + tile_offset<NP>(ar, ac));
    }
    for (int h = h0; h < h0 + a.hpc; ++h) {
        chunk_sums(a, t0, len, h, cum, wr);
        __syncthreads();
        if (threadIdx.x < CL) fac[threadIdx.x] = wr[threadIdx.x] * expf(cum[CL - 1] - cum[threadIdx.x]);
        if (threadIdx.x == 0) a.tot[(size_t)blockIdx.x * a.heads + h] = cum[CL - 1];
        __syncthreads();
        split_rows<VP>(v_h, v_l, a.v + (size_t)t0 * a.ld_v + (size_t)h * a.vd, a.ld_v, a.vd, len, fac);
        __syncthreads();
        float* dst = a.ws + ((size_t)blockIdx.x * a.heads + h) * a.dim * a.pitch;
        for (int n2 = share; n2 < VP / 16; n2 += SHARES) {
            float c[2][4] = {};
#pragma unroll
            for (int kk = 0; kk < CL / 16; ++kk) {
                uint32_t bh[4], bl[4];
                const int br = kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), bc = n2 * 2 + (lane >> 4);
                ldmatrix_x4_trans(bh, v_h + tile_offset<VP>(br, bc));
                ldmatrix_x4_trans(bl, v_l + tile_offset<VP>(br, bc));
                mma3(c[0], ah[kk], al[kk], bh[0], bh[1], bl[0], bl[1]);
                mma3(c[1], ah[kk], al[kk], bh[2], bh[3], bl[2], bl[3]);
            }
            const int row = mt * 16 + (lane >> 2);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const int col = n2 * 16 + n * 8 + (lane & 3) * 2;
                if (col < a.pitch) {        // an even pitch: both or none (columns behind vd hold zeros)
                    if (row < a.dim) *reinterpret_cast<float2*>(dst + (size_t)row * a.pitch + col) = make_float2(c[n][0], c[n][1]);
                    if (row + 8 < a.dim) *reinterpret_cast<float2*>(dst + (size_t)(row + 8) * a.pitch + col) = make_float2(c[n][2], c[n][3]);
                }
            }
        }
        __syncthreads();
    }
}

// The states before every chunk, in place of the chunks' contributions and already split into two bfloat16 numbers each; the
// state behind the last one into the slot. A thread a pack of eight columns of one row.
__global__ void __launch_bounds__(256)
decay_chunk_pass_kernel(const ChunkArgs a, float* __restrict__ state, long long slot_stride, int n_slots, int vec, int* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.x, h = blockIdx.y;
    const int packs = a.pitch / 8, i = blockIdx.z * 256 + threadIdx.x, row = i / packs, c0 = (i % packs) * 8;
    int first = 0, n = 0;
    for (int bb = 0; bb <= b; ++bb) {
        const int len = a.cu_seqlens[bb + 1] - a.cu_seqlens[bb];
        first += n;
        n = len < a.min_len ? 0 : (len + CL - 1) / CL;
    }
    if (n == 0 || row >= a.dim) return;
    const int slot = a.slot_ids[b];
    if (slot < 0 || slot >= n_slots) { if (threadIdx.x == 0) atomicOr(err, CELLM_DEV_BAD_SLOT); return; }
    float* st = state + (size_t)slot * slot_stride + ((size_t)h * a.dim + row) * a.vd;
    float* w = a.ws + (((size_t)first * a.heads + h) * a.dim + row) * a.pitch + c0;
    const size_t step = (size_t)a.heads * a.dim * a.pitch;
    const float* tot = a.tot + (size_t)first * a.heads + h;
    float s[8];
    load8(s, st, c0, a.vd, true, vec != 0);
    constexpr int AHEAD = 4;
    for (int k0 = 0; k0 < n; k0 += AHEAD) {
        float d[AHEAD][8], f[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (k0 + u < n) {
                load8(d[u], w + (size_t)(k0 + u) * step, 0, 8, true, true);
                f[u] = expf(tot[(size_t)(k0 + u) * a.heads]);
            }
        }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            if (k0 + u < n) {
                uint4* dst = reinterpret_cast<uint4*>(w + (size_t)(k0 + u) * step);
                uint4 hi, lo;
                split8(s, hi, lo);
                dst[0] = hi;
                dst[1] = lo;
#pragma unroll
                for (int e = 0; e < 8; ++e) s[e] = fmaf(f[u], s[e], d[u][e]);
            }
        }
    }
    if (vec) {
        *reinterpret_cast<float4*>(st + c0) = make_float4(s[0], s[1], s[2], s[3]);
        *reinterpret_cast<float4*>(st + c0 + 4) = make_float4(s[4], s[5], s[6], s[7]);
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e)
            if (c0 + e < a.vd) st[c0 + e] = s[e];
    }
}

// The packs of a head's state before the chunk into a tile [NP][VP] (zeros behind its rows and columns), by asynchronous copies.
template <int NP, int VP>
__device__ __forceinline__ void copy_state(const ChunkArgs& a, uint8_t* hi, uint8_t* lo, int chunk, int h) {
    constexpr int CH = VP / 8;
    const float* src = a.ws + ((size_t)chunk * a.heads + h) * a.dim * a.pitch;
#pragma unroll 2
    for (int i = threadIdx.x; i < NP * CH; i += THREADS) {
        const int row = i / CH, c = i % CH;
        const bool ok = row < a.dim && c * 8 < a.pitch;
        const float* p = ok ? src + (size_t)row * a.pitch + c * 8 : src;
        const int off = tile_offset<VP>(row, c);
        cp_async16(hi + off, p, ok ? 16 : 0);
        cp_async16(lo + off, p + 4, ok ? 16 : 0);
    }
}

// Eight warps: four row tiles of 16 tokens, and two halves of the value's columns. A head's state arrives by asynchronous
// copies while the head before is at work, in the keys' place and its own by turns (where the keys' tile is large enough);
// its values are fetched into registers under the products with the state.
template <int NP, int VP>
__global__ void __launch_bounds__(THREADS, VP == 128 ? 1 : 2)
decay_chunk_outputs_kernel(const ChunkArgs a, float* __restrict__ o_out) {
    extern __shared__ __align__(128) uint8_t dc_smem[];
    uint8_t* q_h = dc_smem;
    uint8_t* q_l = q_h + CL * NP * 2;
    uint8_t* k_h = q_l + CL * NP * 2;
    uint8_t* k_l = k_h + CL * NP * 2;
    uint8_t* v_h = k_l + CL * NP * 2;
    uint8_t* v_l = v_h + CL * VP * 2;
    uint8_t* s_h = v_l + CL * VP * 2;
    constexpr bool TURNS = VP <= CL;
    constexpr int STATE = NP * VP * 2;
    auto state_tile = [&](int n) { return TURNS && (n & 1) ? k_h : s_h; };
    __shared__ float cum[CL], wr[CL];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rt = warp & 3, half = warp >> 2;
    pdl_trigger();
    pdl_wait();
    int t0 = 0;
    const int len = find_chunk(a, blockIdx.x, t0);
    if (len == 0) return;
    const int h0 = blockIdx.y * a.hpc, grp = h0 / (a.heads / a.groups);
    copy_state<NP, VP>(a, s_h, s_h + STATE, blockIdx.x, h0);
    cp_async_commit();
    split_rows<NP>(q_h, q_l, a.q + (size_t)t0 * a.ld_q + (size_t)grp * a.dim, a.ld_q, a.dim, len, nullptr);
    split_rows<NP>(k_h, k_l, a.k + (size_t)t0 * a.ld_k + (size_t)grp * a.dim, a.ld_k, a.dim, len, nullptr);
    __syncthreads();
    // q_t . k_s for the warp's 16 tokens and the keys up to them
    float qk[CL / 8][4];
#pragma unroll
    for (int n = 0; n < CL / 8; ++n) qk[n][0] = qk[n][1] = qk[n][2] = qk[n][3] = 0.f;
    const int qr = rt * 16 + (lane & 15), qc = lane >> 4;
#pragma unroll 2
    for (int ks = 0; ks < NP / 16; ++ks) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, q_h + tile_offset<NP>(qr, ks * 2 + qc));
        ldmatrix_x4(al, q_l + tile_offset<NP>(qr, ks * 2 + qc));
#pragma unroll
        for (int n2 = 0; n2 < CL / 16; ++n2) {
            if (n2 <= rt) {
                uint32_t bh[4], bl[4];
                const int br = n2 * 16 + (lane & 7) + ((lane >> 4) << 3), bc = ks * 2 + ((lane >> 3) & 1);
                ldmatrix_x4(bh, k_h + tile_offset<NP>(br, bc));
                ldmatrix_x4(bl, k_l + tile_offset<NP>(br, bc));
                mma3(qk[2 * n2], ah, al, bh[0], bh[1], bl[0], bl[1]);
                mma3(qk[2 * n2 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
            }
        }
    }
    const int row_a = rt * 16 + (lane >> 2), row_b = row_a + 8;
    constexpr int VCH = VP / 8, VIT = CL * VCH / THREADS;          // packs of the values a thread fetches
    const bool v_vec = rows_of_packs(a.v + (size_t)t0 * a.ld_v, a.ld_v, a.vd);
    for (int n = 0; n < a.hpc; ++n) {
        const int h = h0 + n;
        __syncthreads();            // the keys, and the head before's tiles and sums, are used up
        chunk_sums(a, t0, len, h, cum, wr);
        float vx[VIT][8];
#pragma unroll
        for (int it = 0; it < VIT; ++it) {
            const int i = threadIdx.x + it * THREADS, row = i / VCH;
            load8(vx[it], a.v + (size_t)(t0 + (row < len ? row : 0)) * a.ld_v + (size_t)h * a.vd, (i % VCH) * 8, a.vd, row < len, v_vec);
        }
        if (TURNS) {
            if (n + 1 < a.hpc) {
                uint8_t* next = state_tile(n + 1);
                copy_state<NP, VP>(a, next, next + STATE, blockIdx.x, h + 1);
            }
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            if (n > 0) { copy_state<NP, VP>(a, s_h, s_h + STATE, blockIdx.x, h); cp_async_commit(); }
            cp_async_wait<0>();
        }
        __syncthreads();
        const uint8_t* st_h = state_tile(n);
        const uint8_t* st_l = st_h + STATE;
        float acc[VP / 16][4];
#pragma unroll
        for (int n = 0; n < VP / 16; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
        // the state before the chunk
#pragma unroll 2
        for (int ks = 0; ks < NP / 16; ++ks) {
            uint32_t ah[4], al[4];
            ldmatrix_x4(ah, q_h + tile_offset<NP>(qr, ks * 2 + qc));
            ldmatrix_x4(al, q_l + tile_offset<NP>(qr, ks * 2 + qc));
            const int br = ks * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
            for (int n2 = 0; n2 < VP / 32; ++n2) {
                uint32_t bh[4], bl[4];
                const int bc = half * (VP / 16) + n2 * 2 + (lane >> 4);
                ldmatrix_x4_trans(bh, st_h + tile_offset<VP>(br, bc));
                ldmatrix_x4_trans(bl, st_l + tile_offset<VP>(br, bc));
                mma3(acc[2 * n2], ah, al, bh[0], bh[1], bl[0], bl[1]);
                mma3(acc[2 * n2 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
            }
        }
#pragma unroll
        for (int it = 0; it < VIT; ++it) {
            const int i = threadIdx.x + it * THREADS, off = tile_offset<VP>(i / VCH, i % VCH);
            split8(vx[it], *reinterpret_cast<uint4*>(v_h + off), *reinterpret_cast<uint4*>(v_l + off));
        }
        __syncthreads();
        const float ca = cum[row_a], cb = cum[row_b], ea = expf(ca), eb = expf(cb);
#pragma unroll
        for (int n = 0; n < VP / 16; ++n) { acc[n][0] *= ea; acc[n][1] *= ea; acc[n][2] *= eb; acc[n][3] *= eb; }
        // the chunk's own tokens
#pragma unroll
        for (int kk = 0; kk < CL / 16; ++kk) {
            if (kk <= rt) {
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const int s = kk * 16 + n * 8 + (lane & 3) * 2;
                    const float c0 = cum[s], c1 = cum[s + 1], w0 = wr[s], w1 = wr[s + 1];
                    const float (&x)[4] = qk[2 * kk + n];
                    const float p0 = s <= row_a ? x[0] * (w0 * expf(ca - c0)) : 0.f, p1 = s + 1 <= row_a ? x[1] * (w1 * expf(ca - c1)) : 0.f;
                    const float p2 = s <= row_b ? x[2] * (w0 * expf(cb - c0)) : 0.f, p3 = s + 1 <= row_b ? x[3] * (w1 * expf(cb - c1)) : 0.f;
                    const __nv_bfloat162 t0_ = __floats2bfloat162_rn(p0, p1), t1_ = __floats2bfloat162_rn(p2, p3);
                    const float2 f0 = __bfloat1622float2(t0_), f1 = __bfloat1622float2(t1_);
                    ph[2 * n] = *reinterpret_cast<const uint32_t*>(&t0_);
                    ph[2 * n + 1] = *reinterpret_cast<const uint32_t*>(&t1_);
                    pl[2 * n] = pack_bf16(p0 - f0.x, p1 - f0.y);
                    pl[2 * n + 1] = pack_bf16(p2 - f1.x, p3 - f1.y);
                }
                const int br = kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
#pragma unroll
                for (int n2 = 0; n2 < VP / 32; ++n2) {
                    uint32_t bh[4], bl[4];
                    const int bc = half * (VP / 16) + n2 * 2 + (lane >> 4);
                    ldmatrix_x4_trans(bh, v_h + tile_offset<VP>(br, bc));
                    ldmatrix_x4_trans(bl, v_l + tile_offset<VP>(br, bc));
                    mma3(acc[2 * n2], ph, pl, bh[0], bh[1], bl[0], bl[1]);
                    mma3(acc[2 * n2 + 1], ph, pl, bh[2], bh[3], bl[2], bl[3]);
                }
            }
        }
        float* oa = o_out + (size_t)(t0 + row_a) * a.heads * a.vd + (size_t)h * a.vd;
        float* ob = oa + (size_t)8 * a.heads * a.vd;
#pragma unroll
        for (int n = 0; n < VP / 16; ++n) {
            const int j = half * (VP / 2) + n * 8 + (lane & 3) * 2;
            if (j + 1 < a.vd && (a.vd & 1) == 0) {
                if (row_a < len) *reinterpret_cast<float2*>(oa + j) = make_float2(acc[n][0], acc[n][1]);
                if (row_b < len) *reinterpret_cast<float2*>(ob + j) = make_float2(acc[n][2], acc[n][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    if (j + e < a.vd && row_a < len) oa[j + e] = acc[n][e];
                    if (j + e < a.vd && row_b < len) ob[j + e] = acc[n][2 + e];
                }
            }
        }
    }
}

template <int NP, int VP>
int launch_chunks(const ChunkArgs& a, float* o_out, float* state, long long slot_stride, int n_slots, int n_chunks, int* err, cudaStream_t stream) {
    const size_t smem_s = (size_t)CL * (NP + VP) * 4, smem_o = (size_t)CL * (2 * NP + VP) * 4 + (size_t)NP * VP * 4;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(decay_chunk_states_kernel<NP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_s);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_outputs_kernel<NP, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const dim3 grid((unsigned)n_chunks, (unsigned)(a.heads / a.hpc));
    CELLM_RUN((decay_chunk_states_kernel<NP, VP>), grid, THREADS, smem_s, stream, a);
    const int vec = a.vd % 8 == 0 && slot_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
    CELLM_RUN(decay_chunk_pass_kernel, dim3(a.B, a.heads, (a.dim * (a.pitch / 8) + 255) / 256), 256, 0, stream, a, state, slot_stride, n_slots, vec, err);
    CELLM_RUN((decay_chunk_outputs_kernel<NP, VP>), grid, THREADS, smem_o, stream, a, o_out);
    return CELLM_OK;
}

}  // namespace

// Sizes the chunked form is built for.
CELLM_API int cellm_decay_chunks_supports(int dim, int vd) { return dim >= 1 && dim <= 128 && vd >= 1 && vd <= 128; }

// Arguments as cellm_decay_scan's, with the logarithms of the decays (logd, pitch 0: one row of constants). n_chunks: the
// sum over the portions of at least min_len tokens of ceil(length / 64). ws: [n_chunks, heads, dim, vd rounded up to a multiple
// of 8] (16-byte aligned) and tot: [n_chunks, heads] 32-bit scratch. Portions shorter than min_len (at least 1) are not touched.
CELLM_API int cellm_decay_chunks(float* o_out, float* state, long long slot_stride, int n_slots, const float* q, long long ld_q, const float* k,
                                 long long ld_k, const float* v, long long ld_v, const float* logd, long long ld_d, const float* write,
                                 long long ld_w, const int* cu_seqlens, const int* slot_ids, int B, int n_chunks, int min_len, int heads,
                                 int groups, int dim, int vd, float* ws, float* tot, int* err, cudaStream_t stream) {
    if (B <= 0 || n_chunks <= 0) return CELLM_OK;
    if (heads <= 0 || groups <= 0 || heads % groups || min_len < 1 || !cellm_decay_chunks_supports(dim, vd)) return CELLM_ERR_SIZE;
    if (!logd || !ws || !tot) return CELLM_ERR_ARG;
    if (reinterpret_cast<uintptr_t>(ws) & 15) return CELLM_ERR_ALIGN;
    ChunkArgs a;
    a.q = q, a.k = k, a.v = v, a.logd = logd, a.write = write;
    a.ld_q = ld_q, a.ld_k = ld_k, a.ld_v = ld_v, a.ld_d = ld_d, a.ld_w = ld_w;
    a.cu_seqlens = cu_seqlens, a.slot_ids = slot_ids, a.B = B, a.min_len = min_len;
    a.heads = heads, a.groups = groups, a.dim = dim, a.vd = vd, a.pitch = (vd + 7) / 8 * 8, a.ws = ws, a.tot = tot;
    // heads of a group taken by one CTA: as many (a power of two that divides the group) as leave some three CTAs an SM
    a.hpc = 1;
    while ((heads / groups) % (a.hpc * 2) == 0 && (long long)n_chunks * (heads / (a.hpc * 2)) >= 444) a.hpc *= 2;
    if (heads / a.hpc > 65535 || heads > 65535) return CELLM_ERR_SIZE;
#define GO(N_, V_) return launch_chunks<N_, V_>(a, o_out, state, slot_stride, n_slots, n_chunks, err, stream)
    if (dim <= 32) { if (vd <= 32) GO(32, 32); else if (vd <= 64) GO(32, 64); else GO(32, 128); }
    else if (dim <= 64) { if (vd <= 32) GO(64, 32); else if (vd <= 64) GO(64, 64); else GO(64, 128); }
    else { if (vd <= 32) GO(128, 32); else if (vd <= 64) GO(128, 64); else GO(128, 128); }
#undef GO
}
