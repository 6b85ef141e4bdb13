// What lies between the q, k, v projection and the attention itself for an attention whose queries and keys are turned
// first and then divided by their own root mean square, head by head, without a weight. One block a token, a warp a head:
//
//   1. the first `rot` entries of every q and k head turn by pos * f_i (a table that may be scaled), both cos and sin times
//      `amp`;
//   2. q and k heads are divided by sqrt(mean over the head's entries + eps) (norm 0: left as they are);
//   3. q into the step's buffer, k and v into the token's page; rows there are `width` wide, zeros behind a head's entries.
//
// A layer that reads another layer's keys and values has no k and v columns (nkv 0): its queries alone are formed. All
// arithmetic is 32-bit; angles are pos * (hi + lo) in split arithmetic from tables made in 64-bit.
#include "common.cuh"

// M > 0: a lane holds its entries of a head (lane + 32 m, m < M) in registers between the norm's sum and the store.
template <typename TA, int M>
__global__ void __launch_bounds__(1024)
turned_attn_prep_kernel(TA* __restrict__ q_out, TA* __restrict__ k_pool, TA* __restrict__ v_pool, const float* __restrict__ proj, long long ld,
                        const float* __restrict__ freq, int rot, int interleaved, float amp, int norm, float eps,
                        const int* __restrict__ positions, const int* __restrict__ seq_of_token, const int* __restrict__ block_table,
                        int bt_stride, int num_pages, int page_size, int nh, int nkv, int hd, int vd, int width_k, int width_v,
                        int* __restrict__ err) {
    extern __shared__ float sm[];
    const int half = rot / 2;
    float* cs = sm;             // [rot / 2]
    float* sn = sm + half;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
    pdl_trigger();
    const int t = blockIdx.x, pos = positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float c, s;
        split_sincos((float)pos, freq[2 * i], freq[2 * i + 1], &c, &s);
        cs[i] = c * amp;
        sn[i] = s * amp;
    }
    int page = -1;
    if (nkv > 0) {
        page = block_table[(size_t)seq_of_token[t] * bt_stride + pos / page_size];
        if (page < 0 || page >= num_pages) { if (threadIdx.x == 0) atomicOr(err, CELLM_DEV_BAD_PAGE); page = -1; }
    }
    const int in_page = nkv > 0 ? pos % page_size : 0;
    pdl_wait();
    __syncthreads();
    const float* row = proj + (size_t)t * ld;
    for (int hh = warp; hh < nh + 2 * nkv; hh += nwarps) {
        if (hh >= nh + nkv) {           // a value head: copied
            const int g = hh - nh - nkv;
            const float* x = row + (size_t)(nh + nkv) * hd + (size_t)g * vd;
            if (page >= 0) {
                TA* dst = v_pool + (((size_t)page * nkv + g) * page_size + in_page) * width_v;
                for (int i = lane; i < width_v; i += 32) dst[i] = from_float<TA>(i < vd ? x[i] : 0.f);
            }
            continue;
        }
        const float* x = row + (size_t)hh * hd;
        auto turned = [&](int i) -> float {
            if (i >= rot) return x[i];
            int p, other;
            bool first;
            if (interleaved) { p = i >> 1; first = (i & 1) == 0; other = i ^ 1; }
            else { first = i < half; p = first ? i : i - half; other = first ? i + half : i - half; }
            return first ? x[i] * cs[p] - x[other] * sn[p] : x[i] * cs[p] + x[other] * sn[p];
        };
        TA* dst = nullptr;
        if (hh < nh) dst = q_out + ((size_t)t * nh + hh) * width_k;
        else if (page >= 0) dst = k_pool + (((size_t)page * nkv + (hh - nh)) * page_size + in_page) * width_k;
        if constexpr (M > 0) {
            float v[M], ss = 0.f;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const int i = lane + 32 * m;
                v[m] = i < hd ? turned(i) : 0.f;
                ss = fmaf(v[m], v[m], ss);
            }
            const float inv = norm ? 1.f / sqrtf(warp_sum(ss) / (float)hd + eps) : 1.f;
            if (!dst) continue;
#pragma unroll
            for (int m = 0; m < M; ++m) {
                const int i = lane + 32 * m;
                if (i < width_k) dst[i] = from_float<TA>(v[m] * inv);
            }
        } else {
            float inv = 1.f;
            if (norm) {
                float ss = 0.f;
                for (int i = lane; i < hd; i += 32) { const float v = turned(i); ss = fmaf(v, v, ss); }
                inv = 1.f / sqrtf(warp_sum(ss) / (float)hd + eps);
            }
            if (!dst) continue;
            for (int i = lane; i < width_k; i += 32) dst[i] = from_float<TA>(i < hd ? turned(i) * inv : 0.f);
        }
    }
}

// proj [T, ld] 32-bit: q (nh x hd), then k (nkv x hd) and v (nkv x vd) unless nkv is 0. freq [rot / 2][2] (rot 0: null).
// q_out [T, nh * width_k]; pools [page][kv head][slot in page][width_k | width_v].
CELLM_API int cellm_turned_attn_prep(void* q_out, void* k_pool, void* v_pool, const float* proj, long long ld, const float* freq, int rot,
                                     int interleaved, float amp, int norm, float eps, const int* positions, const int* seq_of_token,
                                     const int* block_table, int bt_stride, int num_pages, int page_size, int T, int nh, int nkv, int hd,
                                     int vd, int width_k, int width_v, int dtype, int* err, cudaStream_t stream) {
    if (T <= 0) return CELLM_OK;
    if (nh <= 0 || nkv < 0 || hd <= 0 || rot < 0 || rot > hd || rot % 2 || rot > 8192 || width_k < hd) return CELLM_ERR_SIZE;
    if (nkv > 0 && (nh % nkv || vd <= 0 || width_v < vd || page_size <= 0)) return CELLM_ERR_SIZE;
    if ((rot > 0 && !freq) || (nkv > 0 && (!k_pool || !v_pool || !block_table))) return CELLM_ERR_ARG;
    const size_t smem = (size_t)rot * sizeof(float);
    // a warp a head: few tokens take a warp for (nearly) every head, many share a block's warps among the heads
    const int heads = nh + 2 * nkv, threads = T >= 296 ? (heads >= 8 ? 256 : 128) : heads >= 32 ? 1024 : heads * 32;
#define TAP_RUN(TA, M)                                                                                                                        \
    CELLM_RUN((turned_attn_prep_kernel<TA, M>), T, threads, smem, stream, (TA*)q_out, (TA*)k_pool, (TA*)v_pool, proj, ld, freq, rot, interleaved, amp, \
              norm, eps, positions, seq_of_token, block_table, bt_stride, num_pages, page_size, nh, nkv, hd, vd, width_k, width_v, err)
    if (dtype == CELLM_F32) {
        if (width_k <= 64) TAP_RUN(float, 2);
        else if (width_k <= 128) TAP_RUN(float, 4);
        else TAP_RUN(float, 0);
    } else if (dtype == CELLM_BF16) {
        if (width_k <= 64) TAP_RUN(__nv_bfloat16, 2);
        else if (width_k <= 128) TAP_RUN(__nv_bfloat16, 4);
        else TAP_RUN(__nv_bfloat16, 0);
    } else return CELLM_ERR_DTYPE;
#undef TAP_RUN
    return CELLM_OK;
}
