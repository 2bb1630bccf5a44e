// What stands between a fused q/k/v product and attention when heads are normed before they are rotated, when keys and
// values differ in width, or when only a strip of a row is rotated.
//
//   norm_rope_kv_write   rows (N, stride) = [q: H heads of DK | k: KV heads of DK | v: KV heads of DV | ...].  The first RD
//                        values of every q and k head are rotated by the token's position; before or after that the head
//                        is optionally divided by its root mean square and, also optionally, multiplied by a weight (DK
//                        values, shared by the heads); q is written back in place, k and v go into the page and slot of
//                        the position: kpool (pages, KV, page, DK), vpool (pages, KV, page, DV).  Values mixed across
//                        layers: v_keep receives the token's values as the product left them, (N, KV DV); with v_first
//                        (rows kept so by another layer of the same step) what is cached is (1 - lam) v + lam v_first.
//                        bias (as wide as q, k and v together, or null) is added to the rows first.
//   latent_rope          the rotated strips of latent attention: of every query head (H heads of q_head values, the
//                        strip at q_off) into the tail of that head's row of `qa` (H rows of qa_head values, the strip
//                        at qa_off), and of the token's shared key strip (kr_off in `rows`) into the tail of the
//                        position's cache row (pool (pages, 1, page, pool_row), the strip at pool_off).
//
// Rotation: pair i of RD/2 turns by position * freqs[i]; pairing 0 pairs value 2i with 2i + 1, pairing 1 value i with
// i + RD/2; cos and sin are multiplied by `gain` (1: a plain rotation).  Norms and angles are float32.
#include "common.cuh"

// v[0 .. W) in shared memory, the first RD values rotated in place by the threads of the block (a barrier before and after
// is the caller's)
__device__ __forceinline__ void rr_rotate(float* v, int RD, int pairing, const float* freqs, float pos, float gain) {
    for (int i = threadIdx.x; i < RD / 2; i += blockDim.x) {
        const int a = pairing ? i : 2 * i, b = pairing ? i + RD / 2 : 2 * i + 1;
        float sn, cs;
        sincosf(pos * freqs[i], &sn, &cs);
        sn *= gain;
        cs *= gain;
        const float u = v[a], w = v[b];
        v[a] = u * cs - w * sn;
        v[b] = w * cs + u * sn;
    }
}

// grid (N, ceil((H + KV) / NR_WARPS)): a block takes NR_WARPS of a token's H + KV heads, a warp a head; the token's cosines
// and sines are made once per block, by all its threads.  Shared memory: RD floats of cos and sin, then DK floats per warp.
#define NR_WARPS 8
enum { NR_NO_NORM = 0, NR_NORM_BEFORE = 1, NR_NORM_AFTER = 2 };
template <typename T>
__global__ void __launch_bounds__(NR_WARPS * 32) norm_rope_kv_write_kernel(
    T* __restrict__ rows, int stride, const float* __restrict__ qw, const float* __restrict__ kw, float eps, int norm_at,
    const float* __restrict__ freqs, int RD, int pairing, float gain, const int* __restrict__ positions,
    const int* __restrict__ tok_row, const int* __restrict__ table, int max_blocks, T* __restrict__ kpool,
    T* __restrict__ vpool, T* __restrict__ v_keep, const T* __restrict__ v_first, float lam, int H, int KV, int DK, int DV,
    int page, int num_pages, int* err, const float* __restrict__ bias) {
    extern __shared__ float smem[];
    float* cs = smem;                       // cos of the RD / 2 pairs, then sin
    const int n = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = RD / 2;
    float* vals = smem + RD + warp * DK;
    const int pos = positions[n];
    if (freqs) {
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            float sn, c;
            sincosf((float)pos * freqs[i], &sn, &c);
            cs[i] = c * gain;
            cs[half + i] = sn * gain;
        }
    }
    __syncthreads();
    size_t slot = 0;
    bool have_page = false;
    if (kpool) {
        const int pg = table[(size_t)tok_row[n] * max_blocks + pos / page];
        if (pg < 0 || pg >= num_pages) {
            if (threadIdx.x == 0) mb_set_error(err, pg < 0 ? MB_ERR_PAGE_MISSING : MB_ERR_PAGE_RANGE);
        } else {
            have_page = true;
            slot = (size_t)pg * KV * page + (pos % page);           // + kv head * page
        }
    }
    for (int b = blockIdx.y * NR_WARPS + warp; b < H + KV; b += gridDim.y * NR_WARPS) {
        const bool is_q = b < H;
        const int kvh = b - H;
        T* src = rows + (size_t)n * stride + (size_t)b * DK;       // the k heads follow the q heads
        const float* w = is_q ? qw : kw;
        float ss = 0.0f;
        for (int d = lane; d < DK; d += 32) {
            float x = mb_load(src + d);
            if (bias) x += bias[(size_t)b * DK + d];
            vals[d] = x;
            ss = fmaf(x, x, ss);
        }
        if (norm_at == NR_NORM_BEFORE) {
            const float r = 1.0f / sqrtf(mb_warp_sum(ss) / (float)DK + eps);
            for (int d = lane; d < DK; d += 32) vals[d] = vals[d] * r * (w ? w[d] : 1.0f);
        }
        __syncwarp();
        if (freqs) {
            for (int i = lane; i < half; i += 32) {
                const int a = pairing ? i : 2 * i, c = pairing ? i + half : 2 * i + 1;
                const float u = vals[a], v = vals[c];
                vals[a] = u * cs[i] - v * cs[half + i];
                vals[c] = v * cs[i] + u * cs[half + i];
            }
        }
        __syncwarp();
        if (norm_at == NR_NORM_AFTER) {
            ss = 0.0f;
            for (int d = lane; d < DK; d += 32) ss = fmaf(vals[d], vals[d], ss);
            const float r = 1.0f / sqrtf(mb_warp_sum(ss) / (float)DK + eps);
            for (int d = lane; d < DK; d += 32) vals[d] = vals[d] * r * (w ? w[d] : 1.0f);     // a lane's own values
        }
        if (is_q) {
            for (int d = lane; d < DK; d += 32) mb_store(src + d, vals[d]);
        } else {
            const size_t row = slot + (size_t)kvh * page, off = ((size_t)n * KV + kvh) * DV;
            if (have_page)
                for (int d = lane; d < DK; d += 32) mb_store(kpool + row * DK + d, vals[d]);
            const T* vs = rows + (size_t)n * stride + (size_t)(H + KV) * DK + (size_t)kvh * DV;
            for (int d = lane; d < DV; d += 32) {
                T v = vs[d];
                if (bias) mb_store(&v, mb_load(&v) + bias[(size_t)(H + KV) * DK + (size_t)kvh * DV + d]);
                if (v_keep) v_keep[off + d] = v;
                if (!have_page) continue;
                if (v_first) mb_store(vpool + row * DV + d, (1.0f - lam) * mb_load(&v) + lam * mb_load(v_first + off + d));
                else vpool[row * DV + d] = v;
            }
        }
        __syncwarp();
    }
}

// four neighbouring values in one access
template <typename T> struct NrQuad;
template <> struct NrQuad<float> { typedef float4 type; };
template <> struct NrQuad<bf16> { typedef uint2 type; };
__device__ __forceinline__ void nr_unpack(const float4& w, float (&x)[4]) { x[0] = w.x; x[1] = w.y; x[2] = w.z; x[3] = w.w; }
__device__ __forceinline__ void nr_unpack(const uint2& w, float (&x)[4]) {
    x[0] = __uint_as_float(w.x << 16); x[1] = __uint_as_float(w.x & 0xffff0000u);
    x[2] = __uint_as_float(w.y << 16); x[3] = __uint_as_float(w.y & 0xffff0000u);
}
__device__ __forceinline__ void nr_pack(float4& w, const float (&x)[4]) { w = make_float4(x[0], x[1], x[2], x[3]); }
__device__ __forceinline__ void nr_pack(uint2& w, const float (&x)[4]) { w = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3])); }

// The same for widths that are multiples of four and neighbours rotated together (or nothing rotated): a head stays in the
// registers of LANES neighbouring threads (QUADS groups of four values each), so one read and one write of global memory
// is all there is.  Shared memory: RD floats, the token's cosines and sines.
template <typename T, int LANES, int QUADS>
__global__ void __launch_bounds__(NR_WARPS * 32) norm_rope_kv_write_quads_kernel(
    T* __restrict__ rows, int stride, const float* __restrict__ qw, const float* __restrict__ kw, float eps, int norm_at,
    const float* __restrict__ freqs, int RD, float gain, const int* __restrict__ positions, const int* __restrict__ tok_row,
    const int* __restrict__ table, int max_blocks, T* __restrict__ kpool, T* __restrict__ vpool, T* __restrict__ v_keep,
    const T* __restrict__ v_first, float lam, int H, int KV, int DK, int DV, int page, int num_pages, int* err,
    const float* __restrict__ bias) {
    typedef typename NrQuad<T>::type Q;
    constexpr int PER = 32 / LANES;                     // heads a warp works on at once
    extern __shared__ float2 turn[];                    // (cos, sin) of a pair
    const int n = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & (LANES - 1), grp = (threadIdx.x & 31) / LANES;
    const int pos = positions[n];
    T* row_n = rows + (size_t)n * stride;
    if (freqs) {
        for (int i = threadIdx.x; i < RD / 2; i += blockDim.x) {
            float sn, c;
            sincosf((float)pos * freqs[i], &sn, &c);
            turn[i] = make_float2(c * gain, sn * gain);
        }
    }
    __syncthreads();
    size_t slot = 0;
    bool have_page = false;
    if (kpool) {
        const int pg = table[(size_t)tok_row[n] * max_blocks + pos / page];
        if (pg < 0 || pg >= num_pages) {
            if (threadIdx.x == 0) mb_set_error(err, pg < 0 ? MB_ERR_PAGE_MISSING : MB_ERR_PAGE_RANGE);
        } else {
            have_page = true;
            slot = (size_t)pg * KV * page + (pos % page);
        }
    }
    const int step = gridDim.y * NR_WARPS * PER;
    for (int b0 = (blockIdx.y * NR_WARPS + warp) * PER; b0 < H + KV; b0 += step) {      // the same trips for a whole warp
        const int b = b0 + grp, kvh = b - H;
        const bool live = b < H + KV, is_q = b < H;
        T* src = row_n + (size_t)(live ? b : 0) * DK;
        const float* w = is_q ? qw : kw;
        float x[QUADS][4];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < QUADS; i++) {
            const int d = (i * LANES + lane) * 4;
            x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.0f;
            if (live && d < DK) {
                nr_unpack(*reinterpret_cast<const Q*>(src + d), x[i]);
                if (bias)
#pragma unroll
                    for (int e = 0; e < 4; e++) x[i][e] += bias[(size_t)b * DK + d + e];
            }
#pragma unroll
            for (int e = 0; e < 4; e++) ss = fmaf(x[i][e], x[i][e], ss);
        }
        auto normed = [&]() {
#pragma unroll
            for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const float r = 1.0f / sqrtf(ss / (float)DK + eps);
#pragma unroll
            for (int i = 0; i < QUADS; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int d = (i * LANES + lane) * 4 + e;
                    x[i][e] = x[i][e] * r * (w && d < DK ? w[d] : 1.0f);
                }
        };
        if (norm_at == NR_NORM_BEFORE) normed();
        if (freqs) {
#pragma unroll
            for (int i = 0; i < QUADS; i++)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int d = (i * LANES + lane) * 4 + e;
                    if (d < RD) {
                        const float2 t = turn[d / 2];
                        const float u = x[i][e], v = x[i][e + 1];
                        x[i][e] = u * t.x - v * t.y;
                        x[i][e + 1] = v * t.x + u * t.y;
                    }
                }
        }
        if (norm_at == NR_NORM_AFTER) {
            ss = 0.0f;
#pragma unroll
            for (int i = 0; i < QUADS; i++)
#pragma unroll
                for (int e = 0; e < 4; e++) ss = fmaf(x[i][e], x[i][e], ss);
            normed();
        }
        if (!live) continue;                            // nothing below is met by the other lanes
        T* dst = is_q ? src : kpool + (slot + (size_t)kvh * page) * DK;
        if (is_q || have_page) {
#pragma unroll
            for (int i = 0; i < QUADS; i++) {
                const int d = (i * LANES + lane) * 4;
                Q o;
                nr_pack(o, x[i]);
                if (d < DK) *reinterpret_cast<Q*>(dst + d) = o;
            }
        }
        if (!is_q) {
            const size_t off = ((size_t)n * KV + kvh) * DV;
            const T* vs = row_n + (size_t)(H + KV) * DK + (size_t)kvh * DV;
            for (int d = lane * 4; d < DV; d += LANES * 4) {
                Q raw = *reinterpret_cast<const Q*>(vs + d);
                if (bias) {
                    float a[4];
                    nr_unpack(raw, a);
#pragma unroll
                    for (int e = 0; e < 4; e++) a[e] += bias[(size_t)(H + KV) * DK + (size_t)kvh * DV + d + e];
                    nr_pack(raw, a);
                }
                if (v_keep) *reinterpret_cast<Q*>(v_keep + off + d) = raw;
                if (!have_page) continue;
                if (v_first) {
                    float a[4], f[4];
                    nr_unpack(raw, a);
                    nr_unpack(*reinterpret_cast<const Q*>(v_first + off + d), f);
#pragma unroll
                    for (int e = 0; e < 4; e++) a[e] = (1.0f - lam) * a[e] + lam * f[e];
                    nr_pack(raw, a);
                }
                *reinterpret_cast<Q*>(vpool + (slot + (size_t)kvh * page) * DV + d) = raw;
            }
        }
    }
}

template <typename T>
static int norm_rope_launch(T* rows, int stride, const float* qw, const float* kw, float eps, int norm_at,
                            const float* freqs, int RD, int pairing, float gain, const int* positions, const int* tok_row,
                            const int* table, int max_blocks, T* kpool, T* vpool, T* v_keep, const T* v_first, float lam,
                            int N, int H, int KV, int DK, int DV, int page, int num_pages, int* err, const float* bias,
                            cudaStream_t st) {
    if (N == 0) return 0;
    if (H < 1 || KV < 1 || H + KV > 65535 * NR_WARPS || DK < 1 || DV < 1 || DK > 1024 || RD < 0 || RD > DK || (RD & 1) ||
        page < 1 || norm_at < NR_NO_NORM || norm_at > NR_NORM_AFTER)
        return -2;
    const uintptr_t ptrs = (uintptr_t)rows | (uintptr_t)kpool | (uintptr_t)vpool | (uintptr_t)v_keep | (uintptr_t)v_first;
    if (DK % 4 == 0 && DV % 4 == 0 && stride % 4 == 0 && (ptrs & 15) == 0 && (!freqs || RD == 0 || pairing == 0) && DK <= 512) {
        // few tokens: a pass of the block's warps over the heads each; many: a block keeps its token's cosines and sines
#define NR_CASE(LANES, QUADS)                                                                                              \
    if (DK <= 4 * LANES * QUADS) {                                                                                         \
        const int per = NR_WARPS * (32 / LANES), passes = (H + KV + per - 1) / per;                                        \
        norm_rope_kv_write_quads_kernel<T, LANES, QUADS>                                                                   \
            <<<dim3(N, N >= 592 ? 1 : passes), NR_WARPS * 32, (size_t)RD * sizeof(float), st>>>(                           \
                rows, stride, qw, kw, eps, norm_at, freqs, RD, gain, positions, tok_row, table, max_blocks, kpool, vpool,  \
                v_keep, v_first, lam, H, KV, DK, DV, page, num_pages, err, bias);                                          \
        MB_LAUNCH_CHECK();                                                                                                 \
        return 0;                                                                                                          \
    }
        NR_CASE(4, 1) NR_CASE(8, 1) NR_CASE(16, 1) NR_CASE(32, 1) NR_CASE(32, 2) NR_CASE(32, 4)
#undef NR_CASE
    }
    norm_rope_kv_write_kernel<T><<<dim3(N, (H + KV + NR_WARPS - 1) / NR_WARPS), NR_WARPS * 32,
                                   (size_t)(RD + NR_WARPS * DK) * sizeof(float), st>>>(
        rows, stride, qw, kw, eps, norm_at, freqs, RD, pairing, gain, positions, tok_row, table, max_blocks, kpool, vpool,
        v_keep, v_first, lam, H, KV, DK, DV, page, num_pages, err, bias);
    MB_LAUNCH_CHECK();
    return 0;
}

template <typename T>
__global__ void latent_rope_kernel(const T* __restrict__ q, int q_stride, int q_head, int q_off, T* __restrict__ qa,
                                   int qa_head, int qa_off, const T* __restrict__ rows, int rows_stride, int kr_off,
                                   T* __restrict__ pool, int pool_row, int pool_off, const float* __restrict__ freqs, int RD,
                                   int W, int pairing, float gain, const int* __restrict__ positions,
                                   const int* __restrict__ tok_row, const int* __restrict__ table, int max_blocks, int H,
                                   int page, int num_pages, int* err) {
    extern __shared__ float vals[];
    const int n = blockIdx.x, h = blockIdx.y;
    const int pos = positions[n];
    const T* src = h < H ? q + (size_t)n * q_stride + (size_t)h * q_head + q_off : rows + (size_t)n * rows_stride + kr_off;
    for (int d = threadIdx.x; d < W; d += blockDim.x) vals[d] = mb_load(src + d);
    __syncthreads();
    if (freqs && RD > 0) rr_rotate(vals, RD, pairing, freqs, (float)pos, gain);
    __syncthreads();
    T* dst;
    if (h < H) {
        dst = qa + ((size_t)n * H + h) * qa_head + qa_off;
    } else {
        if (!pool) return;
        const int pg = table[(size_t)tok_row[n] * max_blocks + pos / page];
        if (pg < 0 || pg >= num_pages) {
            if (threadIdx.x == 0) mb_set_error(err, pg < 0 ? MB_ERR_PAGE_MISSING : MB_ERR_PAGE_RANGE);
            return;
        }
        dst = pool + ((size_t)pg * page + (pos % page)) * pool_row + pool_off;
    }
    for (int d = threadIdx.x; d < W; d += blockDim.x) mb_store(dst + d, vals[d]);
}

#define RR_ENTRIES(SUF, T)                                                                                                 \
    MB_API int mb_norm_rope_kv_write_##SUF(void* rows, int stride, const float* qw, const float* kw, float eps, int norm_at, \
                                           const float* freqs, int RD, int pairing, float gain, const int* positions,      \
                                           const int* tok_row, const int* table, int max_blocks, void* kpool, void* vpool, \
                                           void* v_keep, const void* v_first, float lam, int N, int H, int KV, int DK, int DV, \
                                           int page, int num_pages, int* err, const float* bias, cudaStream_t st) {        \
        return norm_rope_launch<T>((T*)rows, stride, qw, kw, eps, norm_at, freqs, RD, pairing, gain, positions, tok_row, table, \
                                   max_blocks, (T*)kpool, (T*)vpool, (T*)v_keep, (const T*)v_first, lam, N, H, KV, DK, DV, \
                                   page, num_pages, err, bias, st);                                                        \
    }                                                                                                                      \
    MB_API int mb_latent_rope_##SUF(const void* q, int q_stride, int q_head, int q_off, void* qa, int qa_head, int qa_off, \
                                    const void* rows, int rows_stride, int kr_off, void* pool, int pool_row, int pool_off, \
                                    const float* freqs, int RD, int W, int pairing, float gain, const int* positions,     \
                                    const int* tok_row, const int* table, int max_blocks, int N, int H, int page,         \
                                    int num_pages, int* err, cudaStream_t st) {                                           \
        if (N == 0 || W == 0) return 0;                                                                                    \
        if (H < 1 || H + 1 > 65535 || W < 1 || W > 8192 || RD < 0 || RD > W || (RD & 1) || page < 1) return -2;            \
        latent_rope_kernel<T><<<dim3(N, H + 1), 32, (size_t)W * sizeof(float), st>>>(                                      \
            (const T*)q, q_stride, q_head, q_off, (T*)qa, qa_head, qa_off, (const T*)rows, rows_stride, kr_off, (T*)pool,  \
            pool_row, pool_off, freqs, RD, W, pairing, gain, positions, tok_row, table, max_blocks, H, page, num_pages,    \
            err);                                                                                                          \
        MB_LAUNCH_CHECK();                                                                                                 \
        return 0;                                                                                                          \
    }
RR_ENTRIES(f32, float)
RR_ENTRIES(bf16, bf16)
