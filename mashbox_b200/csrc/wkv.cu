// What feeds the wkv recurrence (the gated scan that reads its state before the token joins it):
//
//   token_mix   h' = the row of the token before it in its sequence (a step's first token: the one the sequence's state
//               keeps, zeros at the start);  out[s, n] = h[n] + (h'[n] - h[n]) mu[s] for every stream s; the state is
//               replaced by the sequence's last row of the step
//   tanh_rows   tanh, float32 to the storage type
//   wkv_gates   r, k, v widened to float32; decay = exp(-exp(z + w0)); b = sum_i r_i u_i k_i per head.  z comes from a
//               product, or is made here from the narrow rows: z = W2 tanh(low)
//
// Mixing, tanh, decays and sums are float32 whatever the storage type.
#include "common.cuh"

template <typename T, int VEC>
__device__ __forceinline__ void wk_load(const T* p, float (&x)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; e++) x[e] = mb_load(p + e);
}
template <> __device__ __forceinline__ void wk_load<float, 4>(const float* p, float (&x)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
}
template <> __device__ __forceinline__ void wk_load<bf16, 4>(const bf16* p, float (&x)[4]) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    x[0] = __uint_as_float(v.x << 16); x[1] = __uint_as_float(v.x & 0xffff0000u);
    x[2] = __uint_as_float(v.y << 16); x[3] = __uint_as_float(v.y & 0xffff0000u);
}
template <typename T, int VEC>
__device__ __forceinline__ void wk_store(T* p, const float (&x)[VEC]) {
#pragma unroll
    for (int e = 0; e < VEC; e++) mb_store(p + e, x[e]);
}
template <> __device__ __forceinline__ void wk_store<float, 4>(float* p, const float (&x)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
}
template <> __device__ __forceinline__ void wk_store<bf16, 4>(bf16* p, const float (&x)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]));
}

// grid (N, pieces of a row), a thread VEC channels.  The thread of a sequence's first token of the step is the only one
// that touches the state: it reads the kept row and then writes the row of the sequence's last token in its place.
template <typename T, int VEC>
__global__ void token_mix_kernel(const T* __restrict__ h, const float* __restrict__ mu, const int* __restrict__ tok_seq,
                                 const int* __restrict__ q_start, const int* __restrict__ q_len,
                                 const int* __restrict__ state_slot, float* __restrict__ state, long long state_stride,
                                 T* __restrict__ out, int N, int D, int streams) {
    const int n = blockIdx.x, d = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (d >= D) return;
    const int s = tok_seq[n], first = q_start[s];
    float x[VEC], p[VEC];
    wk_load<T, VEC>(h + (size_t)n * D + d, x);
    if (n > first) {
        wk_load<T, VEC>(h + (size_t)(n - 1) * D + d, p);
    } else {
        float* kept = state + (size_t)state_slot[s] * state_stride + d;
        float last[VEC];
        wk_load<T, VEC>(h + (size_t)(first + q_len[s] - 1) * D + d, last);
        wk_load<float, VEC>(kept, p);
        wk_store<float, VEC>(kept, last);
    }
#pragma unroll
    for (int e = 0; e < VEC; e++) p[e] -= x[e];
    for (int j = 0; j < streams; j++) {
        float m[VEC], y[VEC];
        wk_load<float, VEC>(mu + (size_t)j * D + d, m);
#pragma unroll
        for (int e = 0; e < VEC; e++) y[e] = fmaf(p[e], m[e], x[e]);
        wk_store<T, VEC>(out + ((size_t)j * N + n) * D + d, y);
    }
}

template <typename T>
__global__ void tanh_rows_kernel(const float* __restrict__ x, T* __restrict__ y, long long total) {
    const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < total) mb_store(y + i, tanhf(x[i]));
}

// sum over r of w[r] x[r], x in shared memory
__device__ __forceinline__ float wk_dot(const float* w, const float* x, int R) {
    float acc = 0.0f;
    for (int r = 0; r < R; r++) acc = fmaf(w[r], x[r], acc);
    return acc;
}
__device__ __forceinline__ float wk_dot(const bf16* w, const float* x, int R) {
    float acc = 0.0f;
    if ((R & 7) == 0 && ((uintptr_t)w & 15) == 0) {
#pragma unroll 4
        for (int r = 0; r < R; r += 8) {
            const uint4 v = *reinterpret_cast<const uint4*>(w + r);
            const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int p = 0; p < 4; p++) {
                acc = fmaf(__uint_as_float(u[p] << 16), x[r + 2 * p], acc);
                acc = fmaf(__uint_as_float(u[p] & 0xffff0000u), x[r + 2 * p + 1], acc);
            }
        }
    } else {
        for (int r = 0; r < R; r++) acc = fmaf(__bfloat162float(w[r]), x[r], acc);
    }
    return acc;
}

// grid (N, H).  rows (N, stride) = [r (H dim) | k (H dim) | v (H dim) | ..]; z (N, H dim) float32, or low (N, R) float32 and
// w2 (H dim, R)
template <typename T>
__global__ void wkv_gates_kernel(const T* __restrict__ rows, int stride, const float* __restrict__ z,
                                 const float* __restrict__ low, const T* __restrict__ w2, int R,
                                 const float* __restrict__ w0, const float* __restrict__ u, float* __restrict__ r,
                                 float* __restrict__ k, float* __restrict__ v, float* __restrict__ g, float* __restrict__ b,
                                 int H, int dim) {
    extern __shared__ float narrow[];
    __shared__ float scratch[32];
    const int n = blockIdx.x, h = blockIdx.y, C = H * dim;
    if (low) {
        for (int i = threadIdx.x; i < R; i += blockDim.x) narrow[i] = tanhf(low[(size_t)n * R + i]);
        __syncthreads();
    }
    const T* row = rows + (size_t)n * stride + (size_t)h * dim;
    const size_t at = (size_t)n * C + (size_t)h * dim;
    float sum = 0.0f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        const int c = h * dim + i;
        const float rr = mb_load(row + i), kk = mb_load(row + C + i);
        const float zz = low ? wk_dot(w2 + (size_t)c * R, narrow, R) : z[at + i];
        r[at + i] = rr;
        k[at + i] = kk;
        v[at + i] = mb_load(row + 2 * C + i);
        g[at + i] = expf(-expf(zz + w0[c]));
        sum = fmaf(rr * u[c], kk, sum);
    }
    sum = mb_block_sum(sum, scratch);
    if (threadIdx.x == 0) b[(size_t)n * H + h] = sum;
}

template <typename T>
static int token_mix_launch(const T* h, const float* mu, const int* tok_seq, const int* q_start, const int* q_len,
                            const int* state_slot, float* state, long long state_stride, T* out, int N, int D, int streams,
                            cudaStream_t st) {
    if (N == 0) return 0;
    if (D < 1 || streams < 1 || state_stride < D) return -2;
    const uintptr_t ptrs = (uintptr_t)h | (uintptr_t)mu | (uintptr_t)state | (uintptr_t)out;
    if (D % 4 == 0 && state_stride % 4 == 0 && (ptrs & 15) == 0) {
        const int threads = D >= 512 ? 128 : 64, per = threads * 4;
        token_mix_kernel<T, 4><<<dim3(N, (D + per - 1) / per), threads, 0, st>>>(h, mu, tok_seq, q_start, q_len, state_slot,
                                                                                state, state_stride, out, N, D, streams);
    } else {
        token_mix_kernel<T, 1><<<dim3(N, (D + 127) / 128), 128, 0, st>>>(h, mu, tok_seq, q_start, q_len, state_slot, state,
                                                                         state_stride, out, N, D, streams);
    }
    MB_LAUNCH_CHECK();
    return 0;
}

#define WKV_ENTRIES(SUF, T)                                                                                                \
    MB_API int mb_token_mix_##SUF(const void* h, const float* mu, const int* tok_seq, const int* q_start,                  \
                                  const int* q_len, const int* state_slot, float* state, long long state_stride,           \
                                  void* out, int N, int D, int streams, cudaStream_t st) {                                 \
        return token_mix_launch<T>((const T*)h, mu, tok_seq, q_start, q_len, state_slot, state, state_stride, (T*)out, N,  \
                                   D, streams, st);                                                                        \
    }                                                                                                                      \
    MB_API int mb_tanh_rows_##SUF(const float* x, void* y, long long total, cudaStream_t st) {                             \
        if (total == 0) return 0;                                                                                          \
        tanh_rows_kernel<T><<<(unsigned)((total + 255) / 256), 256, 0, st>>>(x, (T*)y, total);                             \
        MB_LAUNCH_CHECK();                                                                                                 \
        return 0;                                                                                                          \
    }                                                                                                                      \
    MB_API int mb_wkv_gates_##SUF(const void* rows, int stride, const float* z, const float* low, const void* w2, int R,   \
                                  const float* w0, const float* u, float* r, float* k, float* v, float* g, float* b,       \
                                  int N, int H, int dim, cudaStream_t st) {                                                \
        if (N == 0) return 0;                                                                                              \
        if (H < 1 || H > 65535 || dim < 1 || stride < 3 * H * dim || (!z && (!low || !w2 || R < 1 || R > 8192))) return -2; \
        wkv_gates_kernel<T><<<dim3(N, H), dim > 64 ? 128 : dim > 32 ? 64 : 32, z ? 0 : (size_t)R * sizeof(float), st>>>(   \
            (const T*)rows, stride, z, z ? nullptr : low, (const T*)w2, R, w0, u, r, k, v, g, b, H, dim);                  \
        MB_LAUNCH_CHECK();                                                                                                 \
        return 0;                                                                                                          \
    }
WKV_ENTRIES(f32, float)
WKV_ENTRIES(bf16, bf16)
