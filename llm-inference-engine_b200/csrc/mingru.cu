// mingru.cu -- the minGRU mixer (B200_MIXER_MINGRU): a gated recurrence whose gates read the current token only, element by element
//     s_t = (1 - z_t) s_(t-1) + z_t c_t,   z = sigmoid(z-in + b_z),   u = u-in + b_u,   c = u + 1/2 where u >= 0, sigmoid(u) elsewhere,
// result s_t * silu(gate_t).  The state is one fp32 vector per sequence; everything from the projections' outputs on is fp32.
//
// A step is an affine map s -> A s + B with A = 1 - z, B = z c, and maps compose, so a long portion is not a chain of its tokens.  It is cut
// into chunks and every chunk into kSubs runs of tokens, one per warp of a CTA (a lane holds N adjacent channels):
//   * mingru_chunk_kernel forms the map of every run and, composed, of every chunk;
//   * mingru_apply_kernel composes the maps of the chunks before its own (shared out over its warps) and of the runs before each warp's, and
//     walks the tokens.
// The first chunk's map has the sequence's state already applied (its B is the state after the chunk), and its A entry carries the state the
// chunk starts from: the state slot is read by one kernel and written by the next.
// Portions of fewer than kMingruShort tokens (decoded tokens) are walked by one thread per channel in mingru_step_kernel.
#include "hybrid_ops.cuh"

#include <algorithm>

namespace b200 {

// hardware exponential and reciprocal: absolute error of a few 1e-7 over the whole range, 0 and 1 at its ends
__device__ __forceinline__ float sigmoid_m(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }

struct MingruStep { float keep, add; };
__device__ __forceinline__ MingruStep mingru_step(float zin, float u) {
    const float z = sigmoid_m(zin), c = u >= 0.0f ? u + 0.5f : sigmoid_m(u);
    return {1.0f - z, z * c};
}

// N adjacent channels of one token
template <typename T, int N>
struct MingruCols {
    const T *proj;
    int ld, col, cols;
    float bz[N], bu[N];
    __device__ __forceinline__ MingruCols(const T *p, int ld_, int cols_, const float *b, int c) : proj(p), ld(ld_), col(c), cols(cols_) {
#pragma unroll
        for (int i = 0; i < N; ++i) bz[i] = b ? b[c + i] : 0.0f, bu[i] = b ? b[cols + c + i] : 0.0f;
    }
    __device__ __forceinline__ void load(int t, float *z, float *u) const {
        const T *row = proj + (size_t)t * ld + col;
        load_n<T, N>(row, z);
        load_n<T, N>(row + cols, u);
#pragma unroll
        for (int i = 0; i < N; ++i) z[i] += bz[i], u[i] += bu[i];
    }
    __device__ __forceinline__ void gate(int t, float *g) const { load_n<T, N>(proj + (size_t)t * ld + 2 * cols + col, g); }
};

// maps: fp32 [chunks, 1 + kSubs, 2 (A, B), cols]: the chunk's map, then its runs'
constexpr int kSubs = 8;
static_assert((1 + kSubs) * 2 == kMingruMapRows, "the scratch of the chunk maps");

// grid (blocks of 32 * N channels, chunks)
template <typename T, int N>
__global__ void __launch_bounds__(32 * kSubs)
mingru_chunk_kernel(const T *__restrict__ proj, int ld, const float *__restrict__ bias, const float *__restrict__ state, float *__restrict__ maps,
                    const int4 *__restrict__ chunks, const int *__restrict__ seq_pos0, const int *__restrict__ seq_slot, int cols) {
    __shared__ float sa[kSubs][32 * N], sb[kSubs][32 * N];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x * 32 + lane) * N;
    const int4 ch = chunks[blockIdx.y];  // sequence, first packed row, tokens, index in its portion
    const int run = (ch.z + kSubs - 1) / kSubs, t0 = ch.y + min(ch.z, warp * run), t1 = ch.y + min(ch.z, (warp + 1) * run);
    float *m = maps + (size_t)blockIdx.y * (1 + kSubs) * 2 * cols + c;
    float A[N], B[N];
#pragma unroll
    for (int i = 0; i < N; ++i) A[i] = 1.0f, B[i] = 0.0f;
    if (c < cols) {
        const MingruCols<T, N> in(proj, ld, cols, bias, c);
#pragma unroll 8
        for (int t = t0; t < t1; ++t) {
            float z[N], u[N];
            in.load(t, z, u);
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const MingruStep s = mingru_step(z[i], u[i]);
                A[i] *= s.keep, B[i] = fmaf(s.keep, B[i], s.add);
            }
        }
        store_n<float, N>(m + (size_t)(1 + warp) * 2 * cols, A);
        store_n<float, N>(m + (size_t)(1 + warp) * 2 * cols + cols, B);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) sa[warp][lane * N + i] = A[i], sb[warp][lane * N + i] = B[i];
    __syncthreads();
    if (warp > 0 || c >= cols) return;
    float first[N];
#pragma unroll
    for (int i = 0; i < N; ++i) first[i] = 0.0f;
    if (ch.w == 0 && seq_pos0[ch.x] > 0) load_n<float, N>(state + (size_t)seq_slot[ch.x] * cols + c, first);
#pragma unroll
    for (int i = 0; i < N; ++i) {
        A[i] = 1.0f, B[i] = first[i];
#pragma unroll
        for (int w = 0; w < kSubs; ++w) {
            const float a = sa[w][lane * N + i];
            A[i] *= a, B[i] = fmaf(a, B[i], sb[w][lane * N + i]);
        }
    }
    store_n<float, N>(m, ch.w == 0 ? first : A);
    store_n<float, N>(m + cols, B);
}

template <typename T, int N>
__global__ void __launch_bounds__(32 * kSubs)
mingru_apply_kernel(const T *__restrict__ proj, int ld, const float *__restrict__ bias, float *__restrict__ state, const float *__restrict__ maps,
                    T *__restrict__ out, const int4 *__restrict__ chunks, const int *__restrict__ seq_start, const int *__restrict__ seq_slot, int cols) {
    __shared__ float sa[kSubs][32 * N], sb[kSubs][32 * N];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x * 32 + lane) * N;
    const int4 ch = chunks[blockIdx.y];
    const bool live = c < cols;
    const size_t per = (size_t)(1 + kSubs) * 2 * cols;
    const float *m0 = maps + (size_t)(blockIdx.y - ch.w) * per + c, *own = maps + (size_t)blockIdx.y * per + 2 * cols + c;
    float s[N];
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = 0.0f;
    if (live) load_n<float, N>(ch.w == 0 ? m0 : m0 + cols, s);
    if (ch.w > 1) {  // the chunks 1 .. ch.w - 1 (the whole CTA agrees)
        const int share = (ch.w - 1 + kSubs - 1) / kSubs, k0 = 1 + warp * share, k1 = min(ch.w, k0 + share);
        float A[N], B[N];
#pragma unroll
        for (int i = 0; i < N; ++i) A[i] = 1.0f, B[i] = 0.0f;
        if (live) {
#pragma unroll 4
            for (int k = k0; k < k1; ++k) {
                float a[N], b[N];
                load_n<float, N>(m0 + k * per, a);
                load_n<float, N>(m0 + k * per + cols, b);
#pragma unroll
                for (int i = 0; i < N; ++i) A[i] *= a[i], B[i] = fmaf(a[i], B[i], b[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < N; ++i) sa[warp][lane * N + i] = A[i], sb[warp][lane * N + i] = B[i];
        __syncthreads();
#pragma unroll
        for (int w = 0; w < kSubs; ++w)
#pragma unroll
            for (int i = 0; i < N; ++i) s[i] = fmaf(sa[w][lane * N + i], s[i], sb[w][lane * N + i]);
    }
    if (!live) return;
    const MingruCols<T, N> in(proj, ld, cols, bias, c);
#pragma unroll
    for (int w = 0; w < kSubs - 1; ++w) {
        if (w < warp) {
            float a[N], b[N];
            load_n<float, N>(own + (size_t)w * 2 * cols, a);
            load_n<float, N>(own + (size_t)w * 2 * cols + cols, b);
#pragma unroll
            for (int i = 0; i < N; ++i) s[i] = fmaf(a[i], s[i], b[i]);
        }
    }
    const int run = (ch.z + kSubs - 1) / kSubs, t0 = ch.y + min(ch.z, warp * run), t1 = ch.y + min(ch.z, (warp + 1) * run);
#pragma unroll 8
    for (int t = t0; t < t1; ++t) {
        float z[N], u[N], g[N];
        in.load(t, z, u);
        in.gate(t, g);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const MingruStep st = mingru_step(z[i], u[i]);
            s[i] = fmaf(st.keep, s[i], st.add);
            g[i] = s[i] * g[i] * sigmoid_m(g[i]);
        }
        store_n<T, N>(out + (size_t)t * cols + c, g);
    }
    if (t1 > t0 && t1 == seq_start[ch.x + 1]) store_n<float, N>(state + (size_t)seq_slot[ch.x] * cols + c, s);
}

// grid (channel blocks, sequences): portions of fewer than kMingruShort tokens
template <typename T, int N>
__global__ void __launch_bounds__(128)
mingru_step_kernel(const T *__restrict__ proj, int ld, const float *__restrict__ bias, float *__restrict__ state, T *__restrict__ out,
                   const int *__restrict__ seq_start, const int *__restrict__ seq_pos0, const int *__restrict__ seq_slot, int cols) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * N, q = blockIdx.y;
    const int t0 = seq_start[q], t1 = seq_start[q + 1];
    if (c >= cols || t1 == t0 || t1 - t0 >= kMingruShort) return;
    const MingruCols<T, N> in(proj, ld, cols, bias, c);
    float *st = state + (size_t)seq_slot[q] * cols + c;
    float s[N];
#pragma unroll
    for (int i = 0; i < N; ++i) s[i] = 0.0f;
    if (seq_pos0[q] > 0) load_n<float, N>(st, s);
    for (int t = t0; t < t1; ++t) {
        float z[N], u[N], g[N];
        in.load(t, z, u);
        in.gate(t, g);
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const MingruStep m = mingru_step(z[i], u[i]);
            s[i] = fmaf(m.keep, s[i], m.add);
            g[i] = s[i] * g[i] * sigmoid_m(g[i]);
        }
        store_n<T, N>(out + (size_t)t * cols + c, g);
    }
    store_n<float, N>(st, s);
}

int launch_mingru(int dtype, const void *proj, int ld, const float *bias, float *state, float *maps, void *out, const int *chunks, int n_chunks,
                  const int *seq_start, const int *seq_pos0, const int *seq_slot, int n_seqs, int n_short, int cols, cudaStream_t st) {
    const int es = dtype == B200_F32 ? 4 : 2;
    const bool vec = cols % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<size_t>(proj) % (4 * es)) == 0 && (reinterpret_cast<size_t>(out) % (4 * es)) == 0 &&
                     ((reinterpret_cast<size_t>(state) | reinterpret_cast<size_t>(maps)) & 15) == 0;
    const int n = vec ? 4 : 1, threads = std::min(128, ((cols + n - 1) / n + 31) / 32 * 32);
    const int blocks = (cols + n * threads - 1) / (n * threads);
    const int4 *ch = reinterpret_cast<const int4 *>(chunks);
    B200_DISPATCH_DTYPE(dtype, {
        if (n_chunks > 0) {
            auto chunk = vec ? mingru_chunk_kernel<T, 4> : mingru_chunk_kernel<T, 1>;
            auto apply = vec ? mingru_apply_kernel<T, 4> : mingru_apply_kernel<T, 1>;
            const dim3 grid((cols + 32 * n - 1) / (32 * n), n_chunks);
            chunk<<<grid, 32 * kSubs, 0, st>>>((const T *)proj, ld, bias, state, maps, ch, seq_pos0, seq_slot, cols);
            apply<<<grid, 32 * kSubs, 0, st>>>((const T *)proj, ld, bias, state, maps, (T *)out, ch, seq_start, seq_slot, cols);
        }
        if (n_short > 0) {
            auto step = vec ? mingru_step_kernel<T, 4> : mingru_step_kernel<T, 1>;
            step<<<dim3(blocks, n_seqs), threads, 0, st>>>((const T *)proj, ld, bias, state, (T *)out, seq_start, seq_pos0, seq_slot, cols);
        }
    });
    return cuda_status("mingru launch");
}

}  // namespace b200

using namespace b200;

extern "C" int b200_mingru(const void *proj, int ld, const float *bias, float *state, float *maps, void *out, const int *chunks, int n_chunks,
                           const int *seq_start, const int *seq_pos0, const int *seq_slot, int n_seqs, int n_short, int cols, int dtype,
                           b200_stream_t stream) {
    B200_REQUIRE(proj && state && out && seq_start && seq_pos0 && seq_slot, "mingru: null pointer");
    B200_REQUIRE(n_chunks == 0 || (chunks && maps && ((uintptr_t)chunks & 15) == 0), "mingru: chunk list / chunk maps missing or not 16-byte aligned");
    B200_REQUIRE(cols > 0 && ld >= 3 * cols && n_seqs >= 0 && n_chunks >= 0 && n_short >= 0, "mingru: bad shape");
    return launch_mingru(dtype, proj, ld, bias, state, maps, out, chunks, n_chunks, seq_start, seq_pos0, seq_slot, n_seqs, n_short, cols, as_stream(stream));
}
