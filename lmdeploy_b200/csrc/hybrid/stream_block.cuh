// Kernels of blocks whose residual is `S` parallel streams: the normed embedding copied to every stream, and the join of a sublayer's
// output into all streams at once (a learned mix of the streams, a learned factor per stream, a scale per column) fused with the next
// sublayer's weighted read of the streams and its norm.
// Included by hybrid_ops.cu inside namespace b200h, after its helpers and normed_block.cuh (load_row / store_row).
//
// The streams of row t lie at x + t * S * width, one after another (float).

constexpr int kMaxStreams = 8;

// One block per row.  e = table[token] * scale;  with w_embed: e <- rms(e) * w_embed;  x_s = e for every stream;
// u = (sum_s read[s]) * e;  h = rms(u) * w_next as T.  The row stays in shared memory (width floats) between the passes, where a
// thread only meets its own values.
template <typename T, int V>
__global__ void __launch_bounds__(256) embed_streams_kernel(const int* __restrict__ tokens, const T* __restrict__ table, float scale,
                                                           const float* __restrict__ w_embed, float* __restrict__ x, int streams,
                                                           const float* __restrict__ read, const float* __restrict__ w_next, int width,
                                                           float eps, T* __restrict__ h)
{
    extern __shared__ __align__(16) float es_smem[];
    __shared__ float red[32];
    const size_t t = blockIdx.x;
    const T* row = table + (size_t)tokens[t] * width;
    float ss = 0.f, gain = 0.f;
    for (int s = 0; s < streams; ++s) gain += read[s];
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V];
        load_row<V>(row + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) { v[e] *= scale; ss = fmaf(v[e], v[e], ss); }
        store_row<V>(es_smem + i, v);
    }
    float r = 1.0f;
    if (w_embed) r = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    ss = 0.f;
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V];
        load_row<V>(es_smem + i, v);
        if (w_embed) {
            float w[V];
            load_row<V>(w_embed + i, w);
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = v[e] * r * w[e];
        }
        for (int s = 0; s < streams; ++s) store_row<V>(x + (t * streams + s) * width + i, v);
#pragma unroll
        for (int e = 0; e < V; ++e) { v[e] *= gain; ss = fmaf(v[e], v[e], ss); }
        store_row<V>(es_smem + i, v);
    }
    r = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
        float v[V], w[V];
        load_row<V>(es_smem + i, v);
        load_row<V>(w_next + i, w);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * r * w[e];
        store_row<V>(h + t * width + i, v);
    }
}

struct StreamJoin {
    const float* ls;          // [width] or nullptr: one
    const float* mix;         // [S, S], from stream s to stream t at [s * S + t]
    const float* out;         // [S]
    const float* read;        // [S] or nullptr: one
    const float* w_next;      // [width]
    const int* rows;          // the row each block takes, or nullptr: its own number
    int width;
    float eps;
};

// One block per row.  With y:  x_t <- sum_s mix[s, t] x_s + out[t] * (y * ls), all streams from the old ones, written back if `write`;
// then u = sum_s read[s] x_s -> u_out (float, at the block's number) and / or h = rms(u) * w_next as T (at the block's number).
// Shared memory: width floats where h is wanted.
template <typename T, int S, int V>
__global__ void __launch_bounds__(256) join_streams_kernel(float* __restrict__ x, const T* __restrict__ y, StreamJoin j, int write,
                                                          float* __restrict__ u_out, T* __restrict__ h)
{
    extern __shared__ __align__(16) float js_smem[];
    __shared__ float red[32];
    const size_t t = j.rows ? j.rows[blockIdx.x] : blockIdx.x, to = blockIdx.x;
    float mix[S][S], out[S], read[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        read[s] = j.read ? j.read[s] : 1.0f;
        out[s] = y ? j.out[s] : 0.f;
#pragma unroll
        for (int d = 0; d < S; ++d) mix[s][d] = y ? j.mix[s * S + d] : 0.f;
    }
    float* xr = x + t * S * j.width;
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < j.width; i += blockDim.x * V) {
        float v[S][V], u[V];
#pragma unroll
        for (int s = 0; s < S; ++s) load_row<V>(xr + (size_t)s * j.width + i, v[s]);
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = 0.f;
        if (y) {
            float a[V];
            load_row<V>(y + t * j.width + i, a);
            if (j.ls) {
                float l[V];
                load_row<V>(j.ls + i, l);
#pragma unroll
                for (int e = 0; e < V; ++e) a[e] *= l[e];
            }
#pragma unroll
            for (int d = 0; d < S; ++d) {
                float n[V];
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    n[e] = out[d] * a[e];
#pragma unroll
                    for (int s = 0; s < S; ++s) n[e] = fmaf(mix[s][d], v[s][e], n[e]);
                    u[e] = fmaf(read[d], n[e], u[e]);
                }
                if (write) store_row<V>(xr + (size_t)d * j.width + i, n);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s)
#pragma unroll
                for (int e = 0; e < V; ++e) u[e] = fmaf(read[s], v[s][e], u[e]);
        }
        if (u_out) store_row<V>(u_out + to * j.width + i, u);
        if (h) {
            store_row<V>(js_smem + i, u);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(u[e], u[e], ss);
        }
    }
    if (!h) return;
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)j.width + j.eps);
    for (int i = threadIdx.x * V; i < j.width; i += blockDim.x * V) {
        float v[V], w[V];
        load_row<V>(js_smem + i, v);
        load_row<V>(j.w_next + i, w);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = v[e] * r * w[e];
        store_row<V>(h + to * j.width + i, v);
    }
}
