// Paged softmax attention with options that the specialised kernels do not take: value heads of another size than
// the keys', a capped score, a logarithmic or linear distance penalty, first tokens that stay visible behind a sliding
// window, whole blocks of tokens seen as one key and value in front of it, a sink in the softmax's denominator, and a sigmoid gate per head on the output. Prompt portions and decoded tokens
// run through the same kernel: one block per (token, key/value head) that serves the group's query heads.
//
// Token i of a request sees key j iff j <= i and (window == 0 or i - j < window or j < keep_first). For head h:
//   s_j = (q . k_j) * scale;  s_j <- cap * tanh(s_j / cap) if cap > 0;  s_j <- s_j - r1_h * ln(1 + r2_h * (i - j)) if r1;
//   (with r1 alone, no r2: s_j <- s_j - r1_h * (i - j));
//   p_j = exp(s_j) / (sink + sum_j' exp(s_j'));  out = out_scale * sigmoid(gate_h) * sum_j p_j v_j.
// The sink is exp(0), or exp(sinks[h]) where a learned logit per head is given. The output's rows have a pitch of
// their own (ldo elements), so a layer may write its heads into a part of a wider row.
// With blocks of P tokens (a window, nothing kept, no penalty): besides the window, token i sees every block b with
// (b + 1) P - 1 <= i - window as one key and one value, the means that pool_blocks made, in the same softmax. Blocks have
// pages and a block table of their own: a block lies in the page of its last token, in the order of the blocks that end
// in that page.
// Scores, weights and sums are float32. The visible keys are walked in tiles of kTile keys whose borders are
// multiples of kTile counted from position 0 (the kept first tokens come first), so what a token computes, and in
// which order, depends on its position only: not on how the prompt was cut or on what else is in the batch.
#include "common.cuh"

using namespace akas;

namespace {

constexpr int kTile = 128;    // keys per tile = threads per block
constexpr int kMaxGroup = 16;  // query heads of a key/value head that one block serves at a time

// The factor on the queries of a position: 1 + coef ln(floor((pos + 1) / every) + 1); every 0: none.
__device__ __forceinline__ float temperature_of(int pos, float coef, int every) {
  return every > 0 ? fmaf(coef, logf((float)((pos + 1) / every) + 1.f), 1.f) : 1.f;
}

// One block per token: RMSNorm of every head of q and k over D with a plain weight (or none), then (where tables are
// given) the rotation of the first `rot` channels of each head by the token's angles, channel 2i with 2i + 1
// (interleaved) or i with i + rot / 2; q to q_out [N, H * D], k and the untouched v into the pages at the token's
// (page, offset). v may be the very rows of k: the values are then the keys as projected, before the rotation.
// Where biases are given (float32, one per channel of q, k, v), they are added first, in float32; q, k and v may then
// be the float32 result of a product (TI) while the pages hold T, so product plus bias is rounded once.
// unit: there is no norm in front of the rotation; behind it every head of q and k is divided by
// sqrt(mean of its D squares + eps), without a weight. temp_every > 0: last of all, q times its position's temperature.
template <typename TI, typename T>
__global__ void qk_norm_store_kernel(const TI* __restrict__ q, long long ldq, const TI* __restrict__ k, long long ldk,
                                     const TI* __restrict__ v, long long ldv, const float* __restrict__ qw,
                                     const float* __restrict__ kw, float eps, T* __restrict__ q_out,
                                     T* __restrict__ k_pool, T* __restrict__ v_pool, const int* __restrict__ block_table,
                                     int max_blocks, const int* __restrict__ seq_of_token,
                                     const int* __restrict__ positions, int page_size, int H, int G, int D, int V, int write,
                                     const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                                     int interleaved, const float* __restrict__ qb, const float* __restrict__ kb,
                                     const float* __restrict__ vb, int unit, float temp_coef, int temp_every) {
  const int n = blockIdx.x;
  const int req = seq_of_token[n];
  if (req < 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const int pos = positions[n];
  const int page = block_table[(size_t)req * max_blocks + pos / page_size];
  const int off = pos % page_size;
  const float temp = temperature_of(pos, temp_coef, temp_every);
  for (int head = warp; head < H + G; head += warps) {
    const bool is_q = head < H;
    if (!is_q && !write) continue;
    const TI* src = is_q ? q + (size_t)n * ldq + (size_t)head * D : k + (size_t)n * ldk + (size_t)(head - H) * D;
    const float* w = is_q ? qw : kw;
    const float* bias = is_q ? (qb != nullptr ? qb + (size_t)head * D : nullptr) : (kb != nullptr ? kb + (size_t)(head - H) * D : nullptr);
    auto at = [&](int d) { return bias != nullptr ? to_f32(src[d]) + bias[d] : to_f32(src[d]); };
    float inv = 1.f;
    if (unit) {
      // the squares of the rotated channels as the rotation leaves them (its tables may carry an amplitude)
      float ss = 0.f;
      const int turned = cos_t != nullptr ? rot : 0, half = turned / 2;
      for (int i = lane; i < half; i += 32) {
        const float u = at(interleaved ? 2 * i : i), x = at(interleaved ? 2 * i + 1 : i + half);
        const float c = cos_t[(size_t)n * half + i], sn = sin_t[(size_t)n * half + i];
        const float ru = fmaf(u, c, -x * sn), rx = fmaf(x, c, u * sn);
        ss = fmaf(ru, ru, fmaf(rx, rx, ss));
      }
      for (int d = turned + lane; d < D; d += 32) { const float x = at(d); ss = fmaf(x, x, ss); }
      inv = 1.f / sqrtf(warp_sum(ss) / (float)D + eps);
    } else if (w != nullptr) {
      float ss = 0.f;
      for (int d = lane; d < D; d += 32) { const float x = at(d); ss = fmaf(x, x, ss); }
      ss = warp_sum(ss);
      inv = 1.f / sqrtf(ss / (float)D + eps);
    }
    const float last = is_q ? temp : 1.f;
    T* dst = is_q ? q_out + ((size_t)n * H + head) * D
                  : k_pool + (((size_t)page * G + (head - H)) * page_size + off) * D;
    if (cos_t == nullptr) {
      for (int d = lane; d < D; d += 32) dst[d] = from_f32<T>((w != nullptr ? at(d) * inv * w[d] : unit ? at(d) * inv : at(d)) * last);
      continue;
    }
    const int half = rot / 2;
    for (int i = lane; i < half; i += 32) {
      const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
      float u = at(a), x = at(b);
      if (w != nullptr) { u *= inv * w[a]; x *= inv * w[b]; }
      const float c = cos_t[(size_t)n * half + i], sn = sin_t[(size_t)n * half + i];
      const float ru = fmaf(u, c, -x * sn), rx = fmaf(x, c, u * sn);
      dst[a] = from_f32<T>((unit ? ru * inv : ru) * last);
      dst[b] = from_f32<T>((unit ? rx * inv : rx) * last);
    }
    for (int d = rot + lane; d < D; d += 32) dst[d] = from_f32<T>((w != nullptr ? at(d) * inv * w[d] : unit ? at(d) * inv : at(d)) * last);
  }
  if (write) {
    for (int i = threadIdx.x; i < G * V; i += blockDim.x) {
      const int g = i / V, j = i % V;
      const float x = to_f32(v[(size_t)n * ldv + i]);
      v_pool[(((size_t)page * G + g) * page_size + off) * V + j] = from_f32<T>(vb != nullptr ? x + vb[i] : x);
    }
  }
}

// The same for head sizes that are multiples of 8 (at most 256), rotate-half pairs and a rotary width that is a multiple
// of 16, everything on 16 bytes: a thread owns 8 neighbouring channels of a head (LPH threads, D / 8 rounded up to a
// power of two, share one; those past D / 8 only shuffle, as do those past the last head) and reads its rotation partner's 8 channels itself; the
// threads behind the heads' copy the values. A token's heads are spread over gridDim.y blocks.
template <typename TI, typename T>
__global__ void __launch_bounds__(128)
qk_norm_store8_kernel(const TI* __restrict__ q, long long ldq, const TI* __restrict__ k, long long ldk, const TI* __restrict__ v,
                      long long ldv, const float* __restrict__ qw, const float* __restrict__ kw, float eps, T* __restrict__ q_out,
                      T* __restrict__ k_pool, T* __restrict__ v_pool, const int* __restrict__ block_table, int max_blocks,
                      const int* __restrict__ seq_of_token, const int* __restrict__ positions, int page_size, int H, int G, int D,
                      int V, int write, const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                      const float* __restrict__ qb, const float* __restrict__ kb, const float* __restrict__ vb, int unit, int lph,
                      float temp_coef, int temp_every) {
  const int n = blockIdx.x;
  const int req = seq_of_token[n];
  if (req < 0) return;
  const int item = blockIdx.y * blockDim.x + threadIdx.x;
  const int heads = write ? H + G : H;
  const int head = item / lph, e0 = item % lph * 8;
  const bool turns = head < heads && e0 < D;
  const bool is_q = head < H;
  long long row = 0;  // the token's row in a pool of one head
  if (write && head >= H) {
    const int pos = positions[n];
    row = (long long)block_table[(size_t)req * max_blocks + pos / page_size] * G * page_size + pos % page_size;
  }
  float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  const int g = head - H;
  const float* w = is_q ? qw : kw;
  const TI* src = is_q ? q + (size_t)n * ldq + (size_t)head * D : k + (size_t)n * ldk + (size_t)g * D;
  const float* bias = is_q ? (qb != nullptr ? qb + (size_t)head * D : nullptr) : (kb != nullptr ? kb + (size_t)g * D : nullptr);
  auto channels = [&](int e, float (&out)[8]) {
    load8(src + e, out);
    if (bias != nullptr) {
      float b[8];
      load8(bias + e, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) out[i] += b[i];
    }
  };
  // one over the root mean square of the head; every lane of the warp takes part (those without channels hold zeros)
  auto inverse_rms = [&]() {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss = fmaf(x[i], x[i], ss);
    for (int o = lph / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    return 1.f / sqrtf(ss / (float)D + eps);
  };
  auto weigh = [&](int e, float inv, float (&out)[8]) {
    float wv[8];
    load8(w + e, wv);
#pragma unroll
    for (int i = 0; i < 8; ++i) out[i] *= inv * wv[i];
  };
  if (turns) channels(e0, x);
  float inv = 1.f;
  if (qw != nullptr) {
    inv = inverse_rms();
    if (turns) weigh(e0, inv, x);
  }
  if (cos_t != nullptr && turns && e0 < rot) {
    const int half = rot / 2;
    const bool low = e0 < half;
    const int p0 = low ? e0 + half : e0 - half, f0 = low ? e0 : e0 - half;
    float other[8], c[8], sn[8];
    channels(p0, other);
    if (qw != nullptr) weigh(p0, inv, other);
    load8(cos_t + (size_t)n * half + f0, c);
    load8(sin_t + (size_t)n * half + f0, sn);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = low ? fmaf(x[i], c[i], -other[i] * sn[i]) : fmaf(x[i], c[i], other[i] * sn[i]);
  }
  if (unit) {
    inv = inverse_rms();
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] *= inv;
  }
  if (turns && is_q && temp_every > 0) {
    const float temp = temperature_of(positions[n], temp_coef, temp_every);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] *= temp;
  }
  if (turns) {
    if (is_q) store8(q_out + ((size_t)n * H + head) * D + e0, x);
    else store8(k_pool + (row + (long long)g * page_size) * D + e0, x);
    return;
  }
  const int at = item - heads * lph;  // the values: 8 channels a thread
  if (write && at >= 0 && at * 8 < G * V) {
    const int c = at * 8, vg = c / V, j = c % V;
    float y[8];
    load8(v + (size_t)n * ldv + c, y);
    if (vb != nullptr) {
      float b[8];
      load8(vb + c, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] += b[i];
    }
    store8(v_pool + (row + (long long)vg * page_size) * V + j, y);
  }
}

// One block per token of the step; those of a token that is the last of its block of `block` tokens make the block's key
// and value per head, the means of its tokens' rows as the pages hold them (float32 sums in the order of the positions),
// in the block's entry of its own pages. A block that began in earlier steps is read from where they left it.
template <typename T>
__global__ void __launch_bounds__(128)
pool_blocks_kernel(const T* __restrict__ k_pool, const T* __restrict__ v_pool, T* __restrict__ k_blocks, T* __restrict__ v_blocks,
                   const int* __restrict__ token_table, int token_width, const int* __restrict__ block_table, int block_width,
                   const int* __restrict__ seq_of_token, const int* __restrict__ positions, int page_size, int block_page,
                   int entries, int block, int G, int D, int V) {
  const int n = blockIdx.x;
  const int req = seq_of_token[n];
  if (req < 0) return;
  const int pos = positions[n];
  if ((pos + 1) % block) return;
  const int* table = token_table + (size_t)req * token_width;
  const int page = block_table[(size_t)req * block_width + pos / block_page];
  const int entry = pos / block - (pos / block_page * block_page) / block;
  const float inv = 1.f / (float)block;
  const int first = pos - block + 1, per = D + V;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < G * per; i += gridDim.y * blockDim.x) {
    const int g = i / per, e = i % per;
    const T* src = e < D ? k_pool + e : v_pool + (e - D);
    const int size = e < D ? D : V;
    float sum = 0.f;
#pragma unroll 8
    for (int t = first; t <= pos; ++t) {
      const long long row = ((long long)table[t / page_size] * G + g) * page_size + t % page_size;
      sum += to_f32(src[row * size]);
    }
    const long long row = ((long long)page * G + g) * entries + entry;
    if (e < D) k_blocks[row * D + e] = from_f32<T>(sum * inv);
    else v_blocks[row * V + (e - D)] = from_f32<T>(sum * inv);
  }
}

// The same for head sizes that are multiples of 8, everything on 16 bytes: a thread owns 8 neighbouring channels of a
// head's key or value and asks for up to 16 of the block's rows before it adds the first. A grid block looks at kPoolTokens
// neighbouring tokens, so that a step of many tokens is not a launch of as many blocks most of which end at once.
constexpr int kPoolTokens = 8;

template <typename T>
__global__ void __launch_bounds__(64)
pool_blocks8_kernel(const T* __restrict__ k_pool, const T* __restrict__ v_pool, T* __restrict__ k_blocks, T* __restrict__ v_blocks,
                    const int* __restrict__ token_table, int token_width, const int* __restrict__ block_table, int block_width,
                    const int* __restrict__ seq_of_token, const int* __restrict__ positions, int page_size, int block_page,
                    int entries, int block, int G, int D, int V, int N) {
  constexpr int ROWS = sizeof(T) == 2 ? 16 : 8;  // rows in flight
  __shared__ int last[kPoolTokens], owner[kPoolTokens];
  if (threadIdx.x < kPoolTokens) {
    const int n = blockIdx.x * kPoolTokens + threadIdx.x;
    const int req = n < N ? seq_of_token[n] : -1;
    const int pos = n < N ? positions[n] : 0;
    last[threadIdx.x] = pos;
    owner[threadIdx.x] = (pos + 1) % block == 0 ? req : -1;
  }
  __syncthreads();
  const int per = (D + V) / 8;
  const int i = blockIdx.y * blockDim.x + threadIdx.x;
  if (i >= G * per) return;
  const int g = i / per, e = i % per * 8;
  const bool key = e < D;
  const T* src = key ? k_pool + e : v_pool + (e - D);
  const int size = key ? D : V;
  const float inv = 1.f / (float)block;
  for (int u = 0; u < kPoolTokens; ++u) {
    const int req = owner[u], pos = last[u];
    if (req < 0) continue;
    const int* table = token_table + (size_t)req * token_width;
    const int page = block_table[(size_t)req * block_width + pos / block_page];
    float sum[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int t0 = pos - block + 1; t0 <= pos; t0 += ROWS) {
      uint4 raw[ROWS][sizeof(T) / 2];
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int t = min(t0 + r, pos);
        const long long row = ((long long)table[t / page_size] * G + g) * page_size + t % page_size;
#pragma unroll
        for (int h = 0; h < (int)sizeof(T) / 2; ++h) raw[r][h] = reinterpret_cast<const uint4*>(src + row * size)[h];
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        if (t0 + r <= pos) {
          float x[8];
          load8(reinterpret_cast<const T*>(&raw[r][0]), x);
#pragma unroll
          for (int c = 0; c < 8; ++c) sum[c] += x[c];
        }
      }
    }
#pragma unroll
    for (int c = 0; c < 8; ++c) sum[c] *= inv;
    const long long row = ((long long)page * G + g) * entries + pos / block - (pos / block_page * block_page) / block;
    if (key) store8(k_blocks + row * D + e, sum);
    else store8(v_blocks + row * V + (e - D), sum);
  }
}

// The blocks that a layer sees in front of its window (block 0: none): their pages, the block table with its width, the
// tokens and the entries of a page, and the tokens of a block.
template <typename T>
struct Blocks {
  const T* k;
  const T* v;
  const int* table;
  int width, page, entries, block;
};

// Scores of one key row against `heads` query rows in shared memory: the row is read once, 16 bytes at a time where
// its size allows, and every head's sum is one ascending chain of fused multiply-adds.
template <typename T>
__device__ __forceinline__ void dot_rows(const T* __restrict__ krow, const float* __restrict__ qs, int D, int heads,
                                         float (&acc)[kMaxGroup]) {
  constexpr int N = Vec<T>::N;
#pragma unroll
  for (int a = 0; a < kMaxGroup; ++a) acc[a] = 0.f;
  int d = 0;
  if ((D * (int)sizeof(T)) % 16 == 0) {
    for (; d + N <= D; d += N) {
      float kv[N];
      load_vec(krow + d, kv);
#pragma unroll
      for (int a = 0; a < kMaxGroup; ++a) {
        if (a < heads) {
#pragma unroll
          for (int e = 0; e < N; ++e) acc[a] = fmaf(qs[a * D + d + e], kv[e], acc[a]);
        }
      }
    }
  }
  for (; d < D; ++d) {
    const float kv = to_f32(krow[d]);
#pragma unroll
    for (int a = 0; a < kMaxGroup; ++a)
      if (a < heads) acc[a] = fmaf(qs[a * D + d], kv, acc[a]);
  }
}

// One block of kTile threads per (token, key/value head). In a tile, thread t owns key t: it computes the scores
// of its key for the group's heads (the key row is read once), the block finds the tile's maxima, and then thread
// c owns value channel c (c, c + kTile, ...) and adds the tile's weighted values to its running sums.
template <typename T, typename TG>
__global__ void __launch_bounds__(kTile)
attention_general_kernel(const T* __restrict__ q, const T* __restrict__ k_pool, const T* __restrict__ v_pool,
                         const int* __restrict__ block_table, int max_blocks, const int* __restrict__ seq_of_token,
                         const int* __restrict__ positions, T* __restrict__ out, float scale, int window, int keep_first,
                         float cap, const float* __restrict__ r1, const float* __restrict__ r2, int sink,
                         const TG* __restrict__ gate, long long ldg, int page_size, int H, int G, int D, int V, int row_words,
                         const float* __restrict__ sinks, float out_scale, long long ldo, long long vpitch, int gate_channels,
                         Blocks<T> blocks) {
  extern __shared__ __align__(16) float smem[];
  const int n = blockIdx.x, g = blockIdx.y;
  const int req = seq_of_token[n];
  if (req < 0) return;
  const int group = H / G;
  const int pos = positions[n];
  const int lo = window > 0 ? max(0, pos - window + 1) : 0;  // first key of the window
  const int kept = window > 0 ? min(keep_first, lo) : 0;      // keys [0, kept) stay visible behind it
  const int* table = block_table + (size_t)req * max_blocks;
  const int tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;

  for (int h0 = 0; h0 < group; h0 += kMaxGroup) {
    const int heads = min(kMaxGroup, group - h0);
    float* qs = smem;                        // [heads][D]
    float* pw = qs + kMaxGroup * D;          // [heads][kTile] weights of the tile
    float* red = pw + kMaxGroup * kTile;     // [kMaxGroup][4] maxima / sums of the warps
    float* stat = red + kMaxGroup * 4;       // [kMaxGroup][2]: running maximum, correction of this tile
    long long* rowbase = reinterpret_cast<long long*>(smem + row_words);  // [kTile] row of each key of the tile in the pools
    __syncthreads();
    for (int i = tid; i < heads * D; i += kTile)
      qs[i] = to_f32(q[((size_t)n * H + (size_t)g * group + h0) * D + i]);
    float m_run[kMaxGroup], l_run[kMaxGroup];
#pragma unroll
    for (int a = 0; a < kMaxGroup; ++a) {
      m_run[a] = sinks != nullptr ? sinks[g * group + h0 + min(a, heads - 1)] : sink ? 0.f : -INFINITY;
      l_run[a] = sinks != nullptr || sink ? 1.f : 0.f;
    }
    // running sums of value channel c = tid + kTile * i for every head: kept in shared memory (any V), thread-private
    float* acc = stat + kMaxGroup * 2;  // [kMaxGroup][Vp], Vp = V rounded up to kTile
    const int Vp = (V + kTile - 1) / kTile * kTile;
    for (int i = tid; i < heads * Vp; i += kTile) acc[i] = 0.f;
    __syncthreads();

    // the runs of visible keys: [0, kept), [lo, pos] and the blocks in front of the window; tiles start at multiples of kTile
    const int runs = blocks.block > 0 ? 3 : 2;
    for (int run = 0; run < runs; ++run) {
      const bool pooled = run == 2;
      const int first = run == 1 ? lo : 0, last = run == 0 ? kept : run == 1 ? pos + 1 : lo / blocks.block;  // [first, last)
      if (first >= last) continue;
      const T* keys = pooled ? blocks.k : k_pool;
      const T* values = pooled ? blocks.v : v_pool;
      const long long pitch = pooled ? V : vpitch;
      for (int t0 = first / kTile * kTile; t0 < last; t0 += kTile) {
        const int key = t0 + tid;
        const bool seen = key >= first && key < last;
        float sc[kMaxGroup];
        if (seen) {
          long long base;
          if (pooled) {
            const int at = (key * blocks.block + blocks.block - 1) / blocks.page;  // the page of the block's last token
            base = ((long long)blocks.table[(size_t)req * blocks.width + at] * G + g) * blocks.entries + key - at * blocks.page / blocks.block;
          } else {
            base = ((long long)table[key / page_size] * G + g) * page_size + key % page_size;
          }
          rowbase[tid] = base;
          const float dist = (float)(pos - key);
          dot_rows(keys + (size_t)base * D, qs, D, heads, sc);
#pragma unroll
          for (int a = 0; a < kMaxGroup; ++a) {
            if (a < heads) {
              float s = sc[a] * scale;
              if (cap > 0.f) s = cap * tanhf(s / cap);
              if (r1 != nullptr) {
                const int h = g * group + h0 + a;
                s -= r2 != nullptr ? r1[h] * log1pf(r2[h] * dist) : r1[h] * dist;
              }
              sc[a] = s;
            }
          }
        }
        // maxima of the tile, per head
#pragma unroll
        for (int a = 0; a < kMaxGroup; ++a) {
          if (a < heads) {
            const float mx = warp_max(seen ? sc[a] : -INFINITY);
            if (lane == 0) red[a * 4 + warp] = mx;
          }
        }
        __syncthreads();
#pragma unroll
        for (int a = 0; a < kMaxGroup; ++a) {
          if (a < heads) {
            const float tile_max = fmaxf(fmaxf(red[a * 4], red[a * 4 + 1]), fmaxf(red[a * 4 + 2], red[a * 4 + 3]));
            const float m_new = fmaxf(m_run[a], tile_max);
            const float corr = m_run[a] == -INFINITY ? 0.f : expf(m_run[a] - m_new);
            const float p = seen ? expf(sc[a] - m_new) : 0.f;
            pw[a * kTile + tid] = p;
            m_run[a] = m_new;
            l_run[a] *= corr;
            if (tid == 0) stat[a * 2 + 1] = corr;
            sc[a] = p;
          }
        }
        __syncthreads();  // weights written, maxima read
        // sums of the weights: every thread adds the tile's weights in the same order, so all agree
#pragma unroll
        for (int a = 0; a < kMaxGroup; ++a) {
          if (a < heads) {
            const float part = warp_sum(sc[a]);
            if (lane == 0) red[a * 4 + warp] = part;
          }
        }
        // weighted values: thread c walks the tile's keys
        const int count = min(kTile, last - t0);
        const int begin = max(0, first - t0);
        for (int c = tid; c < V; c += kTile) {
          float add[kMaxGroup];
#pragma unroll
          for (int a = 0; a < kMaxGroup; ++a) add[a] = 0.f;
#pragma unroll 8
          for (int t = begin; t < count; ++t) {  // (the rows' places were found with the scores: these loads do not wait on one another)
            const float vv = to_f32(values[(size_t)rowbase[t] * pitch + c]);
#pragma unroll
            for (int a = 0; a < kMaxGroup; ++a)
              if (a < heads) add[a] = fmaf(pw[a * kTile + t], vv, add[a]);
          }
#pragma unroll
          for (int a = 0; a < kMaxGroup; ++a)
            if (a < heads) acc[a * Vp + c] = fmaf(acc[a * Vp + c], stat[a * 2 + 1], add[a]);
        }
        __syncthreads();  // sums of the warps written; weights and corrections read
#pragma unroll
        for (int a = 0; a < kMaxGroup; ++a)
          if (a < heads) l_run[a] += (red[a * 4] + red[a * 4 + 1]) + (red[a * 4 + 2] + red[a * 4 + 3]);
        __syncthreads();
      }
    }
    for (int c = tid; c < V; c += kTile) {
#pragma unroll
      for (int a = 0; a < kMaxGroup; ++a) {
        if (a < heads) {
          const int h = g * group + h0 + a;
          float o = l_run[a] > 0.f ? acc[a * Vp + c] / l_run[a] : 0.f;
          // one logit per head, or (gate_channels) one per channel of the token's output row
          if (gate != nullptr) o *= 1.f / (1.f + expf(-to_f32(gate[(size_t)n * ldg + (gate_channels ? (size_t)h * V + c : (size_t)h)])));
          out[(size_t)n * ldo + (size_t)h * V + c] = from_f32<T>(o * out_scale);
        }
      }
    }
  }
}

}  // namespace

AKAS_API int akas_qk_norm_store(const void* q, long long ldq, const void* k, long long ldk, const void* v, long long ldv,
                                const float* qw, const float* kw, float eps, void* q_out, void* k_pool, void* v_pool,
                                const int* block_table, int max_blocks, const int* seq_of_token, const int* positions,
                                int page_size, int N, int H, int G, int D, int V, int write, int dtype, const float* cos_t,
                                const float* sin_t, int rot, int interleaved, int in_dtype, const float* qb, const float* kb,
                                const float* vb, int unit, float temp_coef, int temp_every, cudaStream_t stream) {
  if (N <= 0) return 0;
  if (unit && (qw != nullptr || kw != nullptr)) return (int)cudaErrorInvalidValue;
  if ((qw == nullptr) != (kw == nullptr)) return (int)cudaErrorInvalidValue;
  const uintptr_t bases = (uintptr_t)q | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)qw | (uintptr_t)kw |
                          (uintptr_t)cos_t | (uintptr_t)sin_t | (uintptr_t)qb | (uintptr_t)kb | (uintptr_t)vb |
                          (write ? (uintptr_t)k | (uintptr_t)v : 0);
  if (D % 8 == 0 && D <= 256 && V % 8 == 0 && (cos_t == nullptr || (!interleaved && rot % 16 == 0)) && bases % 16 == 0 && ldq % 8 == 0 &&
      (!write || (ldk % 8 == 0 && ldv % 8 == 0))) {
    int lph = 1;
    while (lph < D / 8) lph *= 2;
    const int threads = (write ? H + G : H) * lph + (write ? G * (V / 8) : 0);
    const dim3 grid(N, (threads + 127) / 128);
#define AKAS_STORE8(TI, T)                                                                                                    \
  return launch_ordinary(qk_norm_store8_kernel<TI, T>, grid, dim3(128), 0, stream, (const TI*)q, ldq, (const TI*)k, ldk,      \
                         (const TI*)v, ldv, qw, kw, eps, (T*)q_out, (T*)k_pool, (T*)v_pool, block_table, max_blocks,          \
                         seq_of_token, positions, page_size, H, G, D, V, write, cos_t, sin_t, rot, qb, kb, vb, unit, lph,     \
                         temp_coef, temp_every)
    if (dtype == AKAS_F32) AKAS_STORE8(float, float);
    if (in_dtype == AKAS_F32) AKAS_STORE8(float, bf16);
    AKAS_STORE8(bf16, bf16);
#undef AKAS_STORE8
  }
  if (cos_t != nullptr && (rot <= 0 || rot % 2 || rot > D)) return (int)cudaErrorInvalidValue;
  if (dtype == AKAS_F32 && in_dtype != AKAS_F32) return (int)cudaErrorInvalidValue;
  if (dtype == AKAS_F32)
    return launch_ordinary(qk_norm_store_kernel<float, float>, dim3(N), dim3(128), 0, stream, (const float*)q, ldq, (const float*)k, ldk,
                          (const float*)v, ldv, qw, kw, eps, (float*)q_out, (float*)k_pool, (float*)v_pool, block_table,
                          max_blocks, seq_of_token, positions, page_size, H, G, D, V, write, cos_t, sin_t, rot, interleaved, qb, kb, vb, unit, temp_coef, temp_every);
  if (in_dtype == AKAS_F32)
    return launch_ordinary(qk_norm_store_kernel<float, bf16>, dim3(N), dim3(128), 0, stream, (const float*)q, ldq, (const float*)k, ldk,
                          (const float*)v, ldv, qw, kw, eps, (bf16*)q_out, (bf16*)k_pool, (bf16*)v_pool, block_table, max_blocks,
                          seq_of_token, positions, page_size, H, G, D, V, write, cos_t, sin_t, rot, interleaved, qb, kb, vb, unit, temp_coef, temp_every);
  return launch_ordinary(qk_norm_store_kernel<bf16, bf16>, dim3(N), dim3(128), 0, stream, (const bf16*)q, ldq, (const bf16*)k, ldk,
                        (const bf16*)v, ldv, qw, kw, eps, (bf16*)q_out, (bf16*)k_pool, (bf16*)v_pool, block_table, max_blocks,
                        seq_of_token, positions, page_size, H, G, D, V, write, cos_t, sin_t, rot, interleaved, qb, kb, vb, unit, temp_coef, temp_every);
}

template <typename T, typename TG>
static int launch_general(const void* q, const void* k_pool, const void* v_pool, const int* block_table, int max_blocks,
                          const int* seq_of_token, const int* positions, void* out, float scale, int window, int keep_first,
                          float cap, const float* r1, const float* r2, int sink, const void* gate, long long ldg,
                          int page_size, int N, int H, int G, int D, int V, const float* sinks, float out_scale,
                          long long ldo, long long vpitch, int gate_channels, const void* k_blocks, const void* v_blocks,
                          const int* blocks_table, int blocks_width, int block_page, int block, cudaStream_t stream) {
  const int Vp = (V + kTile - 1) / kTile * kTile;
  const int row_words = (kMaxGroup * D + kMaxGroup * kTile + kMaxGroup * 4 + kMaxGroup * 2 + kMaxGroup * Vp + 1) / 2 * 2;
  const size_t smem = sizeof(float) * (size_t)row_words + sizeof(long long) * kTile;
  if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
  static size_t allowed[64] = {};
  int device = 0;
  cudaGetDevice(&device);
  if (smem > 48 * 1024 && device < 64 && allowed[device] < smem) {
    const cudaError_t e = cudaFuncSetAttribute(attention_general_kernel<T, TG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed[device] = smem;
  }
  return launch_ordinary(attention_general_kernel<T, TG>, dim3(N, G), dim3(kTile), smem, stream, (const T*)q, (const T*)k_pool,
                        (const T*)v_pool, block_table, max_blocks, seq_of_token, positions, (T*)out, scale, window, keep_first,
                        cap, r1, r2, sink, (const TG*)gate, ldg, page_size, H, G, D, V, row_words, sinks, out_scale, ldo, vpitch, gate_channels,
                        Blocks<T>{(const T*)k_blocks, (const T*)v_blocks, blocks_table, blocks_width, block_page,
                                  block > 0 ? (block_page + block - 1) / block : 0, block});
}

AKAS_API int akas_attention_general(const void* q, const void* k_pool, const void* v_pool, const int* block_table,
                                    int max_blocks, const int* seq_of_token, const int* positions, void* out, float scale,
                                    int window, int keep_first, float cap, const float* r1, const float* r2, int sink,
                                    const void* gate, long long ldg, int page_size, int N, int H, int G, int D, int V,
                                    int dtype, const float* sinks, float out_scale, long long ldo, long long vpitch,
                                    int gate_channels, int gate_dtype, const void* k_blocks, const void* v_blocks,
                                    const int* blocks_table, int blocks_width, int block_page, int block, cudaStream_t stream) {
  if (N <= 0) return 0;
  if (G <= 0 || H % G || vpitch < V) return (int)cudaErrorInvalidValue;
  // blocks: a window in front of which they lie, and none of the options that the walk over them does not know
  if (block < 0 || (block > 0 && (window <= 0 || keep_first > 0 || r1 != nullptr || block_page <= 0 || k_blocks == nullptr ||
                                  v_blocks == nullptr || blocks_table == nullptr)))
    return (int)cudaErrorInvalidValue;
  if (dtype == AKAS_BF16 && gate != nullptr && gate_dtype == AKAS_F32)  // the gate's logits as a float32 product left them
    return launch_general<bf16, float>(q, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions, out, scale, window,
                                       keep_first, cap, r1, r2, sink, gate, ldg, page_size, N, H, G, D, V, sinks, out_scale, ldo, vpitch, gate_channels, k_blocks, v_blocks,
                                        blocks_table, blocks_width, block_page, block, stream);
  if (dtype == AKAS_F32 && gate != nullptr && gate_dtype != AKAS_F32) return (int)cudaErrorInvalidValue;
  if (dtype == AKAS_F32)
    return launch_general<float, float>(q, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions, out, scale, window,
                                        keep_first, cap, r1, r2, sink, gate, ldg, page_size, N, H, G, D, V, sinks, out_scale, ldo, vpitch, gate_channels, k_blocks, v_blocks,
                                        blocks_table, blocks_width, block_page, block, stream);
  return launch_general<bf16, bf16>(q, k_pool, v_pool, block_table, max_blocks, seq_of_token, positions, out, scale, window,
                                    keep_first, cap, r1, r2, sink, gate, ldg, page_size, N, H, G, D, V, sinks, out_scale, ldo, vpitch, gate_channels, k_blocks, v_blocks,
                                        blocks_table, blocks_width, block_page, block, stream);
}

// The means of every block of `block` tokens that a token of this step completes; block_page: tokens of a page of the
// blocks' pools, whose pages hold ceil(block_page / block) entries.
AKAS_API int akas_pool_blocks(const void* k_pool, const void* v_pool, void* k_blocks, void* v_blocks, const int* token_table,
                              int token_width, const int* block_table, int block_width, const int* seq_of_token,
                              const int* positions, int page_size, int block_page, int block, int N, int G, int D, int V, int dtype,
                              cudaStream_t stream) {
  if (N <= 0) return 0;
  if (block <= 0 || block_page <= 0 || page_size <= 0) return (int)cudaErrorInvalidValue;
  const int entries = (block_page + block - 1) / block;
  const uintptr_t bases = (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)k_blocks | (uintptr_t)v_blocks;
  if (D % 8 == 0 && V % 8 == 0 && bases % 16 == 0) {
    const dim3 grid8((N + kPoolTokens - 1) / kPoolTokens, (G * ((D + V) / 8) + 63) / 64);
#define AKAS_POOL8(T)                                                                                                          \
  return launch_ordinary(pool_blocks8_kernel<T>, grid8, dim3(64), 0, stream, (const T*)k_pool, (const T*)v_pool, (T*)k_blocks, \
                         (T*)v_blocks, token_table, token_width, block_table, block_width, seq_of_token, positions, page_size, \
                         block_page, entries, block, G, D, V, N)
    if (dtype == AKAS_F32) AKAS_POOL8(float);
    AKAS_POOL8(bf16);
#undef AKAS_POOL8
  }
  const dim3 grid(N, max(1, min(16, (G * (D + V) + 127) / 128)));
  if (dtype == AKAS_F32)
    return launch_ordinary(pool_blocks_kernel<float>, grid, dim3(128), 0, stream, (const float*)k_pool, (const float*)v_pool,
                           (float*)k_blocks, (float*)v_blocks, token_table, token_width, block_table, block_width, seq_of_token,
                           positions, page_size, block_page, entries, block, G, D, V);
  return launch_ordinary(pool_blocks_kernel<bf16>, grid, dim3(128), 0, stream, (const bf16*)k_pool, (const bf16*)v_pool,
                         (bf16*)k_blocks, (bf16*)v_blocks, token_table, token_width, block_table, block_width, seq_of_token,
                         positions, page_size, block_page, entries, block, G, D, V);
}
