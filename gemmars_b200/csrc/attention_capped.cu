// Softmax attention whose scores are capped, whose keys and values have different widths, and
// whose q, k and v pass a short causal filter over time before the rotation.  Plain kernels for
// any precision and size; the arithmetic for one (token, head) depends on its position and the
// cache alone, so prompts, parts of prompts and single tokens give the same bits.
//
//   gb_filter_rope_cache:  u [T, q | k | v] -> filter over time -> RMS norm of every q and k head
//                          with a weight over its dims (when weights are given) -> rotation of the
//                          first `rot` dims of every q and k head (dim i pairs with i + rot/2, or with
//                          `pairs` dim 2i with 2i + 1; angle float(pos) * inv_freq[i], float32; cosines
//                          and sines times `rot_mag`) -> with `unit_after` every q and k head divided by
//                          its root mean square (no weight) -> q times 1 + qt_coef ln(floor((pos + 1) /
//                          qt_every) + 1) (when qt_every) -> q rows, keys and values into pages.  With
//                          `v_from_k` the rows hold q | k only and a value head is its key head as
//                          projected and filtered, before norm and rotation
//   gb_attention_capped:   score = (q . k) * scale; score <- cap * tanh(score / cap) when cap > 0;
//                          keys lo..p with lo = max(0, p + 1 - window), and with `keep_first` the
//                          keys 0..keep_first-1 as well, wherever the window stands; softmax, whose
//                          denominator also holds exp(sink[head]) when sinks are given (a term
//                          without key or value); output times sigmoid(gate) * out_scale when a
//                          gate is given (a number per output channel, or with gate_per_head one
//                          per head)
//
// Cache layout as everywhere in the package: keys [pages, kv_heads, page_size, D], values
// transposed inside a page [pages, kv_heads, Vd, page_size].
#include "common.cuh"

constexpr int CHUNK = 128;
constexpr int MAX_TAPS = 8;
constexpr int VPT = 4;   // value dims a thread keeps: values up to VPT * CHUNK wide

template <typename T>
__device__ __forceinline__ float filtered(const T* __restrict__ u, long long ldu, int row0, int local,
                                          const float* __restrict__ hist, const float* __restrict__ taps, int C, int c, int K) {
  float acc = 0.f;
  for (int j = 0; j < K; ++j) {
    const int at = local - (K - 1) + j;
    const float in = at >= 0 ? to_f32(u[(size_t)(row0 + at) * ldu + c]) : hist[(size_t)(K - 1 + at) * C + c];
    acc = fmaf(taps[(size_t)c * K + j], in, acc);
  }
  return acc;
}

// One block per (token, head): the H query heads, then the G key heads, then the G value heads.
// A q or k head is filtered into shared memory first, a dim a thread, beside the cosines and sines
// of the token's angles; then every dim takes its partner from there (with each thread filtering
// its partner again and taking its own sine and cosine, the kernel was bound by instructions).
constexpr int MAX_HEAD = 512;

template <typename T>
__global__ void __launch_bounds__(128) filter_rope_cache_kernel(
    const T* __restrict__ u, long long ldu, const float* __restrict__ taps, const float* __restrict__ state, int K,
    const float* __restrict__ inv_freq, int rot, const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
    const int* __restrict__ seq_slot, const int* __restrict__ cu, const int* __restrict__ page_table, int table_width,
    int page_size, T* __restrict__ q_out, long long ldq, T* __restrict__ kcache, T* __restrict__ vcache, int H, int G, int D,
    int Vd, const float* __restrict__ q_norm, const float* __restrict__ k_norm, float norm_eps, float rot_mag, float qt_coef,
    int qt_every, int v_from_k, int pairs, int unit_after) {
  __shared__ float vals[MAX_HEAD], cs[MAX_HEAD];   // cs: cos[rot / 2], then sin[rot / 2]
  __shared__ float scratch[33];
  pdl_release_next();
  pdl_wait_prior();
  const int t = blockIdx.x, hh = blockIdx.y, b = tok_seq[t], pos = tok_pos[t], slot = seq_slot[b];
  const int row0 = cu[b], local = t - row0, half = rot / 2;
  const int C = (H + G) * D + (v_from_k ? 0 : G * Vd);
  const float* hist = K > 1 ? state + (size_t)slot * (K - 1) * C : nullptr;
  const int page = page_table ? page_table[(size_t)slot * table_width + (pos / page_size) % table_width] : 0;
  const int off = pos % page_size;
  if (hh >= H + G) {                  // a value head: filtered, then into its page (a dim's positions contiguous)
    if (!vcache) return;
    const int g = hh - H - G;
    for (int d = threadIdx.x; d < Vd; d += blockDim.x) {
      const int c = (v_from_k ? H * D : (H + G) * D) + g * Vd + d;
      const float val = K > 1 ? filtered(u, ldu, row0, local, hist, taps, C, c, K) : to_f32(u[(size_t)t * ldu + c]) * (K == 1 ? taps[c] : 1.f);
      vcache[(((size_t)page * G + g) * Vd + d) * page_size + off] = from_f32<T>(val);
    }
    return;
  }
  if (hh >= H && !kcache) return;
  const float* norm_w = hh < H ? q_norm : k_norm;
  float ss = 0.f;
  for (int i = threadIdx.x; i < D; i += blockDim.x) {
    const int e = hh * D + i;
    const float x = K > 1 ? filtered(u, ldu, row0, local, hist, taps, C, e, K) : to_f32(u[(size_t)t * ldu + e]) * (K == 1 ? taps[e] : 1.f);
    vals[i] = x;
    ss = fmaf(x, x, ss);
    if (i < half) {
      float sn, cn;
      sincosf((float)pos * inv_freq[i], &sn, &cn);
      cs[half + i] = sn * rot_mag;
      cs[i] = cn * rot_mag;
    }
  }
  if (norm_w) {            // the head divided by its root mean square, times the weight of each dim
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)D + norm_eps);
    for (int i = threadIdx.x; i < D; i += blockDim.x) vals[i] = vals[i] * inv * norm_w[i];
  }
  __syncthreads();
  const float temper = (hh < H && qt_every > 0) ? 1.0f + qt_coef * logf((float)((pos + 1) / qt_every + 1)) : 1.0f;
  float turned[MAX_HEAD / 128], ss_after = 0.f;
#pragma unroll
  for (int u = 0; u < MAX_HEAD / 128; ++u) {
    const int i = threadIdx.x + u * 128;
    if (i >= D) break;
    float val = vals[i];
    if (i < rot) {
      // the pair (a, b) = (dim j, dim j + half), or (2j, 2j + 1), becomes (a cos - b sin, b cos + a sin)
      const bool first = pairs ? (i & 1) == 0 : i < half;
      const int j = pairs ? i >> 1 : (first ? i : i - half), step = pairs ? 1 : half;
      val = first ? val * cs[j] - vals[i + step] * cs[half + j] : val * cs[j] + vals[i - step] * cs[half + j];
    }
    turned[u] = val;
    ss_after = fmaf(val, val, ss_after);
  }
  const float unit = unit_after ? 1.0f / sqrtf(block_sum(ss_after, scratch) / (float)D + norm_eps) : 1.0f;
#pragma unroll
  for (int u = 0; u < MAX_HEAD / 128; ++u) {
    const int i = threadIdx.x + u * 128;
    if (i >= D) break;
    if (hh < H) q_out[(size_t)t * ldq + hh * D + i] = from_f32<T>(turned[u] * unit * temper);
    else kcache[(((size_t)page * G + (hh - H)) * page_size + off) * D + i] = from_f32<T>(turned[u] * unit);
  }
}

// The same without a filter, for bfloat16 steps of many tokens.  A block owns ROWS_T consecutive tokens of
// the step and a run of heads: the angles of its tokens are taken once for all its heads, a warp turns a
// (token, head) at a time with both dims of a pair in one lane, and values pass through shared memory so
// that a dim's neighbouring positions are written together.
constexpr int ROWS_T = 16, ROWS_WARPS = 8, VCH = 64;   // tokens a block; warps; value dims a warp turns at a time

template <int NP>     // pairs of dims a lane holds: heads up to 64 * NP wide
__global__ void __launch_bounds__(ROWS_WARPS * 32) rope_cache_rows_kernel(
    const bf16* __restrict__ u, long long ldu, const float* __restrict__ inv_freq, int rot, const int* __restrict__ tok_pos,
    const int* __restrict__ tok_seq, const int* __restrict__ seq_slot, const int* __restrict__ page_table, int table_width,
    int page_size, bf16* __restrict__ q_out, long long ldq, bf16* __restrict__ kcache, bf16* __restrict__ vcache, int ntok, int H,
    int G, int D, int Vd, const float* __restrict__ q_norm, const float* __restrict__ k_norm, float norm_eps, float rot_mag,
    float qt_coef, int qt_every, int v_from_k, int pairs, int unit_after, int heads_a_block, int two) {
  extern __shared__ float2 turn[];                      // [ROWS_T][rot / 2] (cos, sin)
  __shared__ int page_of[ROWS_T], off_of[ROWS_T];
  __shared__ float temper_of[ROWS_T];
  __shared__ bf16 tile[ROWS_WARPS][ROWS_T][VCH + 2];
  pdl_release_next();
  pdl_wait_prior();
  const int t0 = blockIdx.x * ROWS_T, nt = min(ROWS_T, ntok - t0), half = rot / 2;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < nt) {
    const int t = t0 + threadIdx.x, pos = tok_pos[t];
    page_of[threadIdx.x] = page_table ? page_table[(size_t)seq_slot[tok_seq[t]] * table_width + (pos / page_size) % table_width] : 0;
    off_of[threadIdx.x] = pos % page_size;
    temper_of[threadIdx.x] = qt_every > 0 ? 1.0f + qt_coef * logf((float)((pos + 1) / qt_every + 1)) : 1.0f;
  }
  for (int e = threadIdx.x; e < nt * half; e += ROWS_WARPS * 32) {
    float sn, cn;
    sincosf((float)tok_pos[t0 + e / half] * inv_freq[e % half], &sn, &cn);
    turn[e] = make_float2(cn * rot_mag, sn * rot_mag);
  }
  __syncthreads();
  const int hb = blockIdx.y * heads_a_block, he = min(H + 2 * G, hb + heads_a_block);
  // ---- queries and keys
  const int qk_end = min(he, H + G);
  for (int w = warp; w < (qk_end - hb) * nt; w += ROWS_WARPS) {
    const int hh = hb + w / nt, tt = w % nt;
    if (hh >= H && !kcache) break;
    const bf16* src = u + (size_t)(t0 + tt) * ldu + (size_t)hh * D;
    const float* norm_w = hh < H ? q_norm : k_norm;
    float a[NP], b[NP], ss = 0.f;
    int da[NP], db[NP];
#pragma unroll
    for (int s = 0; s < NP; ++s) {
      const int p = lane + 32 * s;
      const bool turns = p < half;
      da[s] = turns ? (pairs ? 2 * p : p) : rot + 2 * (p - half);
      db[s] = turns && !pairs ? p + half : da[s] + 1;
      a[s] = b[s] = 0.f;
      if (da[s] < D) {
        if (two && db[s] == da[s] + 1) {                 // D is even here: db < D
          const float2 v = __bfloat1622float2(*(const __nv_bfloat162*)(src + da[s]));
          a[s] = v.x;
          b[s] = v.y;
        } else {
          a[s] = to_f32(src[da[s]]);
          if (db[s] < D) b[s] = to_f32(src[db[s]]);
        }
      }
      ss = fmaf(a[s], a[s], fmaf(b[s], b[s], ss));
    }
    if (norm_w) {
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)D + norm_eps);
#pragma unroll
      for (int s = 0; s < NP; ++s) {
        if (da[s] < D) a[s] *= inv * norm_w[da[s]];
        if (db[s] < D) b[s] *= inv * norm_w[db[s]];
      }
    }
    ss = 0.f;
#pragma unroll
    for (int s = 0; s < NP; ++s) {
      const int p = lane + 32 * s;
      if (p < half) {
        const float2 cs = turn[tt * half + p];
        const float x = a[s] * cs.x - b[s] * cs.y;
        b[s] = b[s] * cs.x + a[s] * cs.y;
        a[s] = x;
      }
      ss = fmaf(a[s], a[s], fmaf(b[s], b[s], ss));
    }
    float factor = hh < H ? temper_of[tt] : 1.0f;
    if (unit_after) factor *= 1.0f / sqrtf(warp_sum(ss) / (float)D + norm_eps);
    bf16* dst = hh < H ? q_out + (size_t)(t0 + tt) * ldq + (size_t)hh * D
                       : kcache + (((size_t)page_of[tt] * G + (hh - H)) * page_size + off_of[tt]) * D;
#pragma unroll
    for (int s = 0; s < NP; ++s) {
      if (da[s] >= D) continue;
      if (two && db[s] == da[s] + 1) {
        *(__nv_bfloat162*)(dst + da[s]) = __floats2bfloat162_rn(a[s] * factor, b[s] * factor);
      } else {
        dst[da[s]] = from_f32<bf16>(a[s] * factor);
        if (db[s] < D) dst[db[s]] = from_f32<bf16>(b[s] * factor);
      }
    }
  }
  // ---- values: rows in, a dim's positions out
  if (!vcache || he <= H + G) return;
  const int v_first = max(hb, H + G) - (H + G), v_heads = he - max(hb, H + G), pieces = (Vd + VCH - 1) / VCH;
  for (int w = warp; w < v_heads * pieces; w += ROWS_WARPS) {
    const int g = v_first + w / pieces, d0 = (w % pieces) * VCH, nd = min(VCH, Vd - d0);
    const bf16* src = u + (size_t)t0 * ldu + (v_from_k ? H * D : (H + G) * D) + (size_t)g * Vd + d0;
    for (int tt = 0; tt < nt; ++tt)
      for (int d = lane; d < nd; d += 32) tile[warp][tt][d] = src[(size_t)tt * ldu + d];
    __syncwarp();
    const int tt = lane % ROWS_T;
    if (tt < nt) {
      bf16* dst = vcache + (((size_t)page_of[tt] * G + g) * Vd + d0) * page_size + off_of[tt];
      for (int d = lane / ROWS_T; d < nd; d += 32 / ROWS_T) dst[(size_t)d * page_size] = tile[warp][tt][d];
    }
    __syncwarp();
  }
}

constexpr int ROWS_MIN_TOKENS = 64, ROWS_MAX_ROT = 384;   // the angles (8 bytes a pair and token) beside the tiles in 48 KB

// taps: [(H + G) D + G Vd, K] float32 (K = 0: no filter); state: [slots, K - 1, channels] float32.
// G = 0: the rows hold queries only (a layer that reads another layer's keys and values).
// q_norm, k_norm: float32 [D] or null (norm_eps is theirs, or unit_after's: not both); v_from_k needs Vd == D.
GB_EXPORT int gb_filter_rope_cache_ext(const void* u, int dtype, long long ldu, const float* taps, const float* state, int K,
                                       const float* inv_freq, int rot, const int* tok_pos, const int* tok_seq,
                                       const int* seq_slot, const int* cu, const int* page_table, int table_width,
                                       int page_size, void* q_out, long long ldq, void* kcache, void* vcache, int ntok, int H,
                                       int G, int D, int Vd, const float* q_norm, const float* k_norm, float norm_eps,
                                       float rot_mag, float qt_coef, int qt_every, int v_from_k, int pairs, int unit_after,
                                       cudaStream_t stream) {
  if (ntok <= 0) return 0;
  if (K < 0 || K > MAX_TAPS || rot < 0 || rot > D || rot % 2 || H <= 0 || G < 0 || D <= 0 || D > MAX_HEAD || Vd <= 0)
    return GB_ERR_SIZE;
  if (v_from_k && (Vd != D || K > 1)) return GB_ERR_SIZE;
  if (unit_after && (q_norm || k_norm)) return GB_ERR_ARG;
  if ((K > 0 && !taps) || (K > 1 && !state) || (rot > 0 && !inv_freq) || qt_every < 0) return GB_ERR_ARG;
  if (dtype == GB_BF16 && K == 0 && ntok >= ROWS_MIN_TOKENS && rot <= ROWS_MAX_ROT) {
    // blocks for a few rounds of the SMs: heads are dealt out until there are enough
    const int tiles = (ntok + ROWS_T - 1) / ROWS_T, all = H + 2 * G;
    const int runs = min(all, max(1, (4 * 148 + tiles - 1) / tiles)), each = (all + runs - 1) / runs;
    const int two = D % 2 == 0 && ldu % 2 == 0 && ldq % 2 == 0 && !((uintptr_t)u & 3) && !((uintptr_t)q_out & 3) && !((uintptr_t)kcache & 3);
    const size_t smem = (size_t)ROWS_T * (rot / 2) * sizeof(float2);
#define ROWS(NP)                                                                                                               \
  gb_launch(rope_cache_rows_kernel<NP>, dim3(tiles, (all + each - 1) / each), dim3(ROWS_WARPS * 32), smem, stream, (const bf16*)u, \
            ldu, inv_freq, rot, tok_pos, tok_seq, seq_slot, page_table, table_width, page_size, (bf16*)q_out, ldq, (bf16*)kcache,  \
            (bf16*)vcache, ntok, H, G, D, Vd, q_norm, k_norm, norm_eps, rot_mag, qt_coef, qt_every, v_from_k, pairs, unit_after, \
            each, two)
    if (D <= 64) ROWS(1);
    else if (D <= 128) ROWS(2);
    else if (D <= 256) ROWS(4);
    else ROWS(8);
#undef ROWS
    return gb_launch_status();
  }
  const dim3 grid(ntok, H + 2 * G);
  if (dtype == GB_F32)
    gb_launch(filter_rope_cache_kernel<float>, grid, 128, 0, stream, (const float*)u, ldu, taps, state, K, inv_freq, rot,
              tok_pos, tok_seq, seq_slot, cu, page_table, table_width, page_size, (float*)q_out, ldq, (float*)kcache,
              (float*)vcache, H, G, D, Vd, q_norm, k_norm, norm_eps, rot_mag, qt_coef, qt_every, v_from_k, pairs, unit_after);
  else if (dtype == GB_BF16)
    gb_launch(filter_rope_cache_kernel<bf16>, grid, 128, 0, stream, (const bf16*)u, ldu, taps, state, K, inv_freq, rot,
              tok_pos, tok_seq, seq_slot, cu, page_table, table_width, page_size, (bf16*)q_out, ldq, (bf16*)kcache,
              (bf16*)vcache, H, G, D, Vd, q_norm, k_norm, norm_eps, rot_mag, qt_coef, qt_every, v_from_k, pairs, unit_after);
  else
    return GB_ERR_DTYPE;
  return gb_launch_status();
}

GB_EXPORT int gb_filter_rope_cache(const void* u, int dtype, long long ldu, const float* taps, const float* state, int K,
                                   const float* inv_freq, int rot, const int* tok_pos, const int* tok_seq, const int* seq_slot,
                                   const int* cu, const int* page_table, int table_width, int page_size, void* q_out,
                                   long long ldq, void* kcache, void* vcache, int ntok, int H, int G, int D, int Vd,
                                   cudaStream_t stream) {
  return gb_filter_rope_cache_ext(u, dtype, ldu, taps, state, K, inv_freq, rot, tok_pos, tok_seq, seq_slot, cu, page_table,
                                  table_width, page_size, q_out, ldq, kcache, vcache, ntok, H, G, D, Vd, nullptr, nullptr, 0.f,
                                  1.f, 0.f, 0, 0, 0, 0, stream);
}

// One block per (token, query head); online softmax over chunks of 128 keys: first the kept keys
// below the window (chunks from 0), then the window (chunks from lo).  A sink starts the running
// maximum at its value and the running sum at one.
template <typename T>
__global__ void __launch_bounds__(CHUNK) attention_capped_kernel(
    const T* __restrict__ q, long long q_stride, T* __restrict__ out, long long out_stride, const T* __restrict__ kcache,
    const T* __restrict__ vcache, const int* __restrict__ page_table, int table_width, int page_size, int G, int D, int Vd,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_seq, const int* __restrict__ seq_slot, int H, int window,
    int keep_first, const float* __restrict__ sink, float scale, float cap, const T* __restrict__ gate, long long gate_stride,
    float out_scale, int gate_per_head) {
  extern __shared__ float smem[];
  pdl_release_next();
  pdl_wait_prior();
  float* qs = smem;                    // [D]
  float* p = qs + D;                   // [CHUNK]
  float* scratch = p + CHUNK;          // [34]
  size_t* rows = (size_t*)(((uintptr_t)(scratch + 34) + 7) & ~(uintptr_t)7);   // [CHUNK]
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int g = h / (H / G);
  const int pos = tok_pos[t];
  const int slot = seq_slot[tok_seq[t]];
  const int hi = pos + 1;
  const int lo = window > 0 ? max(0, hi - window) : 0;
  const T* qrow = q + (size_t)t * q_stride + (size_t)h * D;
  for (int i = tid; i < D; i += CHUNK) qs[i] = to_f32(qrow[i]);
  __syncthreads();
  const float inv_cap = cap > 0.f ? 1.0f / cap : 0.f;
  float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f, acc[VPT] = {};
  const int kept = min(keep_first, lo);          // kept keys that the window does not cover
  const int kept_chunks = (kept + CHUNK - 1) / CHUNK;
  for (int it = 0; it < kept_chunks || lo + (it - kept_chunks) * CHUNK < hi; ++it) {
    const int c0 = it < kept_chunks ? it * CHUNK : lo + (it - kept_chunks) * CHUNK;
    const int end = it < kept_chunks ? kept : hi;
    const int j = c0 + tid;
    float s = -INFINITY;
    if (j < end) {
      const int page = page_table[(size_t)slot * table_width + (j / page_size) % table_width];
      const int off = j % page_size;
      const T* kr = kcache + (((size_t)page * G + g) * page_size + off) * D;
      rows[tid] = ((size_t)page * G + g) * Vd * page_size + off;
      float d = 0.f;
      for (int i = 0; i < D; ++i) d = fmaf(qs[i], to_f32(kr[i]), d);
      s = d * scale;
      if (cap > 0.f) s = cap * tanhf(s * inv_cap);
    }
    const float m_new = fmaxf(m, block_max(s, scratch));
    const float pj = j < end ? expf(s - m_new) : 0.f;
    p[tid] = pj;
    const float csum = block_sum(pj, scratch);   // also orders the writes of p and rows
    const float alpha = expf(m - m_new);
    l = l * alpha + csum;
    const int n = min(CHUNK, end - c0);
#pragma unroll
    for (int u = 0; u < VPT; ++u) {
      const int d = tid + u * CHUNK;
      if (d < Vd) {
        float a = acc[u] * alpha;
        for (int jj = 0; jj < n; ++jj) a = fmaf(p[jj], to_f32(vcache[rows[jj] + (size_t)d * page_size]), a);
        acc[u] = a;
      }
    }
    m = m_new;
    __syncthreads();
  }
  T* orow = out + (size_t)t * out_stride + (size_t)h * Vd;
#pragma unroll
  for (int u = 0; u < VPT; ++u) {
    const int d = tid + u * CHUNK;
    if (d < Vd) {
      float o = acc[u] / l;
      if (gate) o *= 1.0f / (1.0f + expf(-to_f32(gate[(size_t)t * gate_stride + (gate_per_head ? h : h * Vd + d)])));
      orow[d] = from_f32<T>(o * out_scale);
    }
  }
}

GB_EXPORT int gb_attention_capped(const void* q, long long q_stride, void* out, long long out_stride, int dtype,
                                  const void* kcache, const void* vcache, const int* page_table, int table_width, int page_size,
                                  int G, int D, int Vd, const int* tok_pos, const int* tok_seq, const int* seq_slot, int ntok,
                                  int H, int window, int keep_first, const float* sink, float scale, float cap,
                                  const void* gate, long long gate_stride, float out_scale, int gate_per_head,
                                  cudaStream_t stream) {
  if (ntok <= 0) return 0;
  if (D <= 0 || Vd <= 0 || Vd > VPT * CHUNK || G <= 0 || H % G || keep_first < 0) return GB_ERR_SIZE;
  if (window <= 0) keep_first = 0;      // every key is seen already
  const size_t smem = (size_t)(D + CHUNK + 34) * sizeof(float) + CHUNK * sizeof(size_t) + 8;
  dim3 grid(ntok, H);
  if (dtype == GB_F32)
    gb_launch(attention_capped_kernel<float>, grid, CHUNK, smem, stream, (const float*)q, q_stride, (float*)out, out_stride,
              (const float*)kcache, (const float*)vcache, page_table, table_width, page_size, G, D, Vd, tok_pos, tok_seq,
              seq_slot, H, window, keep_first, sink, scale, cap, (const float*)gate, gate_stride, out_scale, gate_per_head);
  else if (dtype == GB_BF16)
    gb_launch(attention_capped_kernel<bf16>, grid, CHUNK, smem, stream, (const bf16*)q, q_stride, (bf16*)out, out_stride,
              (const bf16*)kcache, (const bf16*)vcache, page_table, table_width, page_size, G, D, Vd, tok_pos, tok_seq, seq_slot,
              H, window, keep_first, sink, scale, cap, (const bf16*)gate, gate_stride, out_scale, gate_per_head);
  else
    return GB_ERR_DTYPE;
  return gb_launch_status();
}
