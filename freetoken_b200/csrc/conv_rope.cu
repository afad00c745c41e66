// Attention with several softmax maps a head over the same values: from the projected rows to what the attention
// kernels read, and from their outputs to the head's output.
//
// conv_rope_store, one pass over the rows q | k | v of the projection (q head by head as [map 1, map 2, ...], k too):
// a causal convolution over time on every channel (the earlier inputs of a request's first tokens from its state slot,
// the last ones left there), the rotation of each map's leading dimensions by the token's position (32-bit, pairs of
// neighbours or halves), and the scatter.  A key row in the cache holds the maps of a KV head side by side, and query
// (head, map) is a row of the same length that is zero outside its map's place: its product with the key row is
// the map's score, so the attention kernels see plain grouped-query heads.  Rows are padded with zeros to pad_dim.
// Tiles are aligned to requests as in conv_act: tile 0 of a request is the only one that reads the old state, and the
// same threads write the new one.
//
// diff_heads, per (token, head): unit(a1 - lambda a2) * scale with the root mean square over the head's vdim values.
#include "common.cuh"

namespace ftk {

constexpr int kCrTile = 16;      // tokens per tile (at least taps - 1)
constexpr int kCrMaxTaps = 16;
constexpr int kCrThreads = 128;  // up to four channels a thread

// VEC: head sizes, rows and pointers allow four channels at a time; then a thread's channels always lie in one head.
template <typename T, int TAPS, bool VEC>
__global__ void __launch_bounds__(kCrThreads) conv_rope_store_kernel(const __grid_constant__ FtkConvRope p) {
  const int dq = (p.dim + 3) >> 2, vq = (p.vdim + 3) >> 2;      // threads a map's head and a value head take
  const int n_qk = (p.n_heads + p.n_kv_heads) * p.maps;         // q and k heads of `dim`
  const int item = blockIdx.y * kCrThreads + threadIdx.x;
  const int qk_items = n_qk * dq;
  const bool is_v = item >= qk_items;
  const bool in_range = item < qk_items + p.n_kv_heads * vq;
  const int head = is_v ? (item - qk_items) / vq : item / dq;   // among the q and k heads, or among the value heads
  const int d0 = (is_v ? (item - qk_items) - head * vq : item - head * dq) * 4;
  const int len = is_v ? p.vdim : p.dim;
  const int c0 = is_v ? n_qk * p.dim + head * p.vdim + d0 : head * p.dim + d0;  // channel of the projection
  const int C = n_qk * p.dim + p.n_kv_heads * p.vdim;
  const int nc = in_range ? min(4, len - d0) : 0;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const int keep = taps - 1;
  constexpr int kMost = TAPS > 0 ? TAPS : kCrMaxTaps;
  // the taps wait for nothing
  float wt[kMost][4];
#pragma unroll
  for (int j = 0; j < (TAPS > 0 ? TAPS : taps); ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) wt[j][i] = i < nc ? p.conv_w[(size_t)(c0 + i) * taps + j] : 0.f;
  pdl_wait();
  pdl_trigger();
  if (nc == 0) return;
  int tile = blockIdx.x, seg = 0, q_start = 0, q_len = 0, kv_len = 0;
  for (; seg < p.n_segs; ++seg) {
    q_start = p.seg_info[seg * 4]; q_len = p.seg_info[seg * 4 + 1]; kv_len = p.seg_info[seg * 4 + 2];
    const int n = q_len > 0 ? (q_len + kCrTile - 1) / kCrTile : 0;
    if (tile < n) break;
    tile -= n;
  }
  if (seg >= p.n_segs || q_start < 0 || q_start + q_len > p.n_tokens || kv_len < q_len) return;
  const int slot = keep ? p.state_slots[seg] : -1;
  const int before = kv_len - q_len;
  float* st = (keep && slot >= 0 && slot < p.n_slots) ? p.state + ((size_t)slot * keep) * C + c0 : nullptr;
  const bool first = tile == 0;
  const int t0 = tile * kCrTile, t1 = min(q_len, t0 + kCrTile);
  const T* x = (const T*)p.x + c0;
  auto input = [&](int s, float (&v)[4]) {  // the request's input `s` places into this step (s >= 0)
    const T* r = x + (size_t)(q_start + s) * p.x_stride;
    if (VEC) Vec4<T>::load(r, v);
    else for (int i = 0; i < 4; ++i) v[i] = i < nc ? to_float(r[i]) : 0.f;
  };
  float old[kMost][4];                      // row r: the input `keep - r` places before this step; tile 0 only
#pragma unroll
  for (int r = 0; r < (TAPS > 0 ? TAPS - 1 : keep); ++r)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      old[r][i] = (first && st && keep - r <= before && i < nc) ? st[(size_t)r * C + i] : 0.f;
  constexpr int K = TAPS > 1 ? TAPS - 1 : 1;
  float win[K][4];                          // TAPS > 1: the inputs t - K .. t - 1, oldest first
  if (TAPS > 1) {
#pragma unroll
    for (int r = 0; r < K; ++r) {
      if (first) {
#pragma unroll
        for (int i = 0; i < 4; ++i) win[r][i] = old[r][i];
      } else {
        input(t0 - K + r, win[r]);
      }
    }
  }
  // where a token's result goes
  const int kv_first = p.n_heads * p.maps;
  const bool is_q = !is_v && head < kv_first;
  const int map = is_v ? 0 : head % p.maps;
  const int row_head = is_v ? head : is_q ? head : (head - kv_first) / p.maps;  // head of the destination
  const int off = (is_v ? 0 : map * p.dim) + d0;                                // column of the destination row
  const bool turns = !is_v && p.table && d0 < p.n_rot;
  const int half = p.n_rot >> 1;
  const int used = is_v ? p.vdim : p.maps * p.dim;
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    float cur[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
    input(t, cur);
    if (TAPS > 1) {
#pragma unroll
      for (int r = 0; r < K; ++r)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(wt[r][i], win[r][i], acc[i]);
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i] = fmaf(wt[K][i], cur[i], acc[i]);
#pragma unroll
      for (int r = 0; r + 1 < K; ++r)
#pragma unroll
        for (int i = 0; i < 4; ++i) win[r][i] = win[r + 1][i];
#pragma unroll
      for (int i = 0; i < 4; ++i) win[K - 1][i] = cur[i];
    } else {
      for (int j = 0; j < taps; ++j) {
        const int s = t - keep + j;
        float in[4];
        if (j == keep) { for (int i = 0; i < 4; ++i) in[i] = cur[i]; }
        else if (s >= 0) input(s, in);
        else if (first) { for (int i = 0; i < 4; ++i) in[i] = old[keep + s][i]; }
        else continue;                      // (tiles hold at least `keep` tokens: never reached)
        for (int i = 0; i < 4; ++i) acc[i] = fmaf(wt[j][i], in[i], acc[i]);
      }
    }
    const int tok = q_start + t;
    if (turns) {
      int pos = p.positions[tok];
      pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
      const float* cs = p.table + (size_t)pos * p.n_rot;
      // neighbours only (the host refuses the halves' layout): pairs (d0, d0 + 1) and (d0 + 2, d0 + 3)
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        if (d0 + i < p.n_rot) {
          const float c = __ldg(cs + ((d0 + i) >> 1)), s = __ldg(cs + half + ((d0 + i) >> 1));
          const float a = acc[i], b = acc[i + 1];
          acc[i] = a * c - b * s;
          acc[i + 1] = b * c + a * s;
        }
      }
    }
    T* row;
    if (is_q) {
      row = (T*)p.q_out + ((size_t)tok * p.n_heads * p.maps + row_head) * p.pad_dim;
    } else {
      const int sl = p.slot_map[tok];
      if (sl < 0 || sl >= p.num_pages * p.page_size) continue;  // not stored
      const unsigned int page = (unsigned int)sl / (unsigned int)p.page_size, o = (unsigned int)sl % (unsigned int)p.page_size;
      row = (T*)(is_v ? p.v_slab : p.k_slab) + (((size_t)page * p.n_kv_heads + row_head) * p.page_size + o) * p.pad_dim;
    }
    if (VEC) Vec4<T>::store(row + off, acc);
    else for (int i = 0; i < nc; ++i) row[off + i] = from_float<T>(acc[i]);
    const float zero[4] = {0.f, 0.f, 0.f, 0.f};
    if (is_q) {                             // the other maps' places, column for column
      for (int m = 0; m < p.maps; ++m) {
        if (m == map) continue;
        T* z = row + m * p.dim + d0;
        if (VEC) Vec4<T>::store(z, zero);
        else for (int i = 0; i < nc; ++i) z[i] = from_float<T>(0.f);
      }
    }
    if (used < p.pad_dim && (is_q || map == 0)) {  // (a query row belongs to one map, a key row to all)
      const int step = ((is_v ? vq : dq)) * 4;
      for (int z0 = used + d0; z0 < p.pad_dim; z0 += step) {
        if (VEC) Vec4<T>::store(row + z0, zero);
        else for (int i = 0; i < 4 && z0 + i < p.pad_dim; ++i) row[z0 + i] = from_float<T>(0.f);
      }
    }
  }
  if (first && st) {                        // the new state: the request's last `keep` inputs, oldest first
#pragma unroll
    for (int r = 0; r < (TAPS > 0 ? TAPS - 1 : keep); ++r) {
      const int s = q_len - keep + r;
      float v[4];
      if (s >= 0) {
        input(s, v);
      } else {
        for (int i = 0; i < 4; ++i) v[i] = 0.f;
#pragma unroll
        for (int k = 0; k < (TAPS > 0 ? TAPS - 1 : keep); ++k)
          if (k == keep + s)
#pragma unroll
            for (int i = 0; i < 4; ++i) v[i] = old[k][i];
      }
      for (int i = 0; i < nc; ++i) st[(size_t)r * C + i] = v[i];
    }
  }
}

template <typename T>
__global__ void diff_heads_kernel(const T* __restrict__ o, int o_stride, const float* __restrict__ lambda, float eps,
                                  float scale, T* __restrict__ out, int n_tokens, int n_heads, int vdim) {
  pdl_wait();
  pdl_trigger();
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (long long)n_tokens * n_heads) return;
  const int lane = threadIdx.x & 31;
  const T* a = o + (size_t)w * 2 * o_stride;
  const T* b = a + o_stride;
  const float lam = *lambda;
  float v[8];  // vdim <= 256
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = lane + 32 * i;
    v[i] = d < vdim ? to_float(a[d]) - lam * to_float(b[d]) : 0.f;
    ss = fmaf(v[i], v[i], ss);
  }
  const float f = rsqrtf(warp_sum(ss) / (float)vdim + eps) * scale;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) out[(size_t)w * vdim + d] = from_float<T>(v[i] * f);
  }
}

// The same for bfloat16 heads of 8 x 2^k values with 16-byte accesses: TPR threads a head, eight values each.
template <int TPR>
__global__ void __launch_bounds__(256) diff_heads_vec_kernel(const __nv_bfloat16* __restrict__ o, int o_stride,
                                                             const float* __restrict__ lambda, float eps, float scale,
                                                             __nv_bfloat16* __restrict__ out, int n_tokens, int n_heads) {
  pdl_wait();
  pdl_trigger();
  constexpr int vdim = TPR * 8;
  const long long w = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / TPR;
  const bool ok = w < (long long)n_tokens * n_heads;
  const int d = (threadIdx.x % TPR) * 8;
  const float lam = *lambda;
  float v[8];
  float ss = 0.f;
  {
    const __nv_bfloat16* a = o + (size_t)(ok ? w : 0) * 2 * o_stride + d;
    const uint4 ra = *reinterpret_cast<const uint4*>(a), rb = *reinterpret_cast<const uint4*>(a + o_stride);
    const __nv_bfloat162* pa = reinterpret_cast<const __nv_bfloat162*>(&ra);
    const __nv_bfloat162* pb = reinterpret_cast<const __nv_bfloat162*>(&rb);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float2 x = __bfloat1622float2(pa[u]), y = __bfloat1622float2(pb[u]);
      v[2 * u] = x.x - lam * y.x;
      v[2 * u + 1] = x.y - lam * y.y;
    }
  }
#pragma unroll
  for (int u = 0; u < 8; ++u) ss = fmaf(v[u], v[u], ss);
#pragma unroll
  for (int s = TPR / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  const float f = rsqrtf(ss / (float)vdim + eps) * scale;
  uint4 res;
  __nv_bfloat162* r2 = reinterpret_cast<__nv_bfloat162*>(&res);
#pragma unroll
  for (int u = 0; u < 4; ++u) r2[u] = __floats2bfloat162_rn(v[2 * u] * f, v[2 * u + 1] * f);
  if (ok) *reinterpret_cast<uint4*>(out + (size_t)w * vdim + d) = res;
}

}  // namespace ftk

using namespace ftk;

extern "C" int ftk_conv_rope_store(const FtkConvRope* args, void* stream) {
  FTK_REQUIRE(args, "conv_rope_store: null arguments");
  const FtkConvRope& p = *args;
  FTK_REQUIRE(dtype_ok(p.dtype), "conv_rope_store: bad dtype %d", p.dtype);
  FTK_REQUIRE(p.taps >= 1 && p.taps <= kCrMaxTaps, "conv_rope_store: %d taps (1 to %d taken)", p.taps, kCrMaxTaps);
  FTK_REQUIRE(p.n_heads >= 1 && p.n_kv_heads >= 1 && p.maps >= 1 && p.dim >= 1 && p.vdim >= 1 && p.n_tokens >= 0 &&
                  p.n_segs >= 1, "conv_rope_store: bad sizes");
  FTK_REQUIRE(p.pad_dim >= p.maps * p.dim && p.pad_dim >= p.vdim, "conv_rope_store: rows of %d do not hold %d maps of %d and values of %d",
              p.pad_dim, p.maps, p.dim, p.vdim);
  FTK_REQUIRE(p.n_rot >= 0 && p.n_rot <= p.dim && p.n_rot % 2 == 0 && (p.n_rot == 0 || p.interleaved),
              "conv_rope_store: turns an even number of leading dimensions in pairs of neighbours");
  if (p.n_tokens == 0) return 0;
  FTK_REQUIRE(p.x && p.conv_w && p.seg_info && p.q_out && p.k_slab && p.v_slab && p.slot_map && p.page_size >= 1 &&
                  p.num_pages >= 1 && (long long)p.num_pages * p.page_size < (1ll << 31) && (p.n_rot == 0 || (p.positions && p.table && p.max_pos >= 1)) &&
                  (p.taps == 1 || (p.state && p.state_slots)), "conv_rope_store: null pointer");
  const int C = (p.n_heads + p.n_kv_heads) * p.maps * p.dim + p.n_kv_heads * p.vdim;
  FTK_REQUIRE(p.x_stride >= C, "conv_rope_store: rows of %lld hold no %d channels", p.x_stride, C);
  const int item = dtype_size(p.dtype);
  auto al = [&](const void* q) { return (reinterpret_cast<uintptr_t>(q) % (4 * item)) == 0; };
  const bool vec = p.dim % 4 == 0 && p.vdim % 4 == 0 && p.x_stride % 4 == 0 && p.pad_dim % 4 == 0 && al(p.x) && al(p.q_out) &&
                   al(p.k_slab) && al(p.v_slab);
  const int items = (p.n_heads + p.n_kv_heads) * p.maps * ((p.dim + 3) / 4) + p.n_kv_heads * ((p.vdim + 3) / 4);
  dim3 grid((p.n_tokens + kCrTile - 1) / kCrTile + p.n_segs, (items + kCrThreads - 1) / kCrThreads);
  FTK_REQUIRE(grid.y <= 65535, "conv_rope_store: too many channels");
  cudaStream_t s = (cudaStream_t)stream;
  FtkConvRope a = p;
  if (a.n_rot == 0) a.table = nullptr;
#define FTK_CR(TY, N)                                                                              \
  do {                                                                                             \
    if (vec) FTK_LAUNCH((conv_rope_store_kernel<TY, N, true>), grid, kCrThreads, 0, s, a);         \
    else FTK_LAUNCH((conv_rope_store_kernel<TY, N, false>), grid, kCrThreads, 0, s, a);            \
  } while (0)
#define FTK_CR_TAPS(TY)                  \
  do {                                   \
    if (p.taps == 2) FTK_CR(TY, 2);      \
    else if (p.taps == 3) FTK_CR(TY, 3); \
    else if (p.taps == 4) FTK_CR(TY, 4); \
    else FTK_CR(TY, 0);                  \
  } while (0)
  if (p.dtype == FTK_F32) FTK_CR_TAPS(float);
  else FTK_CR_TAPS(__nv_bfloat16);
#undef FTK_CR_TAPS
#undef FTK_CR
  FTK_LAUNCH_CHECK("conv_rope_store");
  return 0;
}

extern "C" int ftk_diff_heads(const void* o, int o_stride, int dtype, const float* lambda, float eps, float scale, void* out,
                              int n_tokens, int n_heads, int vdim, void* stream) {
  FTK_REQUIRE(dtype_ok(dtype), "diff_heads: bad dtype %d", dtype);
  FTK_REQUIRE(n_tokens >= 0 && n_heads >= 1 && vdim >= 1 && vdim <= 256 && o_stride >= vdim, "diff_heads: bad sizes");
  if (n_tokens == 0) return 0;
  FTK_REQUIRE(o && lambda && out, "diff_heads: null pointer");
  const long long rows = (long long)n_tokens * n_heads;
  const int tpr = vdim / 8;
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == FTK_BF16 && vdim % 8 == 0 && (tpr & (tpr - 1)) == 0 && o_stride % 8 == 0 &&
      (((uintptr_t)o | (uintptr_t)out) & 15) == 0) {
    const unsigned blocks = (unsigned)((rows * tpr + 255) / 256);
#define FTK_DH(N) FTK_LAUNCH((diff_heads_vec_kernel<N>), blocks, 256, 0, s, (const __nv_bfloat16*)o, o_stride, lambda, eps, scale, \
                             (__nv_bfloat16*)out, n_tokens, n_heads)
    if (tpr == 1) FTK_DH(1);
    else if (tpr == 2) FTK_DH(2);
    else if (tpr == 4) FTK_DH(4);
    else if (tpr == 8) FTK_DH(8);
    else if (tpr == 16) FTK_DH(16);
    else FTK_DH(32);
#undef FTK_DH
    FTK_LAUNCH_CHECK("diff_heads");
    return 0;
  }
  const unsigned blocks = (unsigned)((rows + 7) / 8);
  if (dtype == FTK_F32)
    FTK_LAUNCH(diff_heads_kernel<float>, blocks, 256, 0, s, (const float*)o, o_stride, lambda, eps, scale, (float*)out, n_tokens,
               n_heads, vdim);
  else
    FTK_LAUNCH(diff_heads_kernel<__nv_bfloat16>, blocks, 256, 0, s, (const __nv_bfloat16*)o, o_stride, lambda, eps, scale,
               (__nv_bfloat16*)out, n_tokens, n_heads, vdim);
  FTK_LAUNCH_CHECK("diff_heads");
  return 0;
}
