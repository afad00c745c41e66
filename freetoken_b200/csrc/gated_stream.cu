// Layers whose sub-layer results pass a gate and a norm over groups of channels before they join the 32-bit stream.
//
// stream_step, one pass over a token's row (every part optional):
//   r <- r + vec                                            a vector for every token (what a pass of a loop adds)
//   y  = dense row (or x_scale times it plus x2_scale times a second one), or the sum over the token's expert routes in route order, plus pass_w * passed (experts that hand
//        their input back) and shared_w * shared             (32-bit sums)
//   y <- y * sigmoid(gate + gate_bias)                       element by element
//   r <- r + groupnorm(y) * w_post                           (a factor on the result is folded into w_post), or r <- r + y
//   raw = r rounded to the engine's type                     rows of another tensor (its own row stride)
//   h  = groupnorm(r) * w_pre                                into `out`, as float32 into `norm_f32`
//   u  = h + sum_j conv_w[:, j] h(t - taps + 1 + j)          steps of one token per request: the earlier h come from the
//                                                            request's state slot, which moves on by one
// groupnorm: a row is cut into `groups` equal consecutive parts, each divided by its own sqrt(mean(part^2) + eps).
// With `rows` only those rows are read, and the stream stays as it is.
#include "common.cuh"

namespace ftk {

struct StepArgs {
  FtkStreamStep p;
  int group_size;
  int warps_per_group;  // of the register form
};

constexpr int kStepMaxTaps = 16;

// (results that are rounded to bfloat16 after the norm take the fast exponential and division, about 2^-21 relative each)
template <typename T>
__device__ __forceinline__ float gate_sigmoid(float z) {
  if constexpr (sizeof(T) == 4) return 1.f / (1.f + expf(-z));
  else return __fdividef(1.f, 1.f + __expf(-z));
}

// Four adjacent elements as they lie in memory: a load that may be left out is kept in this form, since widening it beside
// the load would make the branch around it wait for the data.
template <typename T>
struct Raw4;
template <>
struct Raw4<float> {
  float4 v;
  __device__ __forceinline__ void widen(float (&y)[4]) const { y[0] = v.x; y[1] = v.y; y[2] = v.z; y[3] = v.w; }
};
template <>
struct Raw4<__nv_bfloat16> {
  uint2 v;
  __device__ __forceinline__ void widen(float (&y)[4]) const {
    y[0] = __uint_as_float(v.x << 16);
    y[1] = __uint_as_float(v.x & 0xffff0000u);
    y[2] = __uint_as_float(v.y << 16);
    y[3] = __uint_as_float(v.y & 0xffff0000u);
  }
};
template <typename T>
__device__ __forceinline__ Raw4<T> raw_or_zero(const T* p, bool have) {
  Raw4<T> r{};
  if (have) r = *reinterpret_cast<const Raw4<T>*>(p);
  return r;
}

// One element (or four adjacent ones) of the sub-layer's gated result.
template <typename T, int W>
__device__ __forceinline__ void gated_result(const FtkStreamStep& p, int src_row, size_t src, int i, float2 aux, float (&v)[4]) {
  const T* x = (const T*)p.x;
  auto load = [](const T* q, float (&y)[4]) {
    if constexpr (W == 4) Vec4<T>::load(q, y);
    else y[0] = to_float(*q);
  };
  if (p.route_pos) {
#pragma unroll
    for (int u = 0; u < W; ++u) v[u] = 0.f;
    for (int j0 = 0; j0 < p.top_k; j0 += 4) {  // four rows' loads in flight before the first is added, in route order
      float y[4][4];
      int q[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        q[j] = j0 + j < p.top_k ? __ldg(p.route_pos + (size_t)src_row * p.top_k + j0 + j) : -1;
        if (q[j] >= p.n_routes) q[j] = -1;
        if (q[j] >= 0) load(x + (size_t)q[j] * p.hidden + i, y[j]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (q[j] >= 0) {
#pragma unroll
          for (int u = 0; u < W; ++u) v[u] += y[j][u];
        }
    }
    if (p.passed && aux.x != 0.f) {
      float y[4];
      load((const T*)p.passed + src + i, y);
#pragma unroll
      for (int u = 0; u < W; ++u) v[u] = fmaf(aux.x, y[u], v[u]);
    }
    if (p.shared) {
      float y[4];
      load((const T*)p.shared + src + i, y);
#pragma unroll
      for (int u = 0; u < W; ++u) v[u] = fmaf(aux.y, y[u], v[u]);
    }
  } else {
    load(x + src + i, v);
    if (p.x2) {
      float y[4];
      load((const T*)p.x2 + src + i, y);
#pragma unroll
      for (int u = 0; u < W; ++u) v[u] = fmaf(p.x2_scale, y[u], p.x_scale * v[u]);
    }
  }
  if (p.gate) {
    float g[4], b[4];
    load((const T*)p.gate + src + i, g);
    if (p.gate_bias) {
      if constexpr (W == 4) Vec4<float>::load(p.gate_bias + i, b);
      else b[0] = p.gate_bias[i];
    } else {
#pragma unroll
      for (int u = 0; u < W; ++u) b[u] = 0.f;
    }
#pragma unroll
    for (int u = 0; u < W; ++u) v[u] *= gate_sigmoid<T>(g[u] + b[u]);
  }
}

// The convolution of one token per request: `h` holds the channels' normed values as stored (rounded).
template <typename T, int W>
__device__ __forceinline__ void step_conv(const FtkStreamStep& p, int row, size_t dst, int i, const float (&h)[4], bool live,
                                          float* st, int before) {
  const int keep = p.taps - 1;
  float acc[4];
#pragma unroll
  for (int u = 0; u < W; ++u) acc[u] = fmaf(p.conv_w[(size_t)(i + u) * p.taps + keep], h[u], h[u]);
  float next[4];
  for (int r = 0; r < keep; ++r) {  // oldest first; row r holds the value `keep - r` places back
    float o[4];
    const bool have = live && keep - r <= before;
    if (have) {
      if constexpr (W == 4) Vec4<float>::load(st + (size_t)r * p.hidden + i, o);
      else o[0] = st[(size_t)r * p.hidden + i];
    } else {
#pragma unroll
      for (int u = 0; u < W; ++u) o[u] = 0.f;
    }
#pragma unroll
    for (int u = 0; u < W; ++u) acc[u] = fmaf(p.conv_w[(size_t)(i + u) * p.taps + r], o[u], acc[u]);
    if (r > 0 && live) {
      if constexpr (W == 4) Vec4<float>::store(st + (size_t)(r - 1) * p.hidden + i, o);
      else st[(size_t)(r - 1) * p.hidden + i] = o[0];
    }
  }
  if (keep > 0 && live) {
#pragma unroll
    for (int u = 0; u < W; ++u) next[u] = h[u];
    if constexpr (W == 4) Vec4<float>::store(st + (size_t)(keep - 1) * p.hidden + i, next);
    else st[(size_t)(keep - 1) * p.hidden + i] = next[0];
  }
#pragma unroll
  for (int u = 0; u < W; ++u) acc[u] = to_float(from_float<T>(acc[u]));
  if constexpr (W == 4) {
    Vec4<T>::store((T*)p.conv_out + dst + i, acc);
    if (p.conv_out_f32) Vec4<float>::store(p.conv_out_f32 + dst + i, acc);
  } else {
    ((T*)p.conv_out)[dst + i] = from_float<T>(acc[0]);
    if (p.conv_out_f32) p.conv_out_f32[dst + i] = acc[0];
  }
}

// Where the row's request keeps its earlier inputs; false: nowhere (then the convolution sees zeros and keeps nothing).
__device__ __forceinline__ bool step_state(const FtkStreamStep& p, int row, float*& st, int& before) {
  st = nullptr;
  before = 0;
  if (!p.conv_w || p.taps < 2) return false;
  const int slot = p.state_slots[row];
  before = p.seg_info[(size_t)row * 4 + 2] - p.seg_info[(size_t)row * 4 + 1];
  if (slot < 0 || slot >= p.n_slots || before < 0 || p.seg_info[(size_t)row * 4] != row || p.seg_info[(size_t)row * 4 + 1] != 1)
    return false;
  st = p.state + (size_t)slot * (p.taps - 1) * p.hidden;
  return true;
}

// A row in registers: the block has `groups` teams of whole warps, a team takes one group, a thread PER runs of four
// elements.  What a row needs from memory is asked for at once, weights (and with CONV, one token per request, the taps
// and the request's earlier inputs, which a kernel of an earlier step wrote) before the wait on the kernel before.
// ROUTED: the result is a sum over expert routes.  TAPS: the tap count where it is four, else 0.
template <typename T, int PER, bool ROUTED, bool CONV, int TAPS, int MAX_THREADS>
__global__ void __launch_bounds__(MAX_THREADS, MAX_THREADS <= 256 && PER <= 3 ? 2 : 1) stream_step_regs_kernel(const __grid_constant__ StepArgs a) {
  const FtkStreamStep& p = a.p;
  __shared__ float red[2][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int team = warp / a.warps_per_group, team_threads = a.warps_per_group * 32;
  const int tl = threadIdx.x - team * team_threads;
  const int quads = a.group_size >> 2;
  const int r = blockIdx.x;
  int at[PER];   // first element of each run
  bool in[PER];
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    const int quad = q * team_threads + tl;
    in[q] = quad < quads;
    at[q] = team * a.group_size + (in[q] ? quad * 4 : 0);
  }
  float yv[PER][4], zv[PER][4], wp[PER][4], wr[PER][4], gb[PER][4];
  float cw[CONV && TAPS == 4 ? PER : 1][4][4], old[CONV && TAPS == 4 ? PER : 1][3][4];
  if (p.post_w) {
#pragma unroll
    for (int q = 0; q < PER; ++q) Vec4<float>::load(p.post_w + at[q], wp[q]);
  }
  if (p.pre_w) {
#pragma unroll
    for (int q = 0; q < PER; ++q) Vec4<float>::load(p.pre_w + at[q], wr[q]);
  }
#pragma unroll
  for (int q = 0; q < PER; ++q) gb[q][0] = gb[q][1] = gb[q][2] = gb[q][3] = 0.f;
  if (p.gate_bias) {
#pragma unroll
    for (int q = 0; q < PER; ++q) Vec4<float>::load(p.gate_bias + at[q], gb[q]);
  }
  float* st = nullptr;
  int before = 0;
  bool live = false;
  if constexpr (CONV) live = step_state(p, r, st, before);
  if constexpr (CONV && TAPS == 4) {
#pragma unroll
    for (int q = 0; q < PER; ++q)
#pragma unroll
      for (int u = 0; u < 4; ++u) Vec4<float>::load(p.conv_w + (size_t)(at[q] + u) * 4, cw[q][u]);
#pragma unroll
    for (int q = 0; q < PER; ++q)
#pragma unroll
      for (int j = 0; j < 3; ++j) {
        if (live && 3 - j <= before) Vec4<float>::load(st + (size_t)j * p.hidden + at[q], old[q][j]);
        else old[q][j][0] = old[q][j][1] = old[q][j][2] = old[q][j][3] = 0.f;
      }
  }
  pdl_wait();
  pdl_trigger();
  const int src_row = p.rows ? p.rows[r] : r;
  const size_t src = (size_t)src_row * p.hidden, dst = (size_t)r * p.hidden;
  const bool has_y = p.x != nullptr;
  float2 aux = make_float2(0.f, 1.f);
  if (ROUTED && p.aux) aux = *reinterpret_cast<const float2*>(p.aux + (size_t)src_row * 2);
#pragma unroll
  for (int q = 0; q < PER; ++q) Vec4<float>::load(p.residual + src + at[q], zv[q]);
  float ss = 0.f;
  if (has_y) {
    const T* x = (const T*)p.x;
    float gv[PER][4];
    if (p.gate) {
#pragma unroll
      for (int q = 0; q < PER; ++q) Vec4<T>::load((const T*)p.gate + src + at[q], gv[q]);
    }
    if constexpr (ROUTED) {
      Raw4<T> through[PER], common[PER];  // the token's own row and the shared expert's
      const bool passes = p.passed && aux.x != 0.f;
#pragma unroll
      for (int q = 0; q < PER; ++q) {
        yv[q][0] = yv[q][1] = yv[q][2] = yv[q][3] = 0.f;
        common[q] = raw_or_zero((const T*)p.shared + src + at[q], p.shared != nullptr);
        through[q] = raw_or_zero((const T*)p.passed + src + at[q], passes);
      }
      constexpr int J = PER <= 1 ? 8 : PER <= 3 ? 4 : 2;  // routes whose rows are asked for before the first is added
      for (int j0 = 0; j0 < p.top_k; j0 += J) {            // route order
        Raw4<T> y[J][PER];
        int pos[J];
#pragma unroll
        for (int j = 0; j < J; ++j) {
          pos[j] = j0 + j < p.top_k ? __ldg(p.route_pos + (size_t)src_row * p.top_k + j0 + j) : -1;
          if (pos[j] >= p.n_routes) pos[j] = -1;
        }
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
          for (int q = 0; q < PER; ++q) y[j][q] = raw_or_zero(x + (size_t)pos[j] * p.hidden + at[q], pos[j] >= 0);
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
          for (int q = 0; q < PER; ++q) {
            float v[4];
            y[j][q].widen(v);
#pragma unroll
            for (int u = 0; u < 4; ++u) yv[q][u] += v[u];
          }
      }
#pragma unroll
      for (int q = 0; q < PER; ++q) {
        float own[4], sh[4];
        through[q].widen(own);
        common[q].widen(sh);
#pragma unroll
        for (int u = 0; u < 4; ++u) yv[q][u] = fmaf(aux.y, sh[u], fmaf(aux.x, own[u], yv[q][u]));
      }
    } else {
#pragma unroll
      for (int q = 0; q < PER; ++q) Vec4<T>::load(x + src + at[q], yv[q]);
      if (p.x2) {
        float second[PER][4];
#pragma unroll
        for (int q = 0; q < PER; ++q) Vec4<T>::load((const T*)p.x2 + src + at[q], second[q]);
#pragma unroll
        for (int q = 0; q < PER; ++q)
#pragma unroll
          for (int u = 0; u < 4; ++u) yv[q][u] = fmaf(p.x2_scale, second[q][u], p.x_scale * yv[q][u]);
      }
    }
    if (p.gate) {
#pragma unroll
      for (int q = 0; q < PER; ++q)
#pragma unroll
        for (int u = 0; u < 4; ++u) yv[q][u] *= gate_sigmoid<T>(gv[q][u] + gb[q][u]);
    }
#pragma unroll
    for (int q = 0; q < PER; ++q)
      if (in[q]) {
#pragma unroll
        for (int u = 0; u < 4; ++u) ss = fmaf(yv[q][u], yv[q][u], ss);
      }
  }
  if (p.vec) {
#pragma unroll
    for (int q = 0; q < PER; ++q) {
      float v[4];
      Vec4<float>::load(p.vec + at[q], v);
#pragma unroll
      for (int u = 0; u < 4; ++u) zv[q][u] += v[u];
    }
  }
  auto team_sum = [&](float v, float* scratch) {
    v = warp_sum(v);
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int w = 0; w < a.warps_per_group; ++w) t += scratch[team * a.warps_per_group + w];
    return t;
  };
  if (has_y && !p.post_w) {
#pragma unroll
    for (int q = 0; q < PER; ++q)
#pragma unroll
      for (int u = 0; u < 4; ++u) zv[q][u] += yv[q][u];
  } else if (has_y) {
    const float inv = rsqrtf(team_sum(ss, red[0]) / (float)a.group_size + p.post_eps);
#pragma unroll
    for (int q = 0; q < PER; ++q)
#pragma unroll
      for (int u = 0; u < 4; ++u) zv[q][u] = fmaf(yv[q][u] * inv, wp[q][u], zv[q][u]);
  }
  float ss2 = 0.f;
  const bool changed = (has_y || p.vec) && !p.rows;
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    if (!in[q]) continue;
#pragma unroll
    for (int u = 0; u < 4; ++u) ss2 = fmaf(zv[q][u], zv[q][u], ss2);
    if (changed) Vec4<float>::store(p.residual + src + at[q], zv[q]);
    if (p.raw_out) Vec4<T>::store((T*)p.raw_out + (size_t)r * p.raw_stride + at[q], zv[q]);
  }
  if (!p.pre_w) return;
  const float inv = rsqrtf(team_sum(ss2, red[1]) / (float)a.group_size + p.pre_eps);
#pragma unroll
  for (int q = 0; q < PER; ++q) {
    if (!in[q]) continue;
    const int i = at[q];
    float y[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) y[u] = zv[q][u] * inv * wr[q][u];
    if (p.norm_f32 && !p.f32_rounded) Vec4<float>::store(p.norm_f32 + dst + i, y);
#pragma unroll
    for (int u = 0; u < 4; ++u) y[u] = to_float(from_float<T>(y[u]));
    if (p.norm_f32 && p.f32_rounded) Vec4<float>::store(p.norm_f32 + dst + i, y);
    if (p.out) Vec4<T>::store((T*)p.out + dst + i, y);
    if constexpr (CONV && TAPS == 4) {
      float acc[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        acc[u] = fmaf(cw[q][u][3], y[u], y[u]);
#pragma unroll
        for (int j = 0; j < 3; ++j) acc[u] = fmaf(cw[q][u][j], old[q][j][u], acc[u]);
        acc[u] = to_float(from_float<T>(acc[u]));
      }
      if (live) {
        Vec4<float>::store(st + i, old[q][1]);
        Vec4<float>::store(st + p.hidden + i, old[q][2]);
        Vec4<float>::store(st + 2 * (size_t)p.hidden + i, y);
      }
      Vec4<T>::store((T*)p.conv_out + dst + i, acc);
      if (p.conv_out_f32) Vec4<float>::store(p.conv_out_f32 + dst + i, acc);
    } else if constexpr (CONV) {
      step_conv<T, 4>(p, r, dst, i, y, live, st, before);
    }
  }
}

// Rows of any width in any number of groups, through shared memory: a warp takes a group's sum at a time.
template <typename T>
__global__ void __launch_bounds__(256) stream_step_any_kernel(const __grid_constant__ StepArgs a) {
  pdl_wait();
  pdl_trigger();
  const FtkStreamStep& p = a.p;
  extern __shared__ float sm[];  // [hidden] y, [hidden] stream, [groups] factors
  float* yrow = sm;
  float* zrow = sm + p.hidden;
  float* inv = zrow + p.hidden;
  const int r = blockIdx.x;
  const int src_row = p.rows ? p.rows[r] : r;
  const size_t src = (size_t)src_row * p.hidden, dst = (size_t)r * p.hidden;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const bool has_y = p.x != nullptr;
  float2 aux = make_float2(0.f, 1.f);
  if (has_y && p.aux) aux = *reinterpret_cast<const float2*>(p.aux + (size_t)src_row * 2);
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    zrow[i] = p.residual[src + i] + (p.vec ? p.vec[i] : 0.f);
    if (has_y) gated_result<T, 1>(p, src_row, src, i, aux, v);
    yrow[i] = v[0];
  }
  auto factors = [&](const float* row, float eps) {
    __syncthreads();
    for (int g = warp; g < p.groups; g += n_warps) {
      float s = 0.f;
      for (int i = lane; i < a.group_size; i += 32) {
        const float v = row[g * a.group_size + i];
        s = fmaf(v, v, s);
      }
      s = warp_sum(s);
      if (lane == 0) inv[g] = rsqrtf(s / (float)a.group_size + eps);
    }
    __syncthreads();
  };
  if (has_y && p.post_w) factors(yrow, p.post_eps);
  const bool changed = (has_y || p.vec) && !p.rows;
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    if (has_y) zrow[i] = p.post_w ? fmaf(yrow[i] * inv[i / a.group_size], p.post_w[i], zrow[i]) : zrow[i] + yrow[i];
    if (changed) p.residual[src + i] = zrow[i];
    if (p.raw_out) ((T*)p.raw_out)[(size_t)r * p.raw_stride + i] = from_float<T>(zrow[i]);
  }
  if (!p.pre_w) return;
  factors(zrow, p.pre_eps);
  float* st;
  int before;
  const bool live = step_state(p, r, st, before);
  for (int i = threadIdx.x; i < p.hidden; i += blockDim.x) {
    float y[4];
    y[0] = zrow[i] * inv[i / a.group_size] * p.pre_w[i];
    const float exact = y[0];
    y[0] = to_float(from_float<T>(y[0]));
    if (p.norm_f32) p.norm_f32[dst + i] = p.f32_rounded ? y[0] : exact;
    if (p.out) ((T*)p.out)[dst + i] = from_float<T>(y[0]);
    if (p.conv_w) step_conv<T, 1>(p, r, dst, i, y, live, st, before);
  }
}

}  // namespace ftk

using namespace ftk;

extern "C" int ftk_stream_step(const FtkStreamStep* args, void* stream) {
  FTK_REQUIRE(args, "stream_step: null arguments");
  const FtkStreamStep& p = *args;
  FTK_REQUIRE(dtype_ok(p.dtype), "stream_step: bad dtype %d", p.dtype);
  FTK_REQUIRE(p.n_rows >= 0 && p.hidden >= 1 && p.groups >= 1 && p.hidden % p.groups == 0,
              "stream_step: %d channels do not divide into %d groups", p.hidden, p.groups);
  if (p.n_rows == 0) return 0;
  FTK_REQUIRE(p.residual, "stream_step: null stream");
  FTK_REQUIRE(!p.x2 || (p.x && !p.route_pos), "stream_step: a second dense row goes with a first");
  FTK_REQUIRE(!p.route_pos || (p.x && p.top_k >= 1 && p.n_routes >= 0), "stream_step: bad routes");
  FTK_REQUIRE(!p.passed || p.aux, "stream_step: passed rows need their weights");
  FTK_REQUIRE(p.pre_w || (!p.out && !p.norm_f32 && !p.conv_w), "stream_step: an output needs the weight of the stream's norm");
  FTK_REQUIRE(!p.raw_out || p.raw_stride >= p.hidden, "stream_step: rows of the copy overlap");
  if (p.conv_w) {
    FTK_REQUIRE(p.taps >= 1 && p.taps <= kStepMaxTaps && p.conv_out && !p.rows, "stream_step: bad convolution");
    FTK_REQUIRE(p.taps == 1 || (p.state && p.state_slots && p.seg_info && p.n_slots >= 1), "stream_step: the convolution needs its state");
  }
  StepArgs a;
  a.p = p;
  a.group_size = p.hidden / p.groups;
  const int item = dtype_size(p.dtype);
  auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = a.group_size % 4 == 0 && al16(p.residual) && al16(p.x) && al16(p.x2) && al16(p.passed) && al16(p.shared) && al16(p.gate) &&
                   al16(p.gate_bias) && al16(p.post_w) && al16(p.pre_w) && al16(p.vec) && al16(p.out) && al16(p.norm_f32) &&
                   al16(p.conv_out) && al16(p.conv_out_f32) && al16(p.state) && al16(p.conv_w) && (p.raw_stride * item) % (4 * item) == 0 &&
                   (reinterpret_cast<uintptr_t>(p.raw_out) % (4 * item)) == 0;
  cudaStream_t s = (cudaStream_t)stream;
  // teams of warps: steps of single tokens spread a row over up to 768 threads (few rows, each as soon as possible), others
  // over up to 256 (many rows side by side)
  const bool conv = p.conv_w != nullptr, routed = p.route_pos != nullptr;
  const int quads = a.group_size / 4;
  auto shape = [&](int max_threads) {  // (warps a group, runs a thread)
    const int most = max_threads / 32 / p.groups;
    int w = conv ? (quads + 31) / 32 : (quads + 95) / 96;
    w = w < 1 ? 1 : (w > most ? most : w);
    a.warps_per_group = w;
    return w < 1 ? 1 << 20 : (quads + w * 32 - 1) / (w * 32);
  };
  int per = vec && p.groups <= 24 ? shape(conv ? 768 : 256) : 1 << 20;
  bool wide = conv;
  if (!conv && per > 4 && vec && p.groups <= 24) {
    per = shape(768);
    wide = true;
  }
  if (per <= 4 && !(wide && per > 2)) {
    const int threads = a.warps_per_group * 32 * p.groups;
    note_variant(conv ? "stream step: rows in registers, convolution" : "stream step: rows in registers");
#define FTK_STEP(TY, N, RT, CV, TP, MT) FTK_LAUNCH((stream_step_regs_kernel<TY, N, RT, CV, TP, MT>), p.n_rows, threads, 0, s, a)
#define FTK_STEP_R(TY, N, CV, TP, MT)            \
    do {                                         \
      if (routed) FTK_STEP(TY, N, true, CV, TP, MT); \
      else FTK_STEP(TY, N, false, CV, TP, MT);   \
    } while (0)
#define FTK_STEP_ALL(TY)                                                   \
    do {                                                                   \
      if (conv && p.taps == 4 && per <= 1) FTK_STEP_R(TY, 1, true, 4, 768); \
      else if (conv && per <= 1) FTK_STEP_R(TY, 1, true, 0, 768);          \
      else if (conv) FTK_STEP_R(TY, 2, true, 0, 768);                      \
      else if (wide) FTK_STEP_R(TY, 2, false, 0, 768);                     \
      else if (per <= 1) FTK_STEP_R(TY, 1, false, 0, 256);                 \
      else if (per <= 2) FTK_STEP_R(TY, 2, false, 0, 256);                 \
      else if (per <= 3) FTK_STEP_R(TY, 3, false, 0, 256);                 \
      else FTK_STEP_R(TY, 4, false, 0, 256);                               \
    } while (0)
    if (p.dtype == FTK_F32) FTK_STEP_ALL(float);
    else FTK_STEP_ALL(__nv_bfloat16);
#undef FTK_STEP_ALL
#undef FTK_STEP_R
#undef FTK_STEP
    FTK_LAUNCH_CHECK("stream_step");
    return 0;
  }
  a.warps_per_group = 1;
  const size_t smem = ((size_t)2 * p.hidden + p.groups) * sizeof(float);
  FTK_REQUIRE(smem <= 200 * 1024, "stream_step: rows of %d elements do not fit shared memory", p.hidden);
  note_variant("stream step: rows in shared memory");
  auto go = [&](auto kern) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    FTK_LAUNCH(kern, p.n_rows, 256, smem, s, a);
  };
  if (p.dtype == FTK_F32) go(stream_step_any_kernel<float>);
  else go(stream_step_any_kernel<__nv_bfloat16>);
  FTK_LAUNCH_CHECK("stream_step");
  return 0;
}
