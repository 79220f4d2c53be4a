// com.ortb200 operators of hybrid decoders in packed serving form: hyper-connections, the gated delta rule with short
// convolutions, the exponentially gated matrix memory, gated paged attention, latent paged attention, the clamped gated
// linear unit and the soft cap.  These are the device-agnostic versions (tensor library, one token at a time where the mathematics is a recurrence); the GPU provider
// has its own kernels (kernels_cuda4.cc).
//
// Packed form: the tokens of all sequences lie behind one another, sequence b owns rows [cu[b], cu[b + 1]) and its first
// row sits at position past[b].  Recurrent state lives in pools indexed by slot and is updated in place; a sequence with
// past[b] = 0 starts from the zero state.
#include <ATen/ATen.h>

#include <cmath>
#include <limits>

#include "kernel.h"

namespace ortb {

namespace {

using Ctx = OpKernelContext;
constexpr int kMax = 1 << 30;
constexpr const char* FUSED = "com.ortb200";

std::vector<int64_t> HostInts(const at::Tensor& t) {
  at::Tensor c = t.to(at::kCPU, at::kLong).contiguous();
  return std::vector<int64_t>(c.data_ptr<int64_t>(), c.data_ptr<int64_t>() + c.numel());
}

at::Tensor F32(const at::Tensor& t) { return t.to(at::kFloat); }
at::Tensor Rms(const at::Tensor& x, double eps) { return x / at::sqrt(x.square().mean(-1, true) + eps); }

struct Packing {
  std::vector<int64_t> cu, past, slot;
  int64_t B() const { return static_cast<int64_t>(past.size()); }
};
Packing ReadPacking(Ctx& ctx, int cu, int past, int slot) {
  Packing p;
  p.cu = HostInts(ctx.RequiredInput(cu));
  p.past = HostInts(ctx.RequiredInput(past));
  if (slot >= 0) p.slot = HostInts(ctx.RequiredInput(slot));
  ORTB_ENFORCE_ARG(p.cu.size() == p.past.size() + 1 && (slot < 0 || p.slot.size() == p.past.size()),
                   "cumulative lengths, past lengths and slots disagree about the number of sequences");
  return p;
}

// inputs: x, y?, mix?, w_out?, w_in, gamma, rows?   outputs: normed, x_out?
void HyperConnectionNormImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const int64_t streams = n.attr_i("streams", 1);
  const at::Tensor& x_in = ctx.RequiredInput(0);
  const at::ScalarType out_type = ctx.HasInput(1) ? ctx.Input(1).scalar_type() : x_in.scalar_type();
  at::Tensor x = F32(x_in);
  if (x.dim() == 2) x = x.unsqueeze(1).expand({x.size(0), streams, x.size(1)});
  ORTB_ENFORCE_ARG(x.dim() == 3 && x.size(1) == streams, "HyperConnectionNorm: x must be [tokens, streams, width] or [tokens, width]");
  if (ctx.HasInput(1)) {
    x = at::einsum("st,nsw->ntw", {F32(ctx.RequiredInput(2)), x}) +
        F32(ctx.RequiredInput(3)).reshape({1, streams, 1}) * F32(ctx.Input(1)).unsqueeze(1);
  }
  if (ctx.OutputCount() > 1 && ctx.OutputNeeded(1)) ctx.SetOutput(1, x.contiguous());
  if (ctx.HasInput(6)) x = x.index_select(0, ctx.Input(6).to(x.device(), at::kLong));
  at::Tensor u = at::einsum("s,nsw->nw", {F32(ctx.RequiredInput(4)), x});
  ctx.SetOutput(0, (Rms(u, n.attr_f("epsilon", 1e-6f)) * F32(ctx.RequiredInput(5))).to(out_type));
}

// inputs: qkvb, low, conv, a_log, dt_bias, norm, conv_state, state, cu, past, slots
void PackedGatedDeltaImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const int64_t H = n.attr_i("num_heads", 0), G = n.attr_i("kv_num_heads", 0), dk = n.attr_i("head_size", 0), dv = n.attr_i("v_head_size", 0);
  const double eps = n.attr_f("epsilon", 1e-6f), unit_eps = n.attr_f("unit_epsilon", 1e-6f);
  const at::Tensor& qkvb = ctx.RequiredInput(0);
  at::Tensor conv = F32(ctx.RequiredInput(2));
  const int64_t T = qkvb.size(0), C = conv.size(0), K = conv.size(1);
  ORTB_ENFORCE_ARG(H > 0 && G > 0 && H % G == 0 && C == 2 * G * dk + H * dv && qkvb.size(1) >= C + H, "PackedGatedDelta: sizes disagree");
  at::Tensor x = qkvb.narrow(1, 0, C), beta = at::sigmoid(F32(qkvb.narrow(1, C, H)));
  at::Tensor low = F32(ctx.RequiredInput(1));
  at::Tensor rate = at::exp(F32(ctx.RequiredInput(3))).reshape({1, H, 1});
  at::Tensor z = low.narrow(1, 0, H * dk) + F32(ctx.RequiredInput(4)).reshape({1, H * dk});
  at::Tensor decay = at::exp(-rate * (z.clamp_min(0) + at::log1p(at::exp(-z.abs()))).reshape({T, H, dk}));
  at::Tensor gate = at::sigmoid(low.narrow(1, H * dk, H * dv)).reshape({T, H, dv});
  at::Tensor conv_state = ctx.RequiredInput(6), state = ctx.RequiredInput(7);
  const Packing p = ReadPacking(ctx, 8, 9, 10);
  at::Tensor out = at::zeros({T, H, dv}, qkvb.options().dtype(at::kFloat));
  for (int64_t b = 0; b < p.B(); ++b) {
    const int64_t t0 = p.cu[b], L = p.cu[b + 1] - t0, past = p.past[b];
    if (L == 0) continue;
    at::Tensor ring = conv_state[p.slot[b]];                                     // [K, C]
    // the K - 1 inputs in front of this call, oldest first
    at::Tensor virt = at::zeros({K - 1 + L, C}, x.options());
    for (int64_t j = 1; j < K; ++j)
      if (past - j >= 0) virt[K - 1 - j].copy_(ring[(past - j) % K]);
    virt.narrow(0, K - 1, L).copy_(x.narrow(0, t0, L));
    at::Tensor vf = F32(virt), y = at::zeros({L, C}, vf.options());
    for (int64_t j = 0; j < K; ++j) y = y + vf.narrow(0, j, L) * conv.select(1, j);
    y = y * at::sigmoid(y);
    at::Tensor q = y.narrow(1, 0, G * dk).reshape({L, G, dk}), k = y.narrow(1, G * dk, G * dk).reshape({L, G, dk});
    at::Tensor v = y.narrow(1, 2 * G * dk, H * dv).reshape({L, H, dv});
    q = (q / at::sqrt(q.square().sum(-1, true) + unit_eps) / std::sqrt(static_cast<double>(dk))).repeat_interleave(H / G, 1);
    k = (k / at::sqrt(k.square().sum(-1, true) + unit_eps)).repeat_interleave(H / G, 1);
    at::Tensor S = past == 0 ? at::zeros({H, dk, dv}, vf.options()) : state[p.slot[b]].clone();
    for (int64_t t = 0; t < L; ++t) {
      S = S * decay[t0 + t].unsqueeze(-1);
      at::Tensor u = beta[t0 + t].unsqueeze(-1) * (v[t] - at::matmul(k[t].unsqueeze(1), S).squeeze(1));
      S = S + k[t].unsqueeze(-1) * u.unsqueeze(1);
      out[t0 + t].copy_(at::matmul(q[t].unsqueeze(1), S).squeeze(1));
    }
    state[p.slot[b]].copy_(S);
    for (int64_t j = std::max<int64_t>(0, L - K); j < L; ++j) ring[(past + j) % K].copy_(x[t0 + j]);
  }
  out = Rms(out, eps) * F32(ctx.RequiredInput(5)) * gate;
  ctx.SetOutput(0, out.reshape({T, H * dv}).to(qkvb.scalar_type()));
  if (ctx.OutputCount() > 1) ctx.SetOutput(1, conv_state);
  if (ctx.OutputCount() > 2) ctx.SetOutput(2, state);
}

// inputs: packed, i_bias, f_bias, norm, state, aux, cu, past, slots
void PackedMLstmImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const int64_t H = n.attr_i("num_heads", 0), dk = n.attr_i("head_size", 0), dv = n.attr_i("v_head_size", 0);
  const double eps = n.attr_f("epsilon", 1e-6f), den_eps = n.attr_f("denominator_epsilon", 1e-6f), cap = n.attr_f("gate_cap", 1.f);
  const at::Tensor& x = ctx.RequiredInput(0);
  const int64_t T = x.size(0);
  ORTB_ENFORCE_ARG(H > 0 && x.size(1) >= H * (2 * dk + 2 * dv + 2), "PackedMLstm: sizes disagree");
  at::Tensor xf = F32(x);
  at::Tensor q = xf.narrow(1, 0, H * dk).reshape({T, H, dk}) / std::sqrt(static_cast<double>(dk));
  at::Tensor k = xf.narrow(1, H * dk, H * dk).reshape({T, H, dk});
  at::Tensor v = xf.narrow(1, 2 * H * dk, H * dv).reshape({T, H, dv});
  at::Tensor gate = at::sigmoid(xf.narrow(1, H * (2 * dk + dv), H * dv));
  at::Tensor gi = cap * at::tanh((xf.narrow(1, H * (2 * dk + 2 * dv), H) + F32(ctx.RequiredInput(1))) / cap);
  at::Tensor gf = at::log_sigmoid(cap * at::tanh((xf.narrow(1, H * (2 * dk + 2 * dv + 1), H) + F32(ctx.RequiredInput(2))) / cap));
  at::Tensor state = ctx.RequiredInput(4), aux = ctx.RequiredInput(5);
  const Packing p = ReadPacking(ctx, 6, 7, 8);
  at::Tensor out = at::zeros({T, H, dv}, xf.options());
  for (int64_t b = 0; b < p.B(); ++b) {
    const int64_t t0 = p.cu[b], L = p.cu[b + 1] - t0;
    if (L == 0) continue;
    at::Tensor S = at::zeros({H, dk, dv}, xf.options()), nrm = at::zeros({H, dk}, xf.options()), m = at::zeros({H}, xf.options());
    if (p.past[b] > 0) {
      S = state[p.slot[b]].clone();
      nrm = aux[p.slot[b]].narrow(1, 0, dk).clone();
      m = aux[p.slot[b]].select(1, dk).clone();
    }
    for (int64_t t = t0; t < t0 + L; ++t) {
      at::Tensor m_new = at::maximum(gf[t] + m, gi[t]);
      at::Tensor keep = at::exp(gf[t] + m - m_new), add = at::exp(gi[t] - m_new);
      at::Tensor ik = k[t] * add.unsqueeze(-1);
      S = S * keep.reshape({H, 1, 1}) + ik.unsqueeze(-1) * v[t].unsqueeze(1);
      nrm = nrm * keep.unsqueeze(-1) + ik;
      m = m_new;
      at::Tensor den = at::maximum((nrm * q[t]).sum(-1).abs(), at::exp(-m)) + den_eps;
      out[t].copy_(at::matmul(q[t].unsqueeze(1), S).squeeze(1) / den.unsqueeze(-1));
    }
    state[p.slot[b]].copy_(S);
    aux[p.slot[b]].copy_(at::cat({nrm, m.unsqueeze(-1)}, 1));
  }
  out = Rms(out, eps).reshape({T, H * dv}) * F32(ctx.RequiredInput(3)) * gate;
  ctx.SetOutput(0, out.to(x.scalar_type()));
  if (ctx.OutputCount() > 1) ctx.SetOutput(1, state);
  if (ctx.OutputCount() > 2) ctx.SetOutput(2, aux);
}

// A parallel block writes its two sublayers into the columns of one tensor: `base` (when given) receives y in its first
// columns and is the result.
void SetColumns(Ctx& ctx, int base, const at::Tensor& y) {
  if (!ctx.HasInput(base)) {
    ctx.SetOutput(0, y);
    return;
  }
  at::Tensor b = ctx.Input(base);
  ORTB_ENFORCE_ARG(b.dim() == 2 && b.size(0) == y.size(0) && b.size(1) >= y.size(1) && b.scalar_type() == y.scalar_type(), ctx.node().op_type,
                   ": base does not fit the result");
  b.narrow(1, 0, y.size(1)).copy_(y);
  ctx.SetOutput(0, b);
}

// softmax over the last axis of s [heads, L, total], optionally with one more term per head in the denominator
at::Tensor SoftmaxWithSink(at::Tensor s, Ctx& ctx, int sink) {
  const int64_t N = s.size(0), L = s.size(1), total = s.size(2);
  if (ctx.HasInput(sink)) s = at::cat({s, F32(ctx.Input(sink)).reshape({N, 1, 1}).expand({N, L, 1})}, 2);
  return at::softmax(s, -1).narrow(2, 0, total);
}

// inputs: packed, key_cache, value_cache, cu, past, block_table, cos?, sin?, q_norm?, k_norm?, sink?, first_values?, v_mix?, base?
void GatedPagedAttentionImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const int64_t N = n.attr_i("num_heads", 0), Nk = n.attr_i("kv_num_heads", 0), dk = n.attr_i("head_size", 0), dv = n.attr_i("v_head_size", 0);
  const bool shared = n.attr_i("kv_shared", 0) != 0, gated = n.attr_i("gated", 0) != 0;
  const double eps = n.attr_f("epsilon", 1e-6f), scale = n.attr_f("scale", 1.f);
  const int64_t window = n.attr_i("local_window_size", -1), chunk = n.attr_i("chunk_size", 0);
  const at::Tensor& packed = ctx.RequiredInput(0);
  at::Tensor kc = ctx.RequiredInput(1), vc = ctx.RequiredInput(2);
  const int64_t T = packed.size(0), block_size = kc.size(1), kv_cols = shared ? 0 : Nk * (dk + dv);
  ORTB_ENFORCE_ARG(N > 0 && Nk > 0 && N % Nk == 0 && kc.size(3) >= dk && vc.size(3) >= dv && packed.size(1) >= N * dk + kv_cols + (gated ? N * dv : 0),
                   "GatedPagedAttention: sizes disagree");
  const Packing p = ReadPacking(ctx, 3, 4, -1);
  at::Tensor table = ctx.RequiredInput(5).to(at::kCPU, at::kLong);
  at::Tensor xf = F32(packed);
  at::Tensor q = xf.narrow(1, 0, N * dk).reshape({T, N, dk}), k, v;
  if (ctx.HasInput(8)) q = Rms(q, eps) * F32(ctx.Input(8));
  if (!shared) {
    k = xf.narrow(1, N * dk, Nk * dk).reshape({T, Nk, dk});
    v = packed.narrow(1, (N + Nk) * dk, Nk * dv).reshape({T, Nk, dv});
    if (ctx.HasInput(9)) k = Rms(k, eps) * F32(ctx.Input(9));
    if (ctx.HasInput(11)) {   // values of another layer for the same tokens, mixed in before they are stored
      at::Tensor first = F32(ctx.Input(11).narrow(1, n.attr_i("first_values_offset", 0), Nk * dv)).reshape({T, Nk, dv});
      at::Tensor m = F32(ctx.RequiredInput(12)).reshape({1, 1, 1});
      v = ((1 - m) * F32(v) + m * first).to(vc.scalar_type());
    }
  }
  auto rotate = [&](const at::Tensor& x, int64_t first) {   // x [L, heads, dk]
    if (!ctx.HasInput(6)) return x;
    const int64_t half = ctx.Input(6).size(1), L = x.size(0);
    ORTB_ENFORCE_ARG(first + L <= ctx.Input(6).size(0), "GatedPagedAttention: position beyond the rotary tables");
    at::Tensor c = F32(ctx.Input(6)).narrow(0, first, L).unsqueeze(1), s = F32(ctx.RequiredInput(7)).narrow(0, first, L).unsqueeze(1);
    at::Tensor u = x.narrow(2, 0, half), w = x.narrow(2, half, half);
    return at::cat({u * c - w * s, w * c + u * s, x.narrow(2, 2 * half, dk - 2 * half)}, 2);
  };
  at::Tensor out = at::zeros({T, N, dv}, xf.options());
  for (int64_t b = 0; b < p.B(); ++b) {
    const int64_t t0 = p.cu[b], L = p.cu[b + 1] - t0, past = p.past[b], total = past + L;
    if (L == 0) continue;
    at::Tensor qb = rotate(q.narrow(0, t0, L), past).to(packed.scalar_type()).to(at::kFloat);
    if (!shared) {
      at::Tensor kb = rotate(k.narrow(0, t0, L), past).to(kc.scalar_type());
      for (int64_t s = 0; s < L; ++s) {
        const int64_t blk = table[b][(past + s) / block_size].item<int64_t>(), off = (past + s) % block_size;
        kc[blk][off].narrow(1, 0, dk).copy_(kb[s]);
        vc[blk][off].narrow(1, 0, dv).copy_(v[t0 + s]);
      }
    }
    const int64_t nblk = (total + block_size - 1) / block_size;
    at::Tensor blocks = table[b].narrow(0, 0, nblk).to(kc.device());
    auto gather = [&](const at::Tensor& c, int64_t d) {
      return F32(c.index_select(0, blocks).reshape({nblk * block_size, Nk, c.size(3)}).narrow(0, 0, total).narrow(2, 0, d))
          .permute({1, 0, 2}).repeat_interleave(N / Nk, 0);                    // [N, total, d]
    };
    at::Tensor s = at::matmul(qb.permute({1, 0, 2}), gather(kc, dk).transpose(1, 2)) * scale;   // [N, L, total]
    at::Tensor qpos = (at::arange(L, s.options().dtype(at::kLong)) + past).unsqueeze(1);
    at::Tensor kpos = at::arange(total, s.options().dtype(at::kLong)).unsqueeze(0);
    at::Tensor hidden = kpos.gt(qpos);
    if (window > 0) hidden = hidden.logical_or(kpos.le(qpos - window));
    if (chunk > 0) hidden = hidden.logical_or(kpos.lt(qpos - qpos.remainder(chunk)));
    s = s.masked_fill(hidden.unsqueeze(0), -std::numeric_limits<float>::infinity());
    at::Tensor w = SoftmaxWithSink(s, ctx, 10);
    out.narrow(0, t0, L).copy_(at::matmul(w, gather(vc, dv)).permute({1, 0, 2}));
  }
  out = out.reshape({T, N * dv});
  if (gated) out = out * at::sigmoid(xf.narrow(1, N * dk + kv_cols, N * dv));
  SetColumns(ctx, 13, out.to(packed.scalar_type()));
  if (ctx.OutputCount() > 1) ctx.SetOutput(1, kc);
  if (ctx.OutputCount() > 2) ctx.SetOutput(2, vc);
}

// inputs: packed, cache, cu, past, block_table, cos?, sin?, norm, up, sink?, base?, key_starts?
// packed: q (heads * (head_size + rot)) | latent (rank) | rotated key part (rot) | gate (heads).  A cache entry is the
// normed latent, zero-padded to `latent_width`, and the rotated key part behind it.  up: rows of the key map (heads *
// head_size), then of the value map (heads * v_head_size), each of `rank` columns.
void LatentPagedAttentionImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const int64_t N = n.attr_i("num_heads", 0), dk = n.attr_i("head_size", 0), dr = n.attr_i("rotary_size", 0), dv = n.attr_i("v_head_size", 0),
                rank = n.attr_i("latent_size", 0), wide = n.attr_i("latent_width", rank);
  const bool gated = n.attr_i("gated", 0) != 0;
  const double eps = n.attr_f("epsilon", 1e-6f), scale = n.attr_f("scale", 1.f);
  const at::Tensor& packed = ctx.RequiredInput(0);
  at::Tensor cache = ctx.RequiredInput(1);
  const at::Tensor& up = ctx.RequiredInput(8);
  const int64_t T = packed.size(0), block_size = cache.size(1), q_cols = N * (dk + dr);
  ORTB_ENFORCE_ARG(N > 0 && rank > 0 && wide >= rank && cache.dim() == 3 && cache.size(2) >= wide + dr && up.dim() == 2 && up.size(0) == N * (dk + dv) &&
                       up.size(1) == rank && packed.size(1) >= q_cols + rank + dr + (gated ? N : 0),
                   "LatentPagedAttention: sizes disagree");
  const Packing p = ReadPacking(ctx, 2, 3, -1);
  at::Tensor table = ctx.RequiredInput(4).to(at::kCPU, at::kLong);
  at::Tensor xf = F32(packed);
  at::Tensor q = xf.narrow(1, 0, q_cols).reshape({T, N, dk + dr});
  at::Tensor c = (Rms(xf.narrow(1, q_cols, rank), eps) * F32(ctx.RequiredInput(7))).to(cache.scalar_type());
  at::Tensor kr = xf.narrow(1, q_cols + rank, dr).unsqueeze(1);
  // x [L, heads, dr]: neighbours (2 i, 2 i + 1) turn together
  auto rotate = [&](const at::Tensor& x, int64_t first) {
    if (!ctx.HasInput(5)) return x;
    const int64_t half = ctx.Input(5).size(1), L = x.size(0);
    ORTB_ENFORCE_ARG(first + L <= ctx.Input(5).size(0) && 2 * half <= dr, "LatentPagedAttention: position or size beyond the rotary tables");
    at::Tensor cs = F32(ctx.Input(5)).narrow(0, first, L).unsqueeze(1), sn = F32(ctx.RequiredInput(6)).narrow(0, first, L).unsqueeze(1);
    at::Tensor pairs = x.narrow(2, 0, 2 * half).reshape({L, x.size(1), half, 2});
    at::Tensor u = pairs.select(3, 0), v = pairs.select(3, 1);
    at::Tensor turned = at::stack({u * cs - v * sn, v * cs + u * sn}, 3).reshape({L, x.size(1), 2 * half});
    return at::cat({turned, x.narrow(2, 2 * half, dr - 2 * half)}, 2);
  };
  at::Tensor upf = F32(up);
  at::Tensor uk = upf.narrow(0, 0, N * dk).reshape({N, dk, rank}), uv = upf.narrow(0, N * dk, N * dv).reshape({N, dv, rank});
  at::Tensor out = at::zeros({T, N, dv}, xf.options());
  for (int64_t b = 0; b < p.B(); ++b) {
    const int64_t t0 = p.cu[b], L = p.cu[b + 1] - t0, past = p.past[b], total = past + L;
    if (L == 0) continue;
    at::Tensor krb = rotate(kr.narrow(0, t0, L), past).to(cache.scalar_type());
    for (int64_t s = 0; s < L; ++s) {
      at::Tensor entry = cache[table[b][(past + s) / block_size].item<int64_t>()][(past + s) % block_size];
      entry.narrow(0, 0, rank).copy_(c[t0 + s]);
      entry.narrow(0, wide, dr).copy_(krb[s][0]);
    }
    const int64_t nblk = (total + block_size - 1) / block_size;
    at::Tensor all = F32(cache.index_select(0, table[b].narrow(0, 0, nblk).to(cache.device())).reshape({nblk * block_size, cache.size(2)}).narrow(0, 0, total));
    at::Tensor cl = all.narrow(1, 0, rank), qb = q.narrow(0, t0, L);
    at::Tensor qa = at::matmul(qb.narrow(2, 0, dk).permute({1, 0, 2}), uk);                                            // [N, L, rank]
    at::Tensor qr = rotate(qb.narrow(2, dk, dr), past).permute({1, 0, 2});
    at::Tensor s = (at::matmul(qa, cl.t()) + at::matmul(qr, all.narrow(1, wide, dr).t())) * scale;                     // [N, L, total]
    at::Tensor qpos = (at::arange(L, s.options().dtype(at::kLong)) + past).unsqueeze(1);
    at::Tensor kpos = at::arange(total, s.options().dtype(at::kLong)).unsqueeze(0);
    s = s.masked_fill(kpos.gt(qpos).unsqueeze(0), -std::numeric_limits<float>::infinity());
    at::Tensor o = at::matmul(at::matmul(SoftmaxWithSink(s, ctx, 9), cl), uv.transpose(1, 2));                         // [N, L, dv]
    out.narrow(0, t0, L).copy_(o.permute({1, 0, 2}));
  }
  if (gated) out = out * at::sigmoid(xf.narrow(1, q_cols + rank + dr, N)).unsqueeze(2);
  SetColumns(ctx, 10, out.reshape({T, N * dv}).to(packed.scalar_type()));
  if (ctx.OutputCount() > 1) ctx.SetOutput(1, cache);
}

// y = g sigmoid(alpha g) (u + offset), g = min(gate, limit), u = clamp(up, -limit, limit), behind `lead_columns` columns
// that another operator fills
void ClampedSwiGLUImpl(Ctx& ctx) {
  const Node& n = ctx.node();
  const double limit = n.attr_f("limit", std::numeric_limits<float>::infinity()), alpha = n.attr_f("alpha", 1.f), offset = n.attr_f("offset", 0.f);
  const at::Tensor& gate = ctx.RequiredInput(0);
  at::Tensor g = F32(gate).clamp_max(limit), u = F32(ctx.RequiredInput(1)).clamp(-limit, limit);
  at::Tensor y = (g * at::sigmoid(alpha * g) * (u + offset)).to(gate.scalar_type());
  const int64_t lead = n.attr_i("lead_columns", 0);
  if (lead > 0) {
    std::vector<int64_t> shape = y.sizes().vec();
    shape.back() = lead;
    y = at::cat({at::zeros(shape, y.options()), y}, -1);
  }
  ctx.SetOutput(0, y);
}

}  // namespace

void RegisterHybridKernels(KernelRegistry& r) {
  r.RegisterFn(FUSED, "HyperConnectionNorm", 1, kMax, HyperConnectionNormImpl);
  r.RegisterFn(FUSED, "PackedGatedDelta", 1, kMax, PackedGatedDeltaImpl);
  r.RegisterFn(FUSED, "PackedMLstm", 1, kMax, PackedMLstmImpl);
  r.RegisterFn(FUSED, "GatedPagedAttention", 1, kMax, GatedPagedAttentionImpl);
  r.RegisterFn(FUSED, "LatentPagedAttention", 1, kMax, LatentPagedAttentionImpl, {11});
  r.RegisterFn(FUSED, "ClampedSwiGLU", 1, kMax, ClampedSwiGLUImpl);
  r.RegisterFn(FUSED, "SoftCap", 1, kMax, [](Ctx& ctx) {
    const double cap = ctx.node().attr_f("cap", 1.f);
    ctx.SetOutput(0, at::tanh(F32(ctx.RequiredInput(0)) / cap) * cap);
  });
}

}  // namespace ortb
