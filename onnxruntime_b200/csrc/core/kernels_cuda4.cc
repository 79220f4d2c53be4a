// GPU op wrappers, part 4: the packed operators of hybrid decoders (com.ortb200 HyperConnectionNorm, PackedGatedDelta,
// PackedMLstm, GatedPagedAttention, LatentPagedAttention, ClampedSwiGLU, SoftCap) on the kernels of recurrent.cu, hybrid.cu,
// latent.cu, latent_decode_tc.cu, attn_prefill.cu and gqa.cu.
// Operands that the kernels do not take are an error here: none of these operators has another way to run on the GPU.
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>

#include <limits>

#include "cuda_ops.h"
#include "kernel.h"
#include "ortb200_kernels.h"
#include "session.h"

namespace ortb {

namespace {

using Ctx = OpKernelContext;
constexpr const char* FUSED = "com.ortb200";

int DtypeCode(at::ScalarType t) {
  if (t == at::kHalf) return ORTB200_F16;
  if (t == at::kBFloat16) return ORTB200_BF16;
  if (t == at::kFloat) return ORTB200_F32;
  ORTB_THROW(NOT_IMPLEMENTED, "type not supported by the GPU kernels");
}

// an operand the kernels read as it lies: on the GPU, of one type, contiguous
const at::Tensor& Want(Ctx& ctx, int i, at::ScalarType type, const char* what) {
  const at::Tensor& t = ctx.RequiredInput(i);
  ORTB_ENFORCE_ARG(t.is_cuda() && t.scalar_type() == type && t.is_contiguous(), ctx.node().op_type, ": ", what, " must be a contiguous ",
                   c10::toString(type), " tensor on the GPU");
  return t;
}
const float* OptFloats(Ctx& ctx, int i, int64_t numel, const char* what) {
  if (!ctx.HasInput(i)) return nullptr;
  const at::Tensor& t = Want(ctx, i, at::kFloat, what);
  ORTB_ENFORCE_ARG(numel < 0 || t.numel() == numel, ctx.node().op_type, ": ", what, " has ", t.numel(), " elements instead of ", numel);
  return t.data_ptr<float>();
}
const float* Floats(Ctx& ctx, int i, int64_t numel, const char* what) {
  ctx.RequiredInput(i);
  return OptFloats(ctx, i, numel, what);
}
int Pdl(Ctx& ctx) { return ctx.session()->config().Get("ortb200.pdl", "0") == "1" ? 1 : 0; }
int* Status(Ctx& ctx) { return ctx.session()->StatusWord().data_ptr<int>(); }

// Result of a sublayer: columns of `base` (an optional input that another sublayer has written its columns of), or a
// tensor of its own.
struct Columns {
  at::Tensor t;
  int64_t ld() const { return t.size(1); }
};
Columns ResultColumns(Ctx& ctx, int base, int64_t rows, int64_t cols, const at::Tensor& like) {
  if (!ctx.HasInput(base)) return {at::empty({rows, cols}, like.options())};
  const at::Tensor& b = Want(ctx, base, like.scalar_type(), "base");
  ORTB_ENFORCE_ARG(b.dim() == 2 && b.size(0) == rows && b.size(1) >= cols, ctx.node().op_type, ": base does not fit the result");
  return {b};
}

// The tensor-core kernels read a head's sink in the type of the activations; a constant one is converted once.
class TypedSink {
 public:
  TypedSink(const OpKernelInfo& info, int input) {
    if (const at::Tensor* s = info.constant_input(input)) sink_ = *s;
  }
  at::Tensor As(const at::Tensor& sink, at::ScalarType type) const {
    if (!sink_.defined()) return sink.to(type).contiguous();
    if (!typed_.defined() || typed_.scalar_type() != type) typed_ = sink_.to(sink.device(), type).contiguous();
    return typed_;
  }

 private:
  at::Tensor sink_;
  mutable at::Tensor typed_;
};

class HyperConnectionNormKernel final : public OpKernel {
 public:
  explicit HyperConnectionNormKernel(const OpKernelInfo& info) : OpKernel(info) {
    streams_ = info.node.attr_i("streams", 1);
    eps_ = info.node.attr_f("epsilon", 1e-6f);
  }
  void Compute(Ctx& ctx) const override {
    const at::Tensor& x = ctx.RequiredInput(0);
    const bool shared = x.dim() == 2, write = ctx.HasInput(1);
    const at::ScalarType type = write ? ctx.Input(1).scalar_type() : x.scalar_type();
    ORTB_ENFORCE_ARG(shared || (x.dim() == 3 && x.size(1) == streams_ && x.scalar_type() == at::kFloat), "HyperConnectionNorm: x must be float32 ",
                     "[tokens, streams, width] or [tokens, width]");
    ORTB_ENFORCE_ARG(!shared || x.scalar_type() == type, "HyperConnectionNorm: a shared stream must have the type of y");
    ORTB_ENFORCE_ARG(x.is_cuda() && x.is_contiguous(), "HyperConnectionNorm: x must be contiguous on the GPU");
    const int64_t T = x.size(0), W = x.size(-1);
    ortb200_hyper_norm_args a{};
    a.x = x.data_ptr();
    a.x_shared = shared ? 1 : 0;
    if (write) {
      const at::Tensor& y = Want(ctx, 1, type, "y");
      ORTB_ENFORCE_ARG(y.numel() == T * W, "HyperConnectionNorm: y must be [tokens, width]");
      a.y = y.data_ptr();
      a.mix = Floats(ctx, 2, streams_ * streams_, "mix");
      a.w_out = Floats(ctx, 3, streams_, "w_out");
    }
    a.w_in = Floats(ctx, 4, streams_, "w_in");
    a.gamma = Floats(ctx, 5, W, "gamma");
    a.T = static_cast<int>(T);
    a.num_rows = a.T;
    if (ctx.HasInput(6)) {
      const at::Tensor& rows = Want(ctx, 6, at::kLong, "rows");
      a.rows = rows.data_ptr<int64_t>();
      a.num_rows = static_cast<int>(rows.numel());
    }
    const bool keep = ctx.OutputCount() > 1 && ctx.OutputNeeded(1);
    ORTB_ENFORCE_ARG(!keep || a.rows == nullptr, "HyperConnectionNorm: selected rows cannot return the streams");
    at::Tensor out = at::empty({a.num_rows, W}, x.options().dtype(type));
    at::Tensor xo;
    if (keep) {
      xo = at::empty({T, streams_, W}, x.options().dtype(at::kFloat));
      a.x_out = xo.data_ptr<float>();
    }
    a.out = out.data_ptr();
    a.streams = static_cast<int>(streams_);
    a.width = static_cast<int>(W);
    a.eps = eps_;
    a.dtype = DtypeCode(type);
    a.use_pdl = Pdl(ctx);
    a.status = Status(ctx);
    if (a.num_rows > 0) {
      CheckLaunch(ortb200_hyper_norm(&a, ctx.cuda_stream()), "ortb200_hyper_norm");
      ctx.session()->AddLaunches(1);
    }
    ctx.SetOutput(0, out);
    if (keep) ctx.SetOutput(1, xo);
  }

 private:
  int64_t streams_ = 1;
  float eps_ = 1e-6f;
};

class SoftCapKernel final : public OpKernel {
 public:
  explicit SoftCapKernel(const OpKernelInfo& info) : OpKernel(info), cap_(info.node.attr_f("cap", 1.f)) {}
  void Compute(Ctx& ctx) const override {
    at::Tensor x = ctx.RequiredInput(0).contiguous();
    at::Tensor y = at::empty(x.sizes(), x.options().dtype(at::kFloat));
    if (x.numel() > 0) {
      CheckLaunch(ortb200_softcap(x.data_ptr(), y.data_ptr<float>(), x.numel(), cap_, DtypeCode(x.scalar_type()), ctx.cuda_stream()), "ortb200_softcap");
      ctx.session()->AddLaunches(1);
    }
    ctx.SetOutput(0, y);
  }

 private:
  float cap_ = 1.f;
};

class PackedGatedDeltaKernel final : public OpKernel {
 public:
  explicit PackedGatedDeltaKernel(const OpKernelInfo& info) : OpKernel(info) {
    const Node& n = info.node;
    H_ = n.attr_i("num_heads", 0);
    G_ = n.attr_i("kv_num_heads", 0);
    dk_ = n.attr_i("head_size", 0);
    dv_ = n.attr_i("v_head_size", 0);
    eps_ = n.attr_f("epsilon", 1e-6f);
    unit_eps_ = n.attr_f("unit_epsilon", 1e-6f);
  }
  void Compute(Ctx& ctx) const override {
    const at::Tensor& x = ctx.RequiredInput(0);
    const at::ScalarType type = x.scalar_type();
    Want(ctx, 0, type, "qkvb");
    const at::Tensor& low = Want(ctx, 1, type, "low");
    const at::Tensor& conv = Want(ctx, 2, at::kFloat, "conv");
    const at::Tensor& ring = Want(ctx, 6, type, "conv_state");
    const at::Tensor& state = Want(ctx, 7, at::kFloat, "state");
    const at::Tensor &cu = Want(ctx, 8, at::kInt, "cumulative lengths"), &past = Want(ctx, 9, at::kInt, "past lengths"),
                     &slots = Want(ctx, 10, at::kInt, "slots");
    const int64_t T = x.size(0), B = past.numel(), C = 2 * G_ * dk_ + H_ * dv_, taps = conv.size(1);
    ORTB_ENFORCE_ARG(conv.size(0) == C && low.numel() == T * H_ * (dk_ + dv_) && cu.numel() == B + 1 && slots.numel() == B && ring.dim() == 3 &&
                         ring.size(1) == taps && ring.size(2) == C && state.dim() == 4 && state.size(0) == ring.size(0) && state.size(1) == H_ &&
                         state.size(2) == dk_ && state.size(3) == dv_,
                     "PackedGatedDelta: sizes disagree");
    at::Tensor out = at::empty({T, H_ * dv_}, x.options());
    const int64_t bytes = ortb200_recurrent_workspace_bytes(static_cast<int>(T), static_cast<int>(B), static_cast<int>(H_), static_cast<int>(G_),
                                                            static_cast<int>(dk_), static_cast<int>(dv_));
    at::Tensor ws;
    if (bytes > 0) ws = at::empty({bytes}, x.options().dtype(at::kByte));
    ortb200_gated_delta_args a{};
    a.qkvb = x.data_ptr();
    a.low = low.data_ptr();
    a.conv = conv.data_ptr<float>();
    a.a_log = Floats(ctx, 3, H_, "a_log");
    a.dt_bias = Floats(ctx, 4, H_ * dk_, "dt_bias");
    a.norm = Floats(ctx, 5, dv_, "norm");
    a.conv_state = ring.data_ptr();
    a.state = state.data_ptr<float>();
    a.cu_seqlens = cu.data_ptr<int>();
    a.past_seqlens = past.data_ptr<int>();
    a.slots = slots.data_ptr<int>();
    a.out = out.data_ptr();
    a.workspace = bytes > 0 ? static_cast<float*>(ws.data_ptr()) : nullptr;
    a.workspace_bytes = bytes;
    a.T = static_cast<int>(T); a.B = static_cast<int>(B); a.ld = static_cast<int>(x.size(1));
    a.heads = static_cast<int>(H_); a.kv_heads = static_cast<int>(G_); a.dk = static_cast<int>(dk_); a.dv = static_cast<int>(dv_);
    a.taps = static_cast<int>(taps); a.num_slots = static_cast<int>(state.size(0));
    a.norm_eps = eps_;
    a.unit_eps = unit_eps_;
    a.dtype = DtypeCode(type);
    a.use_pdl = Pdl(ctx);
    a.status = Status(ctx);
    CheckLaunch(ortb200_gated_delta(&a, ctx.cuda_stream()), "ortb200_gated_delta");
    ctx.session()->AddLaunches(T == B ? 1 : 3);
    ctx.SetOutput(0, out);
    if (ctx.OutputCount() > 1) ctx.SetOutput(1, ring);
    if (ctx.OutputCount() > 2) ctx.SetOutput(2, state);
  }

 private:
  int64_t H_ = 0, G_ = 0, dk_ = 0, dv_ = 0;
  float eps_ = 1e-6f, unit_eps_ = 1e-6f;
};

class PackedMLstmKernel final : public OpKernel {
 public:
  explicit PackedMLstmKernel(const OpKernelInfo& info) : OpKernel(info) {
    const Node& n = info.node;
    H_ = n.attr_i("num_heads", 0);
    dk_ = n.attr_i("head_size", 0);
    dv_ = n.attr_i("v_head_size", 0);
    cap_ = n.attr_f("gate_cap", 1.f);
    eps_ = n.attr_f("epsilon", 1e-6f);
    den_eps_ = n.attr_f("denominator_epsilon", 1e-6f);
  }
  void Compute(Ctx& ctx) const override {
    const at::Tensor& x = ctx.RequiredInput(0);
    const at::ScalarType type = x.scalar_type();
    Want(ctx, 0, type, "packed projections");
    const at::Tensor &state = Want(ctx, 4, at::kFloat, "state"), &aux = Want(ctx, 5, at::kFloat, "aux");
    const at::Tensor &cu = Want(ctx, 6, at::kInt, "cumulative lengths"), &past = Want(ctx, 7, at::kInt, "past lengths"),
                     &slots = Want(ctx, 8, at::kInt, "slots");
    const int64_t T = x.size(0), B = past.numel();
    ORTB_ENFORCE_ARG(cu.numel() == B + 1 && slots.numel() == B && state.dim() == 4 && state.size(1) == H_ && state.size(2) == dk_ &&
                         state.size(3) == dv_ && aux.numel() == state.size(0) * H_ * (dk_ + 1),
                     "PackedMLstm: sizes disagree");
    at::Tensor out = at::empty({T, H_ * dv_}, x.options());
    const int64_t bytes = ortb200_recurrent_workspace_bytes(static_cast<int>(T), static_cast<int>(B), static_cast<int>(H_), static_cast<int>(H_),
                                                            static_cast<int>(dk_), static_cast<int>(dv_));
    at::Tensor ws;
    if (bytes > 0) ws = at::empty({bytes}, x.options().dtype(at::kByte));
    ortb200_mlstm_args a{};
    a.packed = x.data_ptr();
    a.i_bias = Floats(ctx, 1, H_, "input gate bias");
    a.f_bias = Floats(ctx, 2, H_, "forget gate bias");
    a.norm = Floats(ctx, 3, H_ * dv_, "norm");
    a.state = state.data_ptr<float>();
    a.aux = aux.data_ptr<float>();
    a.cu_seqlens = cu.data_ptr<int>();
    a.past_seqlens = past.data_ptr<int>();
    a.slots = slots.data_ptr<int>();
    a.out = out.data_ptr();
    a.workspace = bytes > 0 ? static_cast<float*>(ws.data_ptr()) : nullptr;
    a.workspace_bytes = bytes;
    a.T = static_cast<int>(T); a.B = static_cast<int>(B); a.ld = static_cast<int>(x.size(1));
    a.heads = static_cast<int>(H_); a.dk = static_cast<int>(dk_); a.dv = static_cast<int>(dv_);
    a.num_slots = static_cast<int>(state.size(0));
    a.gate_cap = cap_;
    a.norm_eps = eps_;
    a.den_eps = den_eps_;
    a.dtype = DtypeCode(type);
    a.use_pdl = Pdl(ctx);
    a.status = Status(ctx);
    CheckLaunch(ortb200_mlstm(&a, ctx.cuda_stream()), "ortb200_mlstm");
    ctx.session()->AddLaunches(T == B ? 1 : 3);
    ctx.SetOutput(0, out);
    if (ctx.OutputCount() > 1) ctx.SetOutput(1, state);
    if (ctx.OutputCount() > 2) ctx.SetOutput(2, aux);
  }

 private:
  int64_t H_ = 0, dk_ = 0, dv_ = 0;
  float cap_ = 1.f, eps_ = 1e-6f, den_eps_ = 1e-6f;
};

class GatedPagedAttentionKernel final : public OpKernel {
 public:
  explicit GatedPagedAttentionKernel(const OpKernelInfo& info) : OpKernel(info), sink_(info, 10) {
    const Node& n = info.node;
    N_ = n.attr_i("num_heads", 0);
    Nk_ = n.attr_i("kv_num_heads", 0);
    dk_ = n.attr_i("head_size", 0);
    dv_ = n.attr_i("v_head_size", 0);
    shared_ = n.attr_i("kv_shared", 0) != 0;
    gated_ = n.attr_i("gated", 0) != 0;
    window_ = n.attr_i("local_window_size", -1);
    scale_ = n.attr_f("scale", 1.f);
    eps_ = n.attr_f("epsilon", 1e-6f);
    chunk_ = info.node.attr_i("chunk_size", 0);
    first_offset_ = info.node.attr_i("first_values_offset", 0);
  }
  void Compute(Ctx& ctx) const override {
    const at::Tensor& x = ctx.RequiredInput(0);
    const at::ScalarType type = x.scalar_type();
    Want(ctx, 0, type, "packed projections");
    const at::Tensor &kc = Want(ctx, 1, type, "key cache"), &vc = Want(ctx, 2, type, "value cache");
    const at::Tensor &cu = Want(ctx, 3, at::kInt, "cumulative lengths"), &past = Want(ctx, 4, at::kInt, "past lengths"),
                     &table = Want(ctx, 5, at::kInt, "block table");
    const int64_t T = x.size(0), B = past.numel(), dkp = kc.size(3), dvp = vc.size(3), block = kc.size(1);
    const int64_t kv_cols = shared_ ? 0 : Nk_ * (dk_ + dv_);
    ORTB_ENFORCE_ARG(kc.dim() == 4 && vc.dim() == 4 && vc.size(0) == kc.size(0) && vc.size(1) == block && kc.size(2) == Nk_ && vc.size(2) == Nk_ &&
                         dkp >= dk_ && dvp >= dv_ && table.dim() == 2 && table.size(0) == B && cu.numel() == B + 1 &&
                         x.size(1) >= N_ * dk_ + kv_cols + (gated_ ? N_ * dv_ : 0),
                     "GatedPagedAttention: sizes disagree");
    const int dt = DtypeCode(type), pdl = Pdl(ctx);
    const bool decode = T == B;
    // 16-bit heads padded to 64 or 128: split-KV kernel for one token per sequence, tcgen05 flash kernel for prompts (its
    // key tiles must not cross a cache block)
    const bool heads_fit = type != at::kFloat && dkp == dvp && (dkp == 64 || dkp == 128) &&
                           ctx.session()->config().Get("ortb200.math_attention", "0") != "1";
    const bool tuned = heads_fit && (decode || block % 128 == 0);
    // queries without norm and rotation whose heads need no padding are read as they lie in the projections
    const bool q_in_place = tuned && dk_ == dkp && !ctx.HasInput(8) && !ctx.HasInput(6) && !shared_ && x.size(1) % 8 == 0;
    at::Tensor q = q_in_place ? x : at::empty({T, N_, dkp}, x.options());
    const int64_t q_ld = q_in_place ? x.size(1) : N_ * dkp;
    ortb200_qk_norm_rope_args p{};
    p.packed = x.data_ptr();
    p.q_out = q_in_place ? nullptr : q.data_ptr();
    if (ctx.HasInput(11)) {
      const at::Tensor& first = Want(ctx, 11, type, "first values");
      ORTB_ENFORCE_ARG(first.dim() == 2 && first.size(0) == T && first.size(1) >= first_offset_ + Nk_ * dv_, "GatedPagedAttention: sizes disagree");
      p.first_values = static_cast<const char*>(first.data_ptr()) + first_offset_ * first.element_size();
      p.first_ld = first.size(1);
      p.v_mix = Floats(ctx, 12, 1, "value mixing weight");
    }
    p.k_cache = kc.data_ptr();
    p.v_cache = vc.data_ptr();
    p.q_norm = OptFloats(ctx, 8, dk_, "query norm");
    p.k_norm = OptFloats(ctx, 9, dk_, "key norm");
    p.table_rows = 1 << 30;
    if (ctx.HasInput(6)) {
      p.cos_table = OptFloats(ctx, 6, -1, "cos table");
      p.sin_table = Floats(ctx, 7, ctx.Input(6).numel(), "sin table");
      p.rot_dim = static_cast<int>(ctx.Input(6).size(1) * 2);
      p.table_rows = static_cast<int>(ctx.Input(6).size(0));
    }
    p.cu_seqlens = cu.data_ptr<int>();
    p.past_seqlens = past.data_ptr<int>();
    p.block_table = table.data_ptr<int>();
    p.T = static_cast<int>(T); p.B = static_cast<int>(B); p.ld = static_cast<int>(x.size(1));
    p.N = static_cast<int>(N_); p.Nk = static_cast<int>(Nk_); p.dk = static_cast<int>(dk_); p.dv = static_cast<int>(dv_);
    p.dk_pad = static_cast<int>(dkp); p.dv_pad = static_cast<int>(dvp);
    p.block_size = static_cast<int>(block); p.max_blocks = static_cast<int>(table.size(1)); p.num_blocks = static_cast<int>(kc.size(0));
    p.kv_shared = shared_ ? 1 : 0;
    p.eps = eps_;
    p.dtype = dt;
    p.use_pdl = pdl;
    p.status = Status(ctx);
    CheckLaunch(ortb200_qk_norm_rope(&p, ctx.cuda_stream()), "ortb200_qk_norm_rope");

    const Columns result = ResultColumns(ctx, 13, T, N_ * dv_, x);
    const at::Tensor& out = result.t;
    const char* gate = gated_ ? static_cast<const char*>(x.data_ptr()) + (N_ * dk_ + kv_cols) * x.element_size() : nullptr;
    if (tuned) {
      // heads of full width without a gate go straight to the result
      const bool direct = !gated_ && dv_ == dvp && result.ld() % 8 == 0;
      at::Tensor padded = direct ? out : at::empty({T, N_, dvp}, x.options());
      const int64_t o_ld = direct ? result.ld() : N_ * dvp;
      at::Tensor sink;
      if (ctx.HasInput(10)) sink = sink_.As(ctx.Input(10), type);
      if (decode) {
        at::Tensor& ws = ctx.session()->AttnWorkspace(ortb200_gqa_decode_workspace_bytes(p.B, p.N, static_cast<int>(dkp)));
        ortb200_gqa_decode_args d{};
        d.q = q.data_ptr();
        d.k_cache = kc.data_ptr();
        d.v_cache = vc.data_ptr();
        d.seqlens_k = past.data_ptr<int>();  // total length - 1 of a one-token step
        d.head_sink = sink.defined() ? sink.data_ptr() : nullptr;
        d.out = padded.data_ptr();
        d.workspace = ws.data_ptr();
        d.workspace_bytes = ws.numel();
        d.B = p.B; d.N = p.N; d.Nk = p.Nk; d.H = static_cast<int>(dkp);
        d.Smax = static_cast<int>(table.size(1) * block);
        d.window = static_cast<int>(window_);
        d.scale = scale_;
        d.dtype = dt;
        d.use_pdl = pdl;
        d.status = p.status;
        d.block_table = p.block_table;
        d.block_size = p.block_size;
        d.max_blocks = p.max_blocks;
        d.num_blocks = p.num_blocks;
        d.split_weights = 1;
        d.chunk = static_cast<int>(chunk_);
        d.q_ld = q_ld;
        d.out_ld = o_ld;
        CheckLaunch(ortb200_gqa_decode(&d, ctx.cuda_stream()), "ortb200_gqa_decode(gated)");
      } else {
        ortb200_attn_prefill_args f{};
        f.q = q.data_ptr();
        f.k = kc.data_ptr();
        f.v = vc.data_ptr();
        f.head_sink = sink.defined() ? sink.data_ptr() : nullptr;
        f.out = padded.data_ptr();
        f.B = p.B; f.N = p.N; f.Nk = p.Nk; f.H = static_cast<int>(dkp);
        f.q_strides[0] = 0; f.q_strides[1] = q_ld; f.q_strides[2] = dkp;
        f.o_strides[0] = 0; f.o_strides[1] = o_ld; f.o_strides[2] = dvp;
        f.chunk = static_cast<int>(chunk_);
        f.causal = 1;
        f.window = static_cast<int>(window_);
        f.scale = scale_;
        f.dtype = dt;
        f.status = p.status;
        f.block_table = p.block_table;
        f.cu_seqlens = p.cu_seqlens;
        f.past_seqlens = p.past_seqlens;
        f.T = p.T; f.block_size = p.block_size; f.max_blocks = p.max_blocks; f.num_blocks = p.num_blocks;
        f.split_weights = 1;
        CheckLaunch(ortb200_attn_prefill(&f, ctx.cuda_stream()), "ortb200_attn_prefill(gated)");
      }
      if (!direct)
        CheckLaunch(ortb200_head_gate(padded.data_ptr(), gate, out.data_ptr(), p.T, p.N, p.dv, static_cast<int>(dvp), x.size(1), result.ld(), dt, pdl,
                                      ctx.cuda_stream()),
                    "ortb200_head_gate");
      ctx.session()->AddLaunches(direct ? 2 : 3);
    } else {
      ortb200_paged_attn_args g{};
      g.q = q.data_ptr();
      g.k_cache = kc.data_ptr();
      g.v_cache = vc.data_ptr();
      g.sink = OptFloats(ctx, 10, N_, "sink");
      g.gate = gate;
      g.out = out.data_ptr();
      g.cu_seqlens = p.cu_seqlens;
      g.past_seqlens = p.past_seqlens;
      g.block_table = p.block_table;
      g.gate_ld = x.size(1);
      g.T = p.T; g.B = p.B; g.N = p.N; g.Nk = p.Nk; g.dk = p.dk; g.dv = p.dv; g.dk_pad = p.dk_pad; g.dv_pad = p.dv_pad;
      g.block_size = p.block_size; g.max_blocks = p.max_blocks; g.num_blocks = p.num_blocks;
      g.window = static_cast<int>(window_);
      g.chunk = static_cast<int>(chunk_);
      g.out_ld = result.ld();
      g.scale = scale_;
      g.dtype = dt;
      g.use_pdl = pdl;
      CheckLaunch(ortb200_paged_attn(&g, ctx.cuda_stream()), "ortb200_paged_attn");
      ctx.session()->AddLaunches(2);
    }
    ctx.SetOutput(0, out);
    if (ctx.OutputCount() > 1) ctx.SetOutput(1, kc);
    if (ctx.OutputCount() > 2) ctx.SetOutput(2, vc);
  }

 private:
  int64_t N_ = 0, Nk_ = 0, dk_ = 0, dv_ = 0, window_ = -1, chunk_ = 0, first_offset_ = 0;
  bool shared_ = false, gated_ = false;
  float scale_ = 1.f, eps_ = 1e-6f;
  TypedSink sink_;
};

class LatentPagedAttentionKernel final : public OpKernel {
 public:
  explicit LatentPagedAttentionKernel(const OpKernelInfo& info) : OpKernel(info), sink_(info, 9) {
    const Node& n = info.node;
    N_ = n.attr_i("num_heads", 0);
    dk_ = n.attr_i("head_size", 0);
    dr_ = n.attr_i("rotary_size", 0);
    dv_ = n.attr_i("v_head_size", 0);
    rank_ = n.attr_i("latent_size", 0);
    wide_ = n.attr_i("latent_width", rank_);
    gated_ = n.attr_i("gated", 0) != 0;
    scale_ = n.attr_f("scale", 1.f);
    eps_ = n.attr_f("epsilon", 1e-6f);
  }
  void Compute(Ctx& ctx) const override {
    const at::Tensor& x = ctx.RequiredInput(0);
    const at::ScalarType type = x.scalar_type();
    Want(ctx, 0, type, "packed projections");
    const at::Tensor& cache = Want(ctx, 1, type, "latent cache");
    const at::Tensor &cu = Want(ctx, 2, at::kInt, "cumulative lengths"), &past = Want(ctx, 3, at::kInt, "past lengths"),
                     &table = Want(ctx, 4, at::kInt, "block table");
    const at::Tensor& up = Want(ctx, 8, type, "key and value maps");
    const int64_t T = x.size(0), B = past.numel(), width = cache.size(-1), q_cols = N_ * (dk_ + dr_), gate_col = q_cols + rank_ + dr_;
    ORTB_ENFORCE_ARG(cache.dim() == 3 && wide_ >= rank_ && width >= wide_ + dr_ && up.dim() == 2 && up.size(0) == N_ * (dk_ + dv_) && up.size(1) == rank_ &&
                         table.dim() == 2 && table.size(0) == B && cu.numel() == B + 1 && x.size(1) >= gate_col + (gated_ ? N_ : 0),
                     "LatentPagedAttention: sizes disagree");
    const int dt = DtypeCode(type), pdl = Pdl(ctx);
    const int block = static_cast<int>(cache.size(1)), max_blocks = static_cast<int>(table.size(1)), num_blocks = static_cast<int>(cache.size(0));
    const Columns result = ResultColumns(ctx, 10, T, N_ * dv_, x);
    ortb200_latent_prep_args p{};
    p.packed = x.data_ptr();
    p.cache = cache.data_ptr();
    p.norm = Floats(ctx, 7, rank_, "latent norm");
    if (ctx.HasInput(5)) {
      p.cos_table = OptFloats(ctx, 5, -1, "cos table");
      p.sin_table = Floats(ctx, 6, ctx.Input(5).numel(), "sin table");
      p.rot_dim = static_cast<int>(ctx.Input(5).size(1) * 2);
      p.table_rows = static_cast<int>(ctx.Input(5).size(0));
    }
    p.cu_seqlens = cu.data_ptr<int>();
    p.past_seqlens = past.data_ptr<int>();
    p.block_table = table.data_ptr<int>();
    p.T = static_cast<int>(T); p.B = static_cast<int>(B); p.ld = static_cast<int>(x.size(1));
    p.N = static_cast<int>(N_); p.dk = static_cast<int>(dk_); p.dr = static_cast<int>(dr_); p.rank = static_cast<int>(rank_);
    p.wide = static_cast<int>(wide_); p.width = static_cast<int>(width);
    p.block_size = block; p.max_blocks = max_blocks; p.num_blocks = num_blocks;
    p.eps = eps_;
    p.dtype = dt;
    p.use_pdl = pdl;
    p.status = Status(ctx);
    const char* gate = gated_ ? static_cast<const char*>(x.data_ptr()) + gate_col * x.element_size() : nullptr;
    // Few tokens per sequence: attend over the latents with absorbed queries.  Prompts: expand keys and values of all
    // tokens and run the flash kernel, whose heads are several times narrower than a latent.
    const bool prompt = T > 16 * B && ctx.HasInput(11) && rank_ % 8 == 0 && x.size(1) % 8 == 0 && result.ld() % 8 == 0 &&
                        ortb200_latent_prefill_supported(p.dk, p.dr, static_cast<int>(dv_), dt) != 0 &&
                        ctx.session()->config().Get("ortb200.math_attention", "0") != "1";
    if (prompt) {
      const at::Tensor& starts = ctx.RequiredInput(11);
      ORTB_ENFORCE_ARG(!starts.is_cuda() && starts.scalar_type() == at::kInt && starts.numel() == B + 1,
                       "LatentPagedAttention: key starts must be an int32 tensor in host memory");
      const int64_t rows = starts.data_ptr<int>()[B];
      ORTB_ENFORCE_ARG(rows >= T, "LatentPagedAttention: fewer keys than tokens");
      at::Tensor q_rot = at::empty({T, N_, dr_}, x.options()), c = at::empty({rows, rank_}, x.options()), kr = at::empty({rows, width - wide_}, x.options());
      p.q_rot = q_rot.data_ptr();
      if (rows == T) {   // nothing cached in front: the new entries are all there is
        p.c_out = c.data_ptr();
        p.k_rot_out = kr.data_ptr();
      }
      CheckLaunch(ortb200_latent_prep(&p, ctx.cuda_stream()), "ortb200_latent_prep");
      if (rows != T)
        CheckLaunch(ortb200_latent_gather(p.cache, p.cu_seqlens, p.past_seqlens, p.block_table, c.data_ptr(), kr.data_ptr(), static_cast<int>(rows), p.B,
                                          p.rank, p.wide, p.width, block, max_blocks, num_blocks, dt, pdl, p.status, ctx.cuda_stream()),
                    "ortb200_latent_gather");
      at::Tensor kv = LaunchGemm(ctx, c, up, N_ * (dk_ + dv_), 0, at::Tensor(), at::Tensor(), ORTB200_ACT_NONE, 1.f);
      at::Tensor sink;
      if (ctx.HasInput(9)) sink = sink_.As(ctx.Input(9), type);
      ortb200_latent_prefill_args f{};
      f.q = x.data_ptr();
      f.q_rot = q_rot.data_ptr();
      f.kv = kv.data_ptr();
      f.k_rot = kr.data_ptr();
      f.head_sink = sink.defined() ? sink.data_ptr() : nullptr;
      f.gate = gate;
      f.out = result.t.data_ptr();
      f.cu_seqlens = p.cu_seqlens;
      f.past_seqlens = p.past_seqlens;
      f.q_ld = x.size(1); f.kv_ld = N_ * (dk_ + dv_); f.k_rot_ld = width - wide_; f.gate_ld = x.size(1); f.out_ld = result.ld();
      f.T = p.T; f.B = p.B; f.N = p.N; f.dk = p.dk; f.dr = p.dr; f.dv = static_cast<int>(dv_); f.key_rows = static_cast<int>(rows);
      f.scale = scale_;
      f.dtype = dt;
      f.status = p.status;
      CheckLaunch(ortb200_latent_prefill(&f, ctx.cuda_stream()), "ortb200_latent_prefill");
      ctx.session()->AddLaunches(rows == T ? 2 : 3);
    } else {
      int parts = 1;
      const bool tc = ctx.session()->config().Get("ortb200.math_attention", "0") != "1" &&
                      ortb200_latent_decode_plan(p.T, p.N, p.wide, p.width, block, max_blocks, dt, &parts) != 0;
      if (!tc) parts = 1;
      at::Tensor q = at::empty({T, N_, width}, x.options().dtype(tc ? type : at::kFloat));
      p.up = up.data_ptr();
      p.q_abs = q.data_ptr();
      p.q_abs_f32 = tc ? 0 : 1;
      CheckLaunch(ortb200_latent_absorb(&p, ctx.cuda_stream()), "ortb200_latent_absorb");
      at::Tensor o = at::empty({T, N_, parts, wide_}, x.options().dtype(at::kFloat)), ml = at::empty({T, N_, parts, 2}, o.options());
      ortb200_latent_decode_args d{};
      d.q_abs = q.data_ptr();
      d.cache = p.cache;
      d.cu_seqlens = p.cu_seqlens; d.past_seqlens = p.past_seqlens; d.block_table = p.block_table;
      d.o = o.data_ptr<float>();
      d.ml = ml.data_ptr<float>();
      d.T = p.T; d.B = p.B; d.N = p.N; d.rank = p.rank; d.wide = p.wide; d.width = p.width; d.parts = parts;
      d.block_size = block; d.max_blocks = max_blocks; d.num_blocks = num_blocks;
      d.scale = scale_;
      d.dtype = dt;
      d.tensor_cores = tc ? 1 : 0;
      d.use_pdl = pdl;
      d.status = p.status;
      CheckLaunch(ortb200_latent_decode(&d, ctx.cuda_stream()), "ortb200_latent_decode");
      ortb200_latent_out_args o_args{};
      o_args.o = d.o;
      o_args.ml = d.ml;
      o_args.sink = OptFloats(ctx, 9, N_, "sink");
      o_args.up_v = static_cast<const char*>(up.data_ptr()) + N_ * dk_ * rank_ * up.element_size();
      o_args.gate = gate;
      o_args.out = result.t.data_ptr();
      o_args.gate_ld = x.size(1); o_args.out_ld = result.ld();
      o_args.T = p.T; o_args.N = p.N; o_args.dv = static_cast<int>(dv_); o_args.rank = p.rank; o_args.wide = p.wide; o_args.parts = parts;
      o_args.dtype = dt;
      o_args.use_pdl = pdl;
      CheckLaunch(ortb200_latent_out(&o_args, ctx.cuda_stream()), "ortb200_latent_out");
      ctx.session()->AddLaunches(3);
    }
    ctx.SetOutput(0, result.t);
    if (ctx.OutputCount() > 1) ctx.SetOutput(1, cache);
  }

 private:
  int64_t N_ = 0, dk_ = 0, dr_ = 0, dv_ = 0, rank_ = 0, wide_ = 0;
  bool gated_ = false;
  float scale_ = 1.f, eps_ = 1e-6f;
  TypedSink sink_;
};

// 32-bit models, and sizes outside the gated GEMM that the optimizer makes of this operator and its two MatMuls
class ClampedSwiGLUKernel final : public OpKernel {
 public:
  explicit ClampedSwiGLUKernel(const OpKernelInfo& info) : OpKernel(info) {
    const Node& n = info.node;
    limit_ = n.attr_f("limit", std::numeric_limits<float>::infinity());
    alpha_ = n.attr_f("alpha", 1.f);
    offset_ = n.attr_f("offset", 0.f);
    lead_ = n.attr_i("lead_columns", 0);
  }
  void Compute(Ctx& ctx) const override {
    at::Tensor gate = ctx.RequiredInput(0).contiguous(), up = ctx.RequiredInput(1).contiguous();
    ORTB_ENFORCE_ARG(gate.is_cuda() && up.is_cuda() && gate.sizes() == up.sizes() && gate.scalar_type() == up.scalar_type() && gate.dim() >= 1,
                     "ClampedSwiGLU: gate and up must agree");
    const int64_t cols = gate.size(-1), rows = cols > 0 ? gate.numel() / cols : 0;
    std::vector<int64_t> shape = gate.sizes().vec();
    shape.back() = lead_ + cols;
    at::Tensor y = at::empty(shape, gate.options());
    if (rows > 0) {
      CheckLaunch(ortb200_gated_unit(gate.data_ptr(), up.data_ptr(), static_cast<char*>(y.data_ptr()) + lead_ * y.element_size(), rows,
                                     static_cast<int>(cols), cols, lead_ + cols, ORTB200_ACT_CLAMPED_SWIGLU, limit_, alpha_, offset_,
                                     DtypeCode(gate.scalar_type()), Pdl(ctx), ctx.cuda_stream()),
                  "ortb200_gated_unit");
      ctx.session()->AddLaunches(1);
    }
    ctx.SetOutput(0, y);
  }

 private:
  float limit_ = 0.f, alpha_ = 1.f, offset_ = 0.f;
  int64_t lead_ = 0;
};

template <typename K>
void Reg(KernelRegistry& r, const std::string& op, std::vector<int> host = {}) {
  KernelDef d;
  d.host_inputs = std::move(host);
  d.domain = FUSED;
  d.op_type = op;
  d.factory = [](const OpKernelInfo& info) { return std::make_unique<K>(info); };
  r.Register(std::move(d));
}

}  // namespace

void RegisterCudaKernels4(KernelRegistry& r) {
  Reg<HyperConnectionNormKernel>(r, "HyperConnectionNorm");
  Reg<SoftCapKernel>(r, "SoftCap");
  Reg<PackedGatedDeltaKernel>(r, "PackedGatedDelta");
  Reg<PackedMLstmKernel>(r, "PackedMLstm");
  Reg<GatedPagedAttentionKernel>(r, "GatedPagedAttention");
  Reg<LatentPagedAttentionKernel>(r, "LatentPagedAttention", {11});
  Reg<ClampedSwiGLUKernel>(r, "ClampedSwiGLU");
}

}  // namespace ortb
