// Python bindings of the mixers with a recurrent state: an extension of its own, so that a process that
// serves only such a model compiles and loads nothing else.
#include "binding_util.h"
#include "launch.h"
#include "mixers.h"

namespace {
using namespace llm_binding;

const __nv_bfloat16* bf16(const Tensor& t, const char* name) {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kBFloat16, name, " must be bfloat16");
    return reinterpret_cast<const __nv_bfloat16*>(t.data_ptr());
}
void want_aligned(const Tensor& t, const char* name) { TORCH_CHECK(reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, name, " must be 16-byte aligned"); }

// What the linear-attention entry points share.  offs: first columns of q, k, v, g; state: S (, n, m); gates with bias_i, bias_f, cap: mLSTM; decay: retention
llm::LinearParams linear_params(const Tensor& in, const std::vector<int64_t>& offs, const OptTensor& gates, const OptTensor& bias_i, const OptTensor& bias_f, double cap,
                                const OptTensor& decay, const OptTensor& angles, double q_scale, double k_scale, const OptTensor& cu, const Tensor& positions,
                                const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps, bool silu_in, bool raw) {
    llm::LinearParams p = {};
    p.silu_in = silu_in; p.raw = raw;
    is_f32(in, "in");
    const int64_t T = in.size(0);
    TORCH_CHECK(offs.size() == 4 && (state.size() == 1 || state.size() == 3), "offsets / state");
    const Tensor& S = state[0];
    want(S, torch::kFloat32, "S");
    TORCH_CHECK(S.dim() == 4, "S must be [slots, heads, vdim, dim]");
    p.n_slots = S.size(0); p.heads = S.size(1); p.vdim = S.size(2); p.dim = S.size(3);
    TORCH_CHECK(in.stride(1) == 1 && in.size(1) >= std::max(std::max(offs[0], offs[1]) + p.heads * p.dim, std::max(offs[2], offs[3]) + p.heads * p.vdim), "in: too few columns");
    p.in = in.data_ptr(); p.in_row = in.stride(0);
    p.q_off = offs[0]; p.k_off = offs[1]; p.v_off = offs[2]; p.g_off = offs[3];
    p.S = S.data_ptr<float>();
    TORCH_CHECK(gates.has_value() != decay.has_value() && gates.has_value() == (state.size() == 3), "either gates (with n and m) or decays");
    if (gates) {
        TORCH_CHECK(is_f32(*gates, "gates") && gates->dim() == 2 && gates->size(0) == T && gates->size(1) == 2 * p.heads && gates->stride(1) == 1, "gates must be float [tokens, 2 heads]");
        p.gates = gates->data_ptr<float>(); p.gate_row = gates->stride(0);
        p.bias_i = floats(bias_i.value(), p.heads, "bias_i"); p.bias_f = floats(bias_f.value(), p.heads, "bias_f");
        p.cap = cap;
        p.n = const_cast<float*>(floats(state[1], (int64_t)p.n_slots * p.heads * p.dim, "n"));
        p.m = const_cast<float*>(floats(state[2], (int64_t)p.n_slots * p.heads, "m"));
    } else {
        p.decay = floats(*decay, p.heads, "decay");
    }
    if (angles) {
        p.angles = angle_ptr(*angles, T); p.half = angles->size(1);
        TORCH_CHECK(2 * p.half <= p.dim, "more angles than a head has pairs");
    }
    p.q_scale = q_scale; p.k_scale = k_scale;
    if (cu) { p.cu = ints(*cu, "cu"); TORCH_CHECK(cu->numel() == slots.numel() + 1, "cu"); }
    else TORCH_CHECK(slots.numel() == T, "one row per sequence");
    p.positions = ints(positions, "positions"); p.slots = ints(slots, "slots");
    TORCH_CHECK(positions.numel() == T, "positions");
    p.true_vdim = true_vdim;
    if (norm_w) p.norm_w = floats(*norm_w, (int64_t)p.heads * p.vdim, "norm_w");
    p.silu = silu;
    TORCH_CHECK(out.dim() == 2 && out.size(0) == T && out.size(1) == p.heads * p.vdim && out.stride(1) == 1, "out must be [tokens, heads * vdim]");
    p.out = out.data_ptr(); p.out_row = out.stride(0);
    p.eps = eps;
    return p;
}

void linear_rows(const Tensor& in, const std::vector<int64_t>& offs, const OptTensor& gates, const OptTensor& bias_i, const OptTensor& bias_f, double cap,
                 const OptTensor& decay, const OptTensor& angles, double q_scale, double k_scale, const OptTensor& cu, const Tensor& positions,
                 const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps, bool silu_in, bool raw) {
    const llm::LinearParams p = linear_params(in, offs, gates, bias_i, bias_f, cap, decay, angles, q_scale, k_scale, cu, positions, slots, state, true_vdim, norm_w, silu, out, eps, silu_in, raw);
    check(llm::launch_linear_rows(p, slots.numel(), is_f32(in, "in"), is_f32(out, "out"), stream()), "linear_rows");
}

// chunks, seqs: int32 [n, 4], see LinearChunks.  cu is the host's view of the sequences and stays unused on the device.
void linear_chunk(const Tensor& in, const std::vector<int64_t>& offs, const OptTensor& gates, const OptTensor& bias_i, const OptTensor& bias_f, double cap,
                  const OptTensor& decay, const OptTensor& angles, double q_scale, double k_scale, const Tensor& cu, const Tensor& positions,
                  const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps,
                  const Tensor& chunks, const Tensor& seqs, const Tensor& scratch, const Tensor& vec, const Tensor& scal, const OptTensor& gate, const Tensor& o, const Tensor& status, bool raw) {
    const llm::LinearParams p = linear_params(in, offs, gates, bias_i, bias_f, cap, decay, angles, q_scale, k_scale, cu, positions, slots, state, true_vdim, norm_w, silu, out, eps, false, raw);
    bf16(in, "in"); bf16(out, "out");
    llm::LinearChunks c = {};
    auto table = [](const Tensor& t, const char* name) {
        TORCH_CHECK(t.dim() == 2 && t.size(1) == 4, name, " must be [n, 4]");
        return reinterpret_cast<const int4*>(ints(t, name));
    };
    c.chunks = table(chunks, "chunks"); c.seqs = table(seqs, "seqs");
    c.n_chunks = chunks.size(0); c.n_seqs = seqs.size(0); c.rows = in.size(0);
    TORCH_CHECK(slots.numel() == c.n_seqs, "one slot per sequence");
    const int64_t units = (int64_t)c.n_chunks * p.heads;
    auto scratch_ptr = [&](const Tensor& t, int64_t n, const char* name) {
        want(t, torch::kFloat32, name);
        TORCH_CHECK(t.numel() >= n, name, " too small");
        want_aligned(t, name);
        return t.data_ptr<float>();
    };
    c.state = scratch_ptr(scratch, units * p.vdim * p.dim, "scratch"); c.vec = scratch_ptr(vec, units * p.dim, "vec"); c.scal = scratch_ptr(scal, units * 4, "scal");
    if (p.gates) c.gate = reinterpret_cast<float4*>(scratch_ptr(gate.value(), units * llm::LINEAR_CHUNK * 4, "gate"));
    TORCH_CHECK(o.is_contiguous() && o.numel() >= (int64_t)c.rows * p.heads * p.vdim, "o too small");
    c.o = const_cast<__nv_bfloat16*>(bf16(o, "o"));
    want(status, torch::kInt32, "status");
    c.status = status.data_ptr<int>();
    check(llm::launch_linear_chunk(p, c, stream()), "linear_chunk");
}

// o, in and out have a row per token; the gate stands in columns [g_off, g_off + n) of in
void joint_gate(const Tensor& o, const Tensor& in, int64_t g_off, const Tensor& norm_w, int64_t true_n, const Tensor& out, double eps) {
    llm::JointGateParams p = {};
    const bool in_f32 = is_f32(in, "in"), f32 = is_f32(out, "out");
    want_like(o, in_f32, "o");
    const int64_t T = o.size(0), n = o.size(1);
    TORCH_CHECK(o.dim() == 2 && out.sizes() == o.sizes() && in.dim() == 2 && in.size(0) == T && o.stride(1) == 1 && in.stride(1) == 1 && out.stride(1) == 1, "joint_gate rows");
    TORCH_CHECK(g_off >= 0 && g_off + n <= in.size(1) && true_n >= 1 && true_n <= n, "joint_gate columns");
    want_aligned(o, "o"); want_aligned(in, "in"); want_aligned(out, "out"); want_aligned(norm_w, "norm_w");
    p.o = o.data_ptr(); p.o_row = o.stride(0); p.in = in.data_ptr(); p.in_row = in.stride(0); p.g_off = g_off;
    p.norm_w = floats(norm_w, n, "norm_w");
    p.out = out.data_ptr(); p.out_row = out.stride(0);
    p.n = n; p.true_n = true_n; p.eps = eps;
    check(llm::launch_joint_gate(p, T, in_f32, f32, stream()), "joint_gate");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("linear_rows", &linear_rows);
    m.def("linear_chunk", &linear_chunk);
    m.def("joint_gate", &joint_gate);
    m.def("linear_chunk_fits", &llm::linear_chunk_fits);
    m.attr("LINEAR_CHUNK") = llm::LINEAR_CHUNK;
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_mixers(reset) | llm::bounds_status_linear_tc(reset); });
}
