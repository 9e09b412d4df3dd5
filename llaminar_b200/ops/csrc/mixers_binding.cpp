// Python bindings of the mixers with grouped-query attention or a recurrent state: an extension of its own, so that a process that
// serves only such a model compiles and loads nothing else.
#include "binding_util.h"
#include "launch.h"
#include "mixers.h"
#include "ops.h"

namespace {
using namespace llm_binding;

const __nv_bfloat16* bf16(const Tensor& t, const char* name) {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kBFloat16, name, " must be bfloat16");
    return reinterpret_cast<const __nv_bfloat16*>(t.data_ptr());
}
void want_aligned(const Tensor& t, const char* name) { TORCH_CHECK(reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, name, " must be 16-byte aligned"); }

// kv [pages, 2, kv heads, 64, dim]
void want_cache(const Tensor& kv, int64_t dim) {
    TORCH_CHECK(kv.is_cuda() && kv.is_contiguous() && kv.dim() == 5 && kv.size(1) == 2 && kv.size(3) == 64 && kv.size(4) == dim, "kv must be [pages, 2, heads, 64, ", dim, "]");
}

void attn_prep(const Tensor& in, int64_t q_off, int64_t k_off, int64_t v_off, const Tensor& q_norm, const Tensor& k_norm, const Tensor& positions,
               const Tensor& seq_ids, const Tensor& block_table, const Tensor& q_out, const Tensor& kv, int64_t true_dim, double eps) {
    const bool in_f32 = is_f32(in, "in"), f32 = is_f32(kv, "kv");
    want_like(q_out, f32, "q_out");
    const int64_t T = in.size(0);
    if (T == 0) return;
    TORCH_CHECK(q_out.is_contiguous() && q_out.dim() == 3 && q_out.size(0) == T, "q_out must be [tokens, heads, dim]");
    const int64_t H = q_out.size(1), D = q_out.size(2), G = kv.size(2);
    want_cache(kv, D);
    TORCH_CHECK(in.stride(1) == 1 && q_off + H * D <= in.size(1) && k_off + G * D <= in.size(1) && v_off + G * D <= in.size(1), "in: too few columns");
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T && true_dim <= D, "rows");
    want_aligned(in, "in"); want_aligned(q_out, "q_out");
    llm::AttnPrepParams p = {};
    p.in = in.data_ptr(); p.in_row = in.stride(0); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
    p.q_norm = floats(q_norm, H * D, "q_norm"); p.k_norm = floats(k_norm, G * D, "k_norm");
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.q_out = q_out.data_ptr(); p.kv = kv.data_ptr();
    p.n_heads = H; p.n_kv_heads = G; p.dim = D; p.true_dim = true_dim; p.eps = eps;
    check(llm::launch_attn_prep(p, T, in_f32, f32, stream()), "attn_prep");
}

void gate_rows(const OptTensor& gate, int64_t T, int64_t cols) {
    if (gate) TORCH_CHECK(gate->dim() == 2 && gate->size(0) == T && gate->size(1) == cols && gate->stride(1) == 1, "gate must be [tokens, ", cols, "]");
}

void window_plain(const Tensor& q, const Tensor& kv, const Tensor& out, const Tensor& positions, const Tensor& seq_ids, const Tensor& block_table,
                  int64_t window, double scale, const OptTensor& sink, const OptTensor& gate) {
    const bool f32 = is_f32(kv, "kv");
    want_like(q, f32, "q"); want_like(out, f32, "out");
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [tokens, heads, dim]");
    const int64_t T = q.size(0), H = q.size(1), D = q.size(2);
    want_cache(kv, D);
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T, "rows");
    gate_rows(gate, T, H * D);
    llm::WindowPlainParams p = {};
    p.q = q.data_ptr(); p.kv = kv.data_ptr(); p.out = out.data_ptr();
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.n_heads = H; p.n_kv_heads = kv.size(2); p.dim = D; p.window = window; p.scale = scale;
    p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    bool gate_f32 = true;
    if (gate) { gate_f32 = is_f32(*gate, "gate"); p.gate = gate->data_ptr(); p.gate_row = gate->stride(0); }
    check(llm::launch_window_plain(p, T, gate_f32, f32, stream()), "window_plain");
}

// one row per sequence: q [batch, heads, dim]
void attn_decode(const Tensor& q, const Tensor& kv, const Tensor& out, const Tensor& block_table, const Tensor& seq_lens, const Tensor& part_o, const Tensor& part_ml,
                 const Tensor& tickets, double scale, int64_t n_splits, int64_t window, const OptTensor& sink, const OptTensor& gate) {
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [batch, heads, dim]");
    const int64_t B = q.size(0), H = q.size(1), D = q.size(2), G = kv.size(2);
    want_cache(kv, D);
    TORCH_CHECK(block_table.size(0) >= B && seq_lens.numel() == B && n_splits >= 1, "batch");
    gate_rows(gate, B, H * D);
    llm::AttnDecodeParams p = {};
    p.q = bf16(q, "q"); p.kv = bf16(kv, "kv"); p.out = const_cast<__nv_bfloat16*>(bf16(out, "out"));
    p.block_table = ints(block_table, "block_table"); p.seq_lens = ints(seq_lens, "seq_lens");
    if (n_splits > 1) {
        want(part_o, torch::kFloat32, "part_o"); want(part_ml, torch::kFloat32, "part_ml"); want(tickets, torch::kInt32, "tickets");
        TORCH_CHECK(part_o.numel() >= B * G * n_splits * 16 * D && part_ml.numel() >= B * G * n_splits * 32 && tickets.numel() >= B * G, "split scratch too small");
        p.part_o = part_o.data_ptr<float>(); p.part_ml = part_ml.data_ptr<float>(); p.tickets = reinterpret_cast<unsigned*>(tickets.data_ptr<int>());
    }
    p.n_heads = H; p.n_kv_heads = G; p.head_dim = D; p.max_pages = block_table.size(1); p.rows_per_seq = 1; p.scale = scale; p.n_pages = kv.size(0);
    p.window = window; p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    if (gate) { TORCH_CHECK(is_f32(*gate, "gate"), "gate must be float32"); p.gate = gate->data_ptr<float>(); p.gate_row = gate->stride(0); }
    check(llm::launch_attn_decode(p, B, n_splits, stream()), "attn_decode");
}

// q [tokens, heads, dim]; status: the tcgen05 form
void attn_prefill(const Tensor& q, const Tensor& kv, const Tensor& out, const Tensor& block_table, const Tensor& cu_q, const Tensor& ctx_lens, double scale,
                  int64_t max_q_len, int64_t window, const OptTensor& sink, const OptTensor& gate, const OptTensor& status) {
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [tokens, heads, dim]");
    const int64_t T = q.size(0), H = q.size(1), D = q.size(2), n = ctx_lens.numel();
    want_cache(kv, D);
    TORCH_CHECK(block_table.size(0) >= n && cu_q.numel() == n + 1, "sequences");
    gate_rows(gate, T, H * D);
    if (n == 0 || max_q_len == 0) return;
    llm::AttnPrefillParams p = {};
    p.q = bf16(q, "q"); p.kv = bf16(kv, "kv"); p.out = const_cast<__nv_bfloat16*>(bf16(out, "out"));
    p.block_table = ints(block_table, "block_table"); p.cu_q = ints(cu_q, "cu_q"); p.ctx_lens = ints(ctx_lens, "ctx_lens");
    p.n_heads = H; p.n_kv_heads = kv.size(2); p.head_dim = D; p.max_pages = block_table.size(1); p.scale = scale; p.n_pages = kv.size(0);
    p.window = window; p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    if (gate) {
        p.gate = bf16(*gate, "gate"); p.gate_row = gate->stride(0);
        want_aligned(*gate, "gate");
        TORCH_CHECK(p.gate_row % 8 == 0, "gate rows must be 16-byte aligned");
    }
    if (status) {
        want(*status, torch::kInt32, "status");
        check(llm::launch_attn_prefill_tc(p, n, max_q_len, status->data_ptr<int>(), stream()), "attn_prefill_tc");
    } else {
        check(llm::launch_attn_prefill(p, n, max_q_len, stream()), "attn_prefill");
    }
}

// What the linear-attention entry points share.  offs: first columns of q, k, v, g; state: S (, n, m); gates with bias_i, bias_f, cap: mLSTM; decay: retention
llm::LinearParams linear_params(const Tensor& in, const std::vector<int64_t>& offs, const OptTensor& gates, const OptTensor& bias_i, const OptTensor& bias_f, double cap,
                                const OptTensor& decay, const OptTensor& angles, double q_scale, double k_scale, const OptTensor& cu, const Tensor& positions,
                                const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps) {
    llm::LinearParams p = {};
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
                 const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps) {
    const llm::LinearParams p = linear_params(in, offs, gates, bias_i, bias_f, cap, decay, angles, q_scale, k_scale, cu, positions, slots, state, true_vdim, norm_w, silu, out, eps);
    check(llm::launch_linear_rows(p, slots.numel(), is_f32(in, "in"), is_f32(out, "out"), stream()), "linear_rows");
}

// chunks, seqs: int32 [n, 4], see LinearChunks.  cu is the host's view of the sequences and stays unused on the device.
void linear_chunk(const Tensor& in, const std::vector<int64_t>& offs, const OptTensor& gates, const OptTensor& bias_i, const OptTensor& bias_f, double cap,
                  const OptTensor& decay, const OptTensor& angles, double q_scale, double k_scale, const Tensor& cu, const Tensor& positions,
                  const Tensor& slots, const std::vector<Tensor>& state, int64_t true_vdim, const OptTensor& norm_w, bool silu, const Tensor& out, double eps,
                  const Tensor& chunks, const Tensor& seqs, const Tensor& scratch, const Tensor& vec, const Tensor& scal, const OptTensor& gate, const Tensor& o, const Tensor& status) {
    const llm::LinearParams p = linear_params(in, offs, gates, bias_i, bias_f, cap, decay, angles, q_scale, k_scale, cu, positions, slots, state, true_vdim, norm_w, silu, out, eps);
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

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("attn_prep", &attn_prep);
    m.def("window_plain", &window_plain);
    m.def("attn_decode", &attn_decode);
    m.def("attn_prefill", &attn_prefill);
    m.def("linear_rows", &linear_rows);
    m.def("linear_chunk", &linear_chunk);
    m.def("linear_chunk_fits", &llm::linear_chunk_fits);
    m.attr("LINEAR_CHUNK") = llm::LINEAR_CHUNK;
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_mixers(reset) | llm::bounds_status_linear_tc(reset); });
}
