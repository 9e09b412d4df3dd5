// Python bindings of grouped-query attention with per-head keys and values: an extension of its own, so that a process that serves
// only such a model compiles and loads nothing else.
#include "binding_util.h"
#include "grouped.h"
#include "launch.h"
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

// rows in, offsets of a head's q, k, v -> checked parameters; gains and angles are checked by the caller
void head_prep(const Tensor& in, int64_t q_off, int64_t k_off, int64_t v_off, const Tensor& q_norm, const Tensor& k_norm, const Tensor& angles, const Tensor& positions,
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
    llm::HeadPrepParams p = {};
    p.in = in.data_ptr(); p.in_row = in.stride(0); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
    p.q_norm = floats(q_norm, D, "q_norm"); p.k_norm = floats(k_norm, D, "k_norm");
    p.angles = angle_ptr(angles, T); p.half = angles.size(1);
    TORCH_CHECK(2 * p.half <= true_dim, "more angles than a head has pairs");
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.q_out = q_out.data_ptr(); p.kv = kv.data_ptr();
    p.n_heads = H; p.n_kv_heads = G; p.dim = D; p.true_dim = true_dim; p.eps = eps;
    check(llm::launch_head_prep(p, T, in_f32, f32, stream()), "head_prep");
}

// taps [n, channels], ring [slots, n, channels]; cu: portions of several rows; first [tokens, kv heads, values]
void conv_prep(const Tensor& in, const Tensor& taps, const Tensor& ring, const Tensor& slots, const OptTensor& cu, const OptTensor& angles, const OptTensor& q_gain,
               const OptTensor& first, const OptTensor& share, const Tensor& positions, const Tensor& seq_ids, const Tensor& block_table, const Tensor& q_out, const Tensor& kv) {
    const bool in_f32 = is_f32(in, "in"), f32 = is_f32(kv, "kv");
    want_like(q_out, f32, "q_out");
    const int64_t T = in.size(0);
    if (T == 0) return;
    TORCH_CHECK(q_out.is_contiguous() && q_out.dim() == 3 && q_out.size(0) == T, "q_out must be [tokens, heads, dim]");
    const int64_t H = q_out.size(1), D = q_out.size(2), G = kv.size(2), cols = (H + 2 * G) * D, n = taps.size(0);
    want_cache(kv, D);
    TORCH_CHECK(in.dim() == 2 && in.stride(1) == 1 && in.size(1) >= cols, "in: too few columns");
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T, "rows");
    want_aligned(in, "in"); want_aligned(q_out, "q_out");
    llm::ConvPrepParams p = {};
    p.in = in.data_ptr(); p.in_row = in.stride(0); p.rows = T;
    p.taps = floats(taps, n * cols, "taps"); p.n_taps = n;
    want(ring, torch::kFloat32, "ring");
    TORCH_CHECK(ring.dim() == 3 && ring.size(1) == n && ring.size(2) == cols, "ring must be [slots, taps, channels]");
    p.ring = ring.data_ptr<float>(); p.n_slots = ring.size(0);
    p.n_seqs = slots.numel(); p.slots = ints(slots, "slots");
    TORCH_CHECK(block_table.size(0) >= p.n_seqs && (cu ? cu->numel() == p.n_seqs + 1 : p.n_seqs == T), "sequences");
    if (cu) p.cu = ints(*cu, "cu");
    if (angles) {
        p.angles = angle_ptr(*angles, T); p.half = angles->size(1);
        TORCH_CHECK(2 * p.half <= D, "more angles than a head has pairs");
    }
    if (q_gain) p.q_gain = floats(*q_gain, H, "q_gain");
    TORCH_CHECK(!share || first, "shared values missing");
    if (first) {
        want(*first, torch::kFloat32, "first");
        TORCH_CHECK(first->dim() == 3 && first->size(0) == T && first->size(1) == G, "first must be [tokens, kv heads, values]");
        p.first = first->data_ptr<float>(); p.first_dim = first->size(2);
        if (share) p.share = floats(*share, 1, "share");
    }
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.q_out = q_out.data_ptr(); p.kv = kv.data_ptr();
    p.n_heads = H; p.n_kv_heads = G; p.dim = D;
    check(llm::launch_conv_prep(p, in_f32, f32, stream()), "conv_prep");
    if (cu) check(llm::launch_conv_keep(p, in_f32, stream()), "conv_keep");
}

// gate [tokens, heads] (one number per head) or [tokens, heads * dim]; returns whether it is per head
bool gate_rows(const OptTensor& gate, int64_t T, int64_t heads, int64_t dim) {
    if (!gate) return false;
    TORCH_CHECK(gate->dim() == 2 && gate->size(0) == T && (gate->size(1) == heads || gate->size(1) == heads * dim) && gate->stride(1) == 1,
                "gate must be [tokens, heads] or [tokens, heads * dim]");
    return gate->size(1) == heads;
}

void attn_plain(const Tensor& q, const Tensor& kv, const Tensor& out, const Tensor& positions, const Tensor& seq_ids, const Tensor& block_table,
                  int64_t window, double scale, const OptTensor& sink, const OptTensor& gate, int64_t chunk, double softcap) {
    const bool f32 = is_f32(kv, "kv");
    want_like(q, f32, "q"); want_like(out, f32, "out");
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [tokens, heads, dim]");
    const int64_t T = q.size(0), H = q.size(1), D = q.size(2);
    want_cache(kv, D);
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T, "rows");
    llm::AttnPlainParams p = {};
    p.gate_heads = gate_rows(gate, T, H, D); p.chunk = chunk; p.softcap = softcap;
    p.q = q.data_ptr(); p.kv = kv.data_ptr(); p.out = out.data_ptr();
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.n_heads = H; p.n_kv_heads = kv.size(2); p.dim = D; p.window = window; p.scale = scale;
    p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    bool gate_f32 = true;
    if (gate) { gate_f32 = is_f32(*gate, "gate"); p.gate = gate->data_ptr(); p.gate_row = gate->stride(0); }
    check(llm::launch_attn_plain(p, T, gate_f32, f32, stream()), "attn_plain");
}

// one row per sequence: q [batch, heads, dim]
void attn_decode(const Tensor& q, const Tensor& kv, const Tensor& out, const Tensor& block_table, const Tensor& seq_lens, const Tensor& part_o, const Tensor& part_ml,
                 const Tensor& tickets, double scale, int64_t n_splits, int64_t window, const OptTensor& sink, const OptTensor& gate,
                 int64_t chunk, double softcap) {
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [batch, heads, dim]");
    const int64_t B = q.size(0), H = q.size(1), D = q.size(2), G = kv.size(2);
    want_cache(kv, D);
    TORCH_CHECK(block_table.size(0) >= B && seq_lens.numel() == B && n_splits >= 1, "batch");
    llm::AttnDecodeParams p = {};
    p.gate_heads = gate_rows(gate, B, H, D); p.chunk = chunk; p.softcap = softcap;
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
                  int64_t max_q_len, int64_t window, const OptTensor& sink, const OptTensor& gate, const OptTensor& status, int64_t chunk, double softcap) {
    TORCH_CHECK(q.is_contiguous() && out.is_contiguous() && q.dim() == 3 && out.numel() == q.numel(), "q / out must be [tokens, heads, dim]");
    const int64_t T = q.size(0), H = q.size(1), D = q.size(2), n = ctx_lens.numel();
    want_cache(kv, D);
    TORCH_CHECK(block_table.size(0) >= n && cu_q.numel() == n + 1, "sequences");
    const bool gate_heads = gate_rows(gate, T, H, D);
    if (n == 0 || max_q_len == 0) return;
    llm::AttnPrefillParams p = {};
    p.q = bf16(q, "q"); p.kv = bf16(kv, "kv"); p.out = const_cast<__nv_bfloat16*>(bf16(out, "out"));
    p.block_table = ints(block_table, "block_table"); p.cu_q = ints(cu_q, "cu_q"); p.ctx_lens = ints(ctx_lens, "ctx_lens");
    p.n_heads = H; p.n_kv_heads = kv.size(2); p.head_dim = D; p.max_pages = block_table.size(1); p.scale = scale; p.n_pages = kv.size(0);
    p.window = window; p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    p.gate_heads = gate_heads; p.chunk = chunk; p.softcap = softcap;
    if (gate) {
        p.gate = bf16(*gate, "gate"); p.gate_row = gate->stride(0);
        if (!gate_heads) {
            want_aligned(*gate, "gate");
            TORCH_CHECK(p.gate_row % 8 == 0, "gate rows must be 16-byte aligned");
        }
    }
    if (status) {
        want(*status, torch::kInt32, "status");
        check(llm::launch_attn_prefill_tc(p, n, max_q_len, status->data_ptr<int>(), stream()), "attn_prefill_tc");
    } else {
        check(llm::launch_attn_prefill(p, n, max_q_len, stream()), "attn_prefill");
    }
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("attn_prep", &attn_prep);
    m.def("head_prep", &head_prep);
    m.def("conv_prep", &conv_prep);
    m.def("attn_plain", &attn_plain);
    m.def("attn_decode", &attn_decode);
    m.def("attn_prefill", &attn_prefill);
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_grouped(reset); });
}
