// Python bindings of the kernels of latent-attention models: an extension of its own, so that a process that serves only such
// a model compiles and loads nothing else.
#include "binding_util.h"
#include "latent.h"
#include "launch.h"

namespace {
using namespace llm_binding;

void latent_prep(const Tensor& down, const Tensor& q_norm, const Tensor& kv_norm, const Tensor& angles, const Tensor& positions, const Tensor& seq_ids,
                 const Tensor& block_table, const Tensor& cq, const Tensor& kv, int64_t rot_dim, int64_t rot_off, double eps) {
    const bool f32 = is_f32(down, "down");
    want_like(cq, f32, "cq"); want_like(kv, f32, "kv");
    const int64_t T = down.size(0), q_rank = q_norm.numel(), kv_rank = kv_norm.numel();
    if (T == 0) return;
    TORCH_CHECK(down.stride(1) == 1 && down.size(1) >= q_rank + kv_rank + rot_dim, "down: too few columns");
    TORCH_CHECK(cq.is_contiguous() && cq.size(0) == T && cq.size(1) >= q_rank, "cq shape");
    TORCH_CHECK(kv.is_contiguous() && kv.dim() == 3 && kv.size(1) == 64, "kv must be [pages, 64, width]");
    TORCH_CHECK(rot_off >= kv_rank && rot_off + rot_dim <= kv.size(2), "cache row too narrow");
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T, "positions / seq_ids");
    llm::LatentPrepParams p = {};
    p.down = down.data_ptr(); p.down_stride = down.stride(0);
    p.q_norm = floats(q_norm, q_rank, "q_norm"); p.kv_norm = floats(kv_norm, kv_rank, "kv_norm");
    p.angles = angle_ptr(angles, T); p.half = angles.size(1);
    TORCH_CHECK(2 * p.half <= rot_dim, "more angles than the rotated part has pairs");
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.cq = cq.data_ptr(); p.cq_stride = cq.size(1); p.kv = kv.data_ptr();
    p.q_rank = q_rank; p.kv_rank = kv_rank; p.rot_dim = rot_dim; p.rot_off = rot_off; p.width = kv.size(2); p.eps = eps;
    check(llm::launch_latent_prep(p, T, f32, stream()), "latent_prep");
}

// q_lat [heads, rows, rot_off]; q [tokens, heads, head size] (contiguous); out [heads, rows, rot_off]
void latent_rows(const Tensor& q_lat, const Tensor& q, int64_t q_rot_off, const Tensor& angles, const OptTensor& rows, const Tensor& positions,
                 const Tensor& seq_ids, const Tensor& block_table, const Tensor& kv, int64_t rot_dim, int64_t window, double scale,
                 const OptTensor& sink, const Tensor& out, const OptTensor& part_o, const OptTensor& part_ml, int64_t n_splits, int64_t group,
                 const OptTensor& status) {
    const bool f32 = is_f32(kv, "kv");
    want_like(q_lat, f32, "q_lat"); want_like(q, f32, "q"); want_like(out, f32, "out");
    const int64_t H = q_lat.size(0), n = q_lat.size(1), R = q_lat.size(2);
    if (n == 0) return;
    TORCH_CHECK(q_lat.stride(2) == 1 && out.stride(2) == 1 && out.sizes() == q_lat.sizes(), "q_lat / out must be [heads, rows, latent]");
    TORCH_CHECK(q.is_contiguous() && q.dim() == 3 && q.size(1) == H && q.size(2) >= q_rot_off + rot_dim, "q must be [tokens, heads, size]");
    TORCH_CHECK(kv.is_contiguous() && kv.dim() == 3 && kv.size(1) == 64 && R + rot_dim <= kv.size(2), "kv must be [pages, 64, width]");
    const int64_t T = q.size(0);
    TORCH_CHECK(positions.numel() == T && seq_ids.numel() == T && (rows ? rows->numel() == n : T == n), "row description");
    llm::LatentRowsParams p = {};
    p.q_lat = q_lat.data_ptr(); p.ql_row = q_lat.stride(1); p.ql_head = q_lat.stride(0);
    p.q = q.data_ptr(); p.q_row = q.stride(0); p.q_head = q.stride(1); p.q_rot_off = q_rot_off;
    p.angles = angle_ptr(angles, T); p.half = angles.size(1);
    TORCH_CHECK(2 * p.half <= rot_dim, "more angles than the rotated part has pairs");
    p.rows = rows ? ints(*rows, "rows") : nullptr;
    p.positions = ints(positions, "positions"); p.seq_ids = ints(seq_ids, "seq_ids"); p.block_table = ints(block_table, "block_table");
    p.n_seqs = block_table.size(0); p.max_pages = block_table.size(1); p.n_pages = kv.size(0);
    p.kv = kv.data_ptr(); p.width = kv.size(2); p.rot_off = R; p.rot_dim = rot_dim;
    p.n_heads = H; p.window = window; p.scale = scale;
    p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    p.out = out.data_ptr(); p.out_row = out.stride(1); p.out_head = out.stride(0);
    // group: heads per CTA of the tcgen05 form, 16 of the mma.sync form, 0 the plain kernel
    const bool tc = group == llm::latent_rows_tc_heads(p.width, p.rot_off, p.rot_dim, H) && group > 0 && status;
    TORCH_CHECK(group == 0 || (!f32 && (tc || (group == 16 && llm::latent_rows_has_kernel(p.width, p.rot_off)))), "no kernel for this group of heads");
    if (group) {
        TORCH_CHECK(p.out_row % 4 == 0 && p.out_head % 4 == 0 && p.ql_row % 8 == 0 && p.ql_head % 8 == 0, "latent strides");
        TORCH_CHECK(n_splits >= 1 && n_splits <= 64, "n_splits");
        if (n_splits > 1) {
            const int64_t parts = n * ((H + group - 1) / group) * n_splits * group;
            want(part_o.value(), torch::kFloat32, "part_o"); want(part_ml.value(), torch::kFloat32, "part_ml");
            TORCH_CHECK(part_o->numel() >= parts * R && part_ml->numel() >= parts * 2, "split scratch too small");
            p.part_o = part_o->data_ptr<float>(); p.part_ml = part_ml->data_ptr<float>();
        }
    }
    if (tc) {
        TORCH_CHECK(q_rot_off % 8 == 0 && q.size(2) % 8 == 0, "the rotated query part must start on a 16-byte boundary");
        want(*status, torch::kInt32, "status");
        check(llm::launch_latent_rows_tc(p, n, n_splits, status->data_ptr<int>(), stream()), "latent_rows_tc");
        if (n_splits > 1) check(llm::launch_latent_merge(p, n, n_splits, group, stream()), "latent_merge");
        return;
    }
    check(llm::launch_latent_rows(p, n, group ? n_splits : 1, f32, group == 0, stream()), "latent_rows");
}

// seqs: int32 [n, 8], see LatentSeq; the limits are the host's view of the same numbers
void latent_gather(const Tensor& kv, const Tensor& seqs, int64_t max_k_len, const Tensor& block_table, const Tensor& out) {
    const bool f32 = is_f32(kv, "kv");
    want_like(out, f32, "out");
    TORCH_CHECK(kv.is_contiguous() && out.is_contiguous() && kv.dim() == 3 && out.size(1) == kv.size(2), "gather shapes");
    TORCH_CHECK((kv.size(2) * kv.element_size()) % 16 == 0, "cache rows must be whole 16-byte units");
    TORCH_CHECK(seqs.dim() == 2 && seqs.size(1) == 8, "seqs must be [n, 8]");
    if (seqs.size(0) == 0 || max_k_len == 0) return;
    check(llm::launch_latent_gather(kv.data_ptr(), reinterpret_cast<const llm::LatentSeq*>(ints(seqs, "seqs")), seqs.size(0), max_k_len,
                                    ints(block_table, "block_table"), block_table.size(1), kv.size(0), kv.size(2), out.data_ptr(), f32, stream()),
          "latent_gather");
}

// k [keys, heads * dim]; v [keys, heads * vdim], or with status (the tcgen05 form) [heads * vdim, keys]
void latent_chunk(const Tensor& q, const Tensor& angles, const Tensor& k, const Tensor& v, const Tensor& lat, int64_t rot_off, const Tensor& seqs,
                  int64_t max_q_len, const Tensor& out, int64_t dim, int64_t rot, int64_t vdim, int64_t window, double scale, const OptTensor& sink,
                  const OptTensor& status, const OptTensor& gate) {
    for (auto& t : {q, k, v, lat, out}) want(t, torch::kBFloat16, "latent_chunk operand");
    const int64_t T = q.size(0), H = q.size(1), n = lat.size(0);
    TORCH_CHECK(q.dim() == 3 && q.size(2) == dim + rot, "q must be [tokens, heads, dim + rot]");
    TORCH_CHECK(k.size(0) == n && k.size(1) == H * dim && rot_off + rot <= lat.size(1), "key buffers");
    TORCH_CHECK(status ? v.size(0) == H * vdim && v.size(1) == n : v.size(0) == n && v.size(1) == H * vdim, "value buffer");
    TORCH_CHECK(out.size(0) == T && out.size(1) == H * vdim, "out must be [tokens, heads * vdim]");
    TORCH_CHECK(seqs.dim() == 2 && seqs.size(1) == 8, "seqs must be [n, 8]");
    TORCH_CHECK(dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && rot_off % 8 == 0 && lat.size(1) % 8 == 0, "sizes must be multiples of 8");
    if (seqs.size(0) == 0) return;
    llm::LatentChunkParams p = {};
    auto b = [](const Tensor& t) { return reinterpret_cast<const __nv_bfloat16*>(t.data_ptr()); };
    p.q = b(q); p.q_row = q.stride(0); p.q_head = q.stride(1);
    p.angles = angle_ptr(angles, T); p.half = angles.size(1);
    TORCH_CHECK(2 * p.half <= rot, "more angles than the rotated part has pairs");
    p.k = b(k); p.v = b(v);
    p.lat = b(lat); p.lat_row = lat.size(1); p.rot_off = rot_off;
    p.seqs = reinterpret_cast<const llm::LatentSeq*>(ints(seqs, "seqs"));
    p.out = reinterpret_cast<__nv_bfloat16*>(out.data_ptr()); p.out_row = out.size(1);
    p.dim = dim; p.rot = rot; p.vdim = vdim; p.n_heads = H; p.window = window; p.scale = scale;
    p.sink = sink ? floats(*sink, H, "sink") : nullptr;
    if (gate) {
        want_like(*gate, false, "gate");
        TORCH_CHECK(gate->dim() == 2 && gate->size(0) == T && gate->size(1) == H * vdim && gate->stride(1) == 1 && gate->stride(0) % 8 == 0 &&
                    reinterpret_cast<uintptr_t>(gate->data_ptr()) % 16 == 0, "gate must be [tokens, heads * vdim] in whole 16-byte units");
        p.gate = b(*gate); p.gate_row = gate->stride(0);
    }
    if (status) {
        want(*status, torch::kInt32, "status");
        check(llm::launch_latent_chunk_tc(p, n, seqs.size(0), max_q_len, status->data_ptr<int>(), stream()), "latent_chunk_tc");
    } else {
        check(llm::launch_latent_chunk(p, seqs.size(0), max_q_len, stream()), "latent_chunk");
    }
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("latent_prep", &latent_prep);
    m.def("latent_rows", &latent_rows);
    m.def("latent_rows_has_kernel", &llm::latent_rows_has_kernel);
    m.def("latent_rows_tc_heads", &llm::latent_rows_tc_heads);
    m.def("latent_chunk_tc_fits", &llm::latent_chunk_tc_fits);
    m.def("latent_gather", &latent_gather);
    m.def("latent_chunk", &latent_chunk);
    m.def("latent_chunk_has_kernel", &llm::latent_chunk_has_kernel);
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_latent(reset) | llm::bounds_status_latent_tc(reset); });
}
