// Gated delta rule of large prompt portions: every size still runs token by token.
#include "delta.cuh"
namespace rewb {
bool delta_chunk_ok(const DeltaDims&) { return false; }
int delta_chunks(int n) { return (n + 31) / 32; }
int2 delta_chunk_rows(const GlaPortion& p, int i) { return make_int2(p.row0 + i * 32, 0); }
size_t delta_chunk_bytes(const DeltaDims&) { return 0; }
int delta_chunk_launch(Ctx*, const DeltaArgs&) { return fail("none"); }
}  // namespace rewb
