#include "gated.h"
namespace nfb {
int64_t gated_chunked_workspace_bytes(int, int, int, int, int) { return 0; }
bool gated_chunked_supported(int, int) { return false; }
const char* gated_chunked(const GatedArgs&, void*, int64_t) { return "gated_chunked: not built"; }
}  // namespace nfb
