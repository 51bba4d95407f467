// Error reporting of the `memory` library: recurrences with one state matrix per head (matrix memory with exponential gates,
// the gated delta rule), and the residual row after a sublayer whose result is normed, with the average over the depth.
#include "common.cuh"

#include <stdarg.h>

static thread_local char g_err[512];
void hb_set_error(const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(g_err, sizeof g_err, fmt, ap);
  va_end(ap);
}
HB_EXPORT const char* hb_last_error() { return g_err; }
HB_EXPORT int hb_memory_abi_version() { return 1; }
int g_hb_pdl = 1;
HB_EXPORT void hb_set_pdl(int on) { g_hb_pdl = on; }
