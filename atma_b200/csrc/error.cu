// The calling thread's last error message, shared by every entry point of a library.
#include "common.cuh"

namespace atma {

char* err_buf() {
  static thread_local char buf[512] = {0};
  return buf;
}

int fail(int code, const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(err_buf(), 512, fmt, ap);
  va_end(ap);
  return code;
}

}  // namespace atma

extern "C" const char* atma_last_error(void) { return atma::err_buf(); }
