// Process-wide switch of programmatic dependent launch (see launch.cuh).
#include "launch.cuh"

namespace saber {
static int g_pdl = 1;
int pdl_enabled() { return g_pdl; }
static thread_local bool t_plain = false;
bool pdl_take_plain() {
  const bool p = t_plain;
  t_plain = false;
  return p;
}
}  // namespace saber

extern "C" void saber_set_pdl(int on) { saber::g_pdl = on; }
extern "C" void saber_pdl_plain_next() { saber::t_plain = true; }
extern "C" int saber_get_pdl() { return saber::g_pdl; }
