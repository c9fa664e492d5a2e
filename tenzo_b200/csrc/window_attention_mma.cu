#include "hybrid_common.cuh"
namespace tz {
bool window_flash_applicable(const WindowAttnArgs&) { return false; }
int launch_window_flash(const WindowAttnArgs&, int, cudaStream_t) { return -1; }
}
