// Tensor-core form: sizes it takes are none yet; callers use the SIMT form.
#include "sx_api.h"
extern "C" int sx_win_decode_ok(int H, int G, int d, int dv) { return 0; }
extern "C" int sx_win_decode(const SxWinAttnArgs* a, cudaStream_t st) { return -1; }
