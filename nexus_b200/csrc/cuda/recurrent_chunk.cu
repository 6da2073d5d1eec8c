#include "nx_api_mixers.h"
extern "C" int nx_ssd_chunk(const NxSsdArgs*, nx_stream_t) { return -1; }
extern "C" int nx_delta_chunk(const NxDeltaArgs*, nx_stream_t) { return -1; }
