// pdl.cuh -- the two halves of a programmatic dependent launch (launch_dependent in common.h).  A kernel launched that way may start
// while its predecessor in the stream still runs.  pdl_release() lets the successor's CTAs be scheduled as soon as every CTA of this
// grid has called it (or exited); pdl_acquire() returns once the predecessor grid has completed and its writes are visible.
// Everything a kernel does before pdl_acquire() may only touch memory no earlier kernel of the stream writes (weights); both are
// no-ops in an ordinary launch.
#pragma once

namespace spt {

__device__ __forceinline__ void pdl_release() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_acquire() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

}  // namespace spt
