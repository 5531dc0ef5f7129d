// The scheduler with the reference's own sampler (src/sampler.h), for GGUF models.
#pragma once

#include "batch_scheduler.h"
#include "sampler.h"

using BatchScheduler = BasicBatchScheduler<Sampler, SamplerParams>;
