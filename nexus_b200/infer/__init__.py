"""Paged-KV inference engine: block allocator with copy-on-write, state slots for recurrent layers, packed prefill/decode
steps, decode CUDA graphs, single-kernel sampler, speculative decoding and weight / KV quantisation."""
from .engine import (Chunk, Engine, EngineConfig, GenerateStats, Gpt2Weights, QuantOptions, SamplingParams,  # noqa: F401
                     SpecStats, StepStats, generate, load_gpt2, speculative_generate)
from .hybrid import HybridEngine  # noqa: F401
from .registry import ModelFamily, create_engine, families, load_model, open_engine, register_family  # noqa: F401
from .sampling import sample_reference  # noqa: F401
