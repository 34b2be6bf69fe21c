"""nfai_b200: the forward paths of NFAI on B200 (sm_100a) behind a C ABI: Llama-3 models from GGUF files and models whose
layers a config.json lists.

`nfai_b200.api` mirrors the reference's model interface (ModelOptions, LlamaModelFactory, LlamaModel) over
libnfai_cuda.so; `nfai_b200.synth` makes the seeded synthetic models; `nfai_b200.gguf_io` reads and writes GGUF;
`nfai_b200.tokenizer` mirrors the reference's Tokenizer over the native byte-pair encoder.
"""
from .api import (CausalModel, CudaContext, LlamaModel, LlamaModelFactory, ModelOptions, NfaiError,  # noqa: F401
                  PlannedModel, config_tensors, create_synthetic_model, synthetic_tensors)
from .gguf_io import ComputeCollection, Parser  # noqa: F401
from .registry import try_create  # noqa: F401
from .tokenizer import Tokenizer  # noqa: F401

__all__ = ["CausalModel", "CudaContext", "PlannedModel", "config_tensors", "try_create", "LlamaModel", "LlamaModelFactory", "ModelOptions", "NfaiError", "ComputeCollection",
           "Parser", "Tokenizer", "create_synthetic_model", "synthetic_tensors"]
