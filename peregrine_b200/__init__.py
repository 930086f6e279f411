"""peregrine_b200: the quantized-inference path of etam103/peregrine on NVIDIA B200 (sm_100a).

    quant     mirror of peregrine::quant  (src/quant.rs)
    gguf      mirror of the block codecs of peregrine::gguf  (src/gguf.rs:284-401)
    gguf_file the GGUF container, mirror of GgufFile  (src/gguf.rs:140-283, 403-567)
    llama     the Llama decode step on the int8 path  (src/models/llama)
    llama_gguf  Llama::from_gguf for that step: config keys, tensor names, transposition, Q|K|V and gate|up fusion
    serial    the quantised serial formats  (src/serial.rs:124-222, 315-443)
    huffman   Huffman-coded int8 weights, mirror of HuffmanTable / HuffmanTensor  (src/huffman.rs:19-476)
    sonalorn  a decoder of gated delta rule and attention layers in bf16 or f32, put together from
    layers    the layer mechanisms (products, delta rule, attention, feed-forwards, experts) and served through
    slot_model, state, engine   slots of caches and states, recorded decode steps, scheduling, greedy generation
    registry  which class serves a GGUF file or a folder with config.json;  trace  replays steps of given token ids
    safetensors_file   the container of such a folder's weights
    runtime   GpuContext / GpuBuffer / init_gpu / with_gpu  (the reference's `metal` seam)
    build     compiles libperegrine_b200.so and libperegrine_b200_lm.so with nvcc

`python -m peregrine_b200 --help` is the command line.
Everything computes in hand-written CUDA behind the C ABI of include/peregrine_b200.h and
include/peregrine_b200_lm.h.
"""
from . import _lib
from ._lib import InvalidArgument, PeregrineError
from .runtime import GpuBuffer, GpuContext, current_gpu, init_gpu, with_gpu
from . import quant, gguf, gguf_file, serial, huffman
from .gguf_file import GgufFile

__all__ = ["quant", "gguf", "gguf_file", "GgufFile", "serial", "huffman", "GpuContext", "GpuBuffer", "init_gpu", "with_gpu", "current_gpu", "PeregrineError", "InvalidArgument"]
