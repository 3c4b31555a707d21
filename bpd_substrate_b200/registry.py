"""Model families by name: which class serves a model folder (config.json names the architecture) or file."""
import json
import os


def _hybrid(spec_class, path, dtype, capacity):
    from . import capi
    from .hybrid import DeviceHybrid
    return DeviceHybrid.from_folder(path, spec_class, dtype=dtype, capacity=capacity, lib=capi.load(part="hybrid"))


def _gurusun(path, dtype, capacity):
    from .hybrid import HybridSpec
    return _hybrid(HybridSpec, path, dtype, capacity)


def _vuzelix(path, dtype, capacity):
    from .vuzelix import VuzelixSpec
    return _hybrid(VuzelixSpec, path, dtype, capacity)


def _llama(path, dtype, capacity):
    from .llama import DeviceLlama, GgufLlama
    if dtype != "bfloat16":
        raise ValueError("the Q8_0 Llama has one arithmetic: int8 products, fp32 activations")
    return DeviceLlama(GgufLlama(path, max_seq_len=capacity))


# architecture -> loader(path, dtype, capacity)
FAMILIES = {"Gurusun": _gurusun, "Vuzelix": _vuzelix, "llama": _llama}


def architecture_of(path):
    """The architecture of a model folder, or of a GGUF file (which only holds Llamas here)."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return json.load(f).get("architecture")
    if path.endswith(".gguf"):
        return "llama"
    raise ValueError(f"{path}: neither a model folder nor a .gguf file")


def load_model(path, dtype="bfloat16", capacity=4096):
    """The model at `path` on the device, ready for an Engine; sequences of up to `capacity` tokens."""
    arch = architecture_of(path)
    if arch not in FAMILIES:
        raise ValueError(f"{path}: architecture {arch!r}; known: {', '.join(sorted(FAMILIES))}")
    return FAMILIES[arch](path, dtype, capacity)
