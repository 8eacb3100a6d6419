"""The models the library can load from disk, by what lies there: a folder whose
config.json names an architecture, or a llama2.c checkpoint file."""
import json
import os

from . import build, gofilorn, vamalix
from .llama import Decoder

# architecture in config.json -> (the dtypes it runs in, load(path, dtype,
# max_seq, batch) -> Decoder, what builds a library that can serve it)
ARCHITECTURES = {
    gofilorn.ARCHITECTURE: (gofilorn.DTYPES, gofilorn.load, build.for_parallel_decoders),
    vamalix.ARCHITECTURE: (vamalix.DTYPES, vamalix.load, build.for_stream_decoders),
}


class UnsupportedDtype(ValueError):
    """The model exists but not in the number format asked for."""


def architecture_of(path):
    with open(os.path.join(path, "config.json")) as f:
        name = json.load(f).get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError("%s: no model class for the architecture %r (there are: %s)"
                         % (path, name, ", ".join(sorted(ARCHITECTURES))))
    return name


def load(path, dtype="bfloat16", max_seq=4096, batch=1):
    """A Decoder for `path`."""
    if os.path.isdir(path):
        dtypes, loader, _ = ARCHITECTURES[architecture_of(path)]
        if dtype not in dtypes:
            raise UnsupportedDtype("%s runs in %s" % (path, " or ".join(dtypes)))
        return loader(path, dtype, max_seq, batch)
    if dtype != "float32":
        raise UnsupportedDtype("a llama2.c checkpoint runs in float32")
    return Decoder.from_llama2c(path, batch, max_seq)


def library(path):
    """A library that can serve the model at `path`, compiled first where it is not."""
    if os.path.isdir(path):
        return ARCHITECTURES[architecture_of(path)][2]()
    return build.for_parallel_decoders()
