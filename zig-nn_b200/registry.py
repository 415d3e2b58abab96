"""Which classes serve which architecture: the host container that reads a model and the engine that runs it.

A model is a GGUF file (its `general.architecture` names the entry) or a folder with config.json (its `architecture`)
and model.safetensors."""
import json
import os

from . import gguf, hostmodel


class UnknownArchitecture(ValueError):
    pass


class Entry:
    def __init__(self, host, engine, load, options=()):
        self.host, self.engine, self.load, self.options = host, engine, load, tuple(options)


ARCHITECTURES = {
    "gpt2": Entry(hostmodel.Gpt2Host, "Gpt2", "from_gguf"),
    "gemma3": Entry(hostmodel.Gemma3Host, "Gemma3", "from_gguf"),
    "Lenisun": Entry(hostmodel.LenisunHost, "Lenisun", "from_folder", ("ctx", "n_seq", "dtype")),
    "Vepinex": Entry(hostmodel.VepinexHost, "Vepinex", "from_folder", ("ctx", "n_seq", "dtype")),
}


def architecture_of(path):
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return json.load(f).get("architecture")
    return gguf.parse(path).get_metadata_string("general.architecture")


def entry(name):
    if name not in ARCHITECTURES:
        raise UnknownArchitecture("architecture %r; known: %s" % (name, ", ".join(sorted(ARCHITECTURES))))
    return ARCHITECTURES[name]


def load_host(path):
    """The host container of the model at `path`."""
    e = entry(architecture_of(path))
    return getattr(e.host, e.load)(path)


def create_engine(host, **options):
    """The engine of a host container. Options that the architecture does not have (ctx, n_seq, dtype) raise."""
    from . import api
    for e in ARCHITECTURES.values():
        if type(host) is e.host:
            unknown = sorted(set(options) - set(e.options))
            if unknown:
                raise ValueError("%s takes no option %s" % (e.engine, ", ".join(unknown)))
            return getattr(api, e.engine)(host, **options)
    raise UnknownArchitecture("no engine for %s" % type(host).__name__)
