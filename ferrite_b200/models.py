"""The model families this library serves.  A family is a module with the decode path's calls - config, weights, upload,
precision, forward, kv_cache, slot - and everything that drives a model (the checkpoint reader, the engine, the command
line) finds it here: by a config's `family`, or, when a checkpoint is opened, by config.json."""
import importlib
from types import SimpleNamespace

FAMILIES = {"llama": "llama", "binutar": "binutar", "labepel": "labepel", "vunadra": "vunadra", "ronavik": "ronavik"}  # a config's family -> its module of this package
ARCHITECTURES = {"Binutar": "binutar", "Labepel": "labepel", "Vunadra": "vunadra", "Ronavik": "ronavik"}  # config.json's "architecture" -> family (Hugging Face configs, which have none, are Llama-like)


def module(family):
    assert family in FAMILIES, f"no model family {family!r}: {', '.join(sorted(FAMILIES))}"
    return importlib.import_module("." + FAMILIES[family], __package__)


def of(c):
    """The family module of a model's config."""
    return module(getattr(c, "family", "llama"))


def family_of_json(j):
    """The family of a parsed config.json."""
    name = j.get("architecture")
    assert name is None or name in ARCHITECTURES, f"architecture {name!r} is not served here: {', '.join(sorted(ARCHITECTURES))}"
    return ARCHITECTURES.get(name, "llama")


def of_json(j):
    """The family module of a parsed config.json."""
    return module(family_of_json(j))


def sizes(x):
    """A parsed config's object, and those inside it, with its keys as names."""
    return SimpleNamespace(**{k: sizes(v) if isinstance(v, dict) else v for k, v in x.items()})
