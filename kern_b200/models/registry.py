"""Model families by name: ``name -> (config, manifest builder, synthetic-weights loader)``.

``kern run|bench|server --model NAME`` builds the manifest in memory and fills the weights with the family's
random-init checkpoint on the device (no files), which is how the benchmarks run without a network."""
from __future__ import annotations

import dataclasses
import json
from pathlib import Path

ARCHITECTURES = {"Barotar": "barotar", "Diderax": "diderax", "Fusasun": "fusasun", "Gafapel": "gafapel"}      # config.json's `architecture` -> the module of its family


def is_folder(name: str) -> bool:
    return (Path(name) / "config.json").is_file()


def from_folder(path, **overrides):
    """A checkpoint folder (config.json + safetensors) -> (config with overrides applied, manifest builder); the family is
    the one config.json's `architecture` names."""
    import importlib

    arch = json.loads((Path(path) / "config.json").read_text()).get("architecture")
    if arch not in ARCHITECTURES:
        raise KeyError(f"{path}: unknown architecture `{arch}`; known: {', '.join(sorted(ARCHITECTURES))}")
    mod = importlib.import_module(f".{ARCHITECTURES[arch]}", __package__)
    return mod.from_folder(path, **{k: v for k, v in overrides.items() if v is not None}), mod.build_manifest


def families() -> dict:
    from . import barotar, dense, diderax, fusasun, gafapel, hybrid, latent, moe

    out = {}
    for cfg in (dense.TOY, dense.TINY, dense.DENSE_8B):
        out[cfg.name] = (cfg, dense.build_manifest, dense.load_random_weights, dense.random_weights)
    for cfg in (hybrid.TOY_HYBRID, hybrid.TINY_HYBRID, hybrid.TINY_HYBRID_K128, hybrid.HYBRID_27B):
        out[cfg.name] = (cfg, hybrid.build_manifest, hybrid.load_random_weights, hybrid.random_weights)
    for cfg in (moe.TOY_MOE, moe.TINY_MOE, moe.MOE_30B):
        out[cfg.name] = (cfg, moe.build_manifest, moe.load_random_weights, moe.random_weights)
    for cfg in (latent.TINY_LATENT, latent.TINY_LATENT_K128, latent.TINY_LATENT_MOE, latent.LATENT_48B):
        out[cfg.name] = (cfg, latent.build_manifest, latent.load_random_weights,
                         lambda cfg, **kw: latent.folded(cfg, latent.random_weights(cfg, **kw)))
    for cfg in (gafapel.TINY_GAFAPEL, gafapel.GAFAPEL_LARGE):
        out[cfg.name] = (cfg, gafapel.build_manifest, gafapel.load_random_weights, gafapel.random_weights)
    for cfg in (barotar.TINY_BAROTAR, barotar.BAROTAR_LARGE):
        out[cfg.name] = (cfg, barotar.build_manifest, barotar.load_random_weights, barotar.random_weights)
    for cfg in (diderax.TINY_DIDERAX, diderax.DIDERAX_LARGE):
        out[cfg.name] = (cfg, diderax.build_manifest, diderax.load_random_weights, diderax.random_weights)
    for cfg in (fusasun.TINY_FUSASUN, fusasun.FUSASUN_LARGE):
        out[cfg.name] = (cfg, fusasun.build_manifest, fusasun.load_random_weights, fusasun.random_weights)
    from . import toy_int

    for lined in (False, True):
        name = "toy-int-stateful" if lined else "toy-int"
        out[name] = (lined, lambda lined: toy_int.build_manifest(lined), lambda rt, cfg: None, lambda cfg: None)
    return out


def resolve(name: str, **overrides):
    """-> (config with overrides applied, builder, device loader, host weights maker). `name`: a family, or a checkpoint folder."""
    if is_folder(name):
        from .common import read_safetensors

        cfg, build = from_folder(name, **overrides)
        files = sorted(str(p) for p in Path(name).glob("*.safetensors"))
        return cfg, build, lambda rt, cfg: rt.load_weights(files), \
            lambda cfg: {k: t for f in files for k, t in read_safetensors(f).items()}
    fam = families()
    if name not in fam:
        raise KeyError(f"unknown model `{name}`; known: {', '.join(sorted(fam))}")
    cfg, build, load, make = fam[name]
    overrides = {k: v for k, v in overrides.items() if v is not None}
    if not dataclasses.is_dataclass(cfg):
        return cfg, build, load, make          # a family without a config object (the integer model)
    return dataclasses.replace(cfg, **overrides), build, load, make
