"""Model families that are opened from a checkpoint directory: ``config.json`` names the architecture, the registry names the
module that reads it. Command lines (engine worker, trace replay) go through :func:`open_checkpoint`; a family is added with one
entry here."""
from __future__ import annotations

import importlib
import json
from dataclasses import dataclass
from pathlib import Path
from typing import Tuple


@dataclass(frozen=True)
class Family:
    architecture: str          # "architecture" of config.json
    module: str                # under ironpangu_b200.models
    decoder: str               # class with from_checkpoint(path, fabric, ...)
    rows: str                  # packed-step executor over that decoder
    exact: bool                # has a true 32-bit mode
    presets: Tuple[str, ...] = ()      # names of PRESETS of the module: configurations served with random weights

    def load(self):
        return importlib.import_module(f"ironpangu_b200.models.{self.module}")


FAMILIES: Tuple[Family, ...] = (Family("Falinex", "falinex", "FalinexDecoder", "FalinexRows", True, ("falinex-tiny", "falinex2b")),
                                Family("Ponenex", "ponenex", "PonenexDecoder", "PonenexRows", True, ("ponenex-tiny", "ponenex-text")),
                                Family("Mikutar", "mikutar", "MikutarDecoder", "MikutarRows", True, ("mikutar-tiny", "mikutar-text")),
                                Family("Fubelorn", "fubelorn", "FubelornDecoder", "FubelornRows", True, ("fubelorn-tiny", "fubelorn-text")))


def family_of(checkpoint_dir) -> Family:
    """The family ``config.json`` of a checkpoint directory names."""
    cfg = json.loads((Path(checkpoint_dir) / "config.json").read_text())
    name = cfg.get("architecture")
    for f in FAMILIES:
        if f.architecture == name:
            return f
    raise ValueError(f"no model family for architecture {name!r} (known: {', '.join(f.architecture for f in FAMILIES)})")


def preset_names() -> Tuple[str, ...]:
    return tuple(n for f in FAMILIES for n in f.presets)


def open_preset(name: str, fabric, *, layers: int = 0, seed: int = 0, max_rows: int = 512, **decoder_options):
    """``(decoder, packed-step executor)`` of a preset configuration with random weights; ``layers`` keeps the first so many."""
    f = next((f for f in FAMILIES if name in f.presets), None)
    if f is None:
        raise ValueError(f"no preset {name!r} (known: {', '.join(preset_names())})")
    mod = f.load()
    cfg = mod.PRESETS[name]()
    if layers:
        cfg.layers = cfg.layers[:layers]
    dec = getattr(mod, f.decoder)(cfg, mod.random_weights(cfg, fabric.device, seed=seed), fabric, **decoder_options)
    return dec, getattr(mod, f.rows)(dec, max_rows=max_rows)


def open_checkpoint(checkpoint_dir, fabric, *, max_rows: int = 512, **decoder_options):
    """``(decoder, packed-step executor)`` of a checkpoint directory."""
    f = family_of(checkpoint_dir)
    mod = f.load()
    dec = getattr(mod, f.decoder).from_checkpoint(checkpoint_dir, fabric, **decoder_options)
    return dec, getattr(mod, f.rows)(dec, max_rows=max_rows)
