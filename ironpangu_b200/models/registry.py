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

    def load(self):
        return importlib.import_module(f"ironpangu_b200.models.{self.module}")


FAMILIES: Tuple[Family, ...] = (Family("Falinex", "falinex", "FalinexDecoder", "FalinexRows", True),)


def family_of(checkpoint_dir) -> Family:
    """The family ``config.json`` of a checkpoint directory names."""
    cfg = json.loads((Path(checkpoint_dir) / "config.json").read_text())
    name = cfg.get("architecture")
    for f in FAMILIES:
        if f.architecture == name:
            return f
    raise ValueError(f"no model family for architecture {name!r} (known: {', '.join(f.architecture for f in FAMILIES)})")


def open_checkpoint(checkpoint_dir, fabric, *, max_rows: int = 512, **decoder_options):
    """``(decoder, packed-step executor)`` of a checkpoint directory."""
    f = family_of(checkpoint_dir)
    mod = f.load()
    dec = getattr(mod, f.decoder).from_checkpoint(checkpoint_dir, fabric, **decoder_options)
    return dec, getattr(mod, f.rows)(dec, max_rows=max_rows)
