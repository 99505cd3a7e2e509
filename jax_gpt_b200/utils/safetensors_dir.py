"""Lazy reading of a model folder's ``*.safetensors`` files."""
from __future__ import annotations

import glob
import os


class SafetensorsDir(dict):
    """All ``*.safetensors`` shards of a folder as one lazy name -> tensor mapping (a tensor is read when asked for)."""

    def __init__(self, model_dir: str):
        super().__init__()
        from safetensors import safe_open
        files = sorted(glob.glob(os.path.join(model_dir, "*.safetensors")))
        if not files:
            raise FileNotFoundError(f"no *.safetensors files in {model_dir}")
        self._where, self._open = {}, {}
        for f in files:
            h = safe_open(f, framework="pt", device="cpu")
            self._open[f] = h
            for k in h.keys():
                self._where[k] = f

    def __contains__(self, k):
        return k in self._where

    def keys(self):
        return self._where.keys()

    def __iter__(self):
        return iter(self._where)

    def __len__(self):
        return len(self._where)

    def __getitem__(self, k):
        return self._open[self._where[k]].get_tensor(k)
