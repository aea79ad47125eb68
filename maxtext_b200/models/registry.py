"""Model folders: `config.json` (with an `architecture` name) plus `model.safetensors`.

`model_dir=<folder>` on any command line makes the folder the model: `config_keys` turns its config.json into configuration keys
(merged like a catalog entry of `configs/models/`), `load_weights` fills the parameter store from its tensors. One entry of
ARCHITECTURES per supported architecture; an entry is a module with `keys_from_json(spec, shapes)` and
`tensors_for(store, config, get)`, a generator of (parameter name, value in the internal layout).
"""
from __future__ import annotations

import json
import os
import struct

import torch

from . import gukirax, silinex, sitivik, tipidra

ARCHITECTURES = {"Gukirax": gukirax, "Silinex": silinex, "Sitivik": sitivik, "Tipidra": tipidra}


def _safetensors_files(path: str) -> list[str]:
  return [os.path.join(path, f) for f in sorted(os.listdir(path)) if f.endswith(".safetensors")]


def tensor_shapes(path: str) -> dict:
  """name -> shape of every tensor of the folder, from the file headers alone."""
  out = {}
  for f in _safetensors_files(path):
    with open(f, "rb") as fh:
      (n,) = struct.unpack("<Q", fh.read(8))
      head = json.loads(fh.read(n))
    out.update({k: tuple(v["shape"]) for k, v in head.items() if k != "__metadata__"})
  return out


def read_spec(path: str) -> dict:
  with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as fh:
    return json.load(fh)


def architecture(spec: dict):
  name = spec.get("architecture")
  if name not in ARCHITECTURES:
    raise ValueError(f"unknown architecture {name!r} (known: {sorted(ARCHITECTURES)})")
  return ARCHITECTURES[name]


def config_keys(path: str) -> dict:
  """Configuration keys of the model folder."""
  spec = read_spec(path)
  return architecture(spec).keys_from_json(spec, tensor_shapes(path))


@torch.no_grad()
def load_weights(path: str, store, config) -> None:
  """Fill every parameter of the store from the folder's tensors; a parameter without a tensor is an error."""
  from safetensors import safe_open
  files = [safe_open(f, framework="pt") for f in _safetensors_files(path)]
  where = {k: f for f in files for k in f.keys()}

  def get(name: str) -> torch.Tensor:
    if name not in where:
      raise KeyError(f"{path}: no tensor {name!r}")
    return where[name].get_tensor(name).float()
  left = set(store.params)
  for name, value in architecture(read_spec(path)).tensors_for(store, config, get):
    want = store.params[name].pdef.global_shape()
    if tuple(value.shape) != tuple(want):
      raise ValueError(f"{name}: tensor of shape {tuple(value.shape)}, expected {tuple(want)}")
    store.load_full(name, store.params[name].pdef.local_slice(value).contiguous())
    left.discard(name)
  if left:
    raise KeyError(f"no tensors for parameters {sorted(left)[:5]}")
  store.sync_compute_from_master()
