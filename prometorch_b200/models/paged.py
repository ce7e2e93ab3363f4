"""What the batching engine (``serve/llm.py``) asks of a model, and the registry that finds the model for a ``config.json``.

The engine owns requests, the page table, the page pool, recurrent states, CUDA graphs and sampling.  A model owns its weights and
the device work of two passes over the engine's cache: a prompt pass (many tokens of several sequences) and a decode pass (one token per
batch row).  A new design is a :class:`PagedModel` with a configuration and a weights class, registered under the name its
``config.json`` carries."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch


@dataclass
class PromptBatch:
    """Tokens of several sequences, concatenated.  ``offs[i]:offs[i + 1]`` are the tokens of sequence i, ``starts[i]`` is the
    position of its first one (0 unless the sequence already has tokens in the cache)."""
    ids: torch.Tensor                  # [n] int32
    pos: torch.Tensor                  # [n] int32, position in the sequence
    req: torch.Tensor                  # [n] int32, row of the page table
    offs: List[int]
    starts: List[int]
    rows: List[int]                    # page-table row of every sequence
    want: Optional[torch.Tensor] = None      # [m] int64, places among the n tokens whose logits are asked for

    def lens(self) -> List[int]:
        return [b - a for a, b in zip(self.offs, self.offs[1:])]


class RowPack:
    """Matrices that read the same input, stacked by rows into one: ``sizes`` maps names to row counts.  Every part starts at a
    multiple of eight rows and the whole has one (what the projection kernel and 16-byte loads of its output ask for); the gaps
    are zeros.  ``at[name]``: a part's first column in the product."""

    def __init__(self, sizes: Dict[str, int]):
        self.sizes, self.at, self.rows = dict(sizes), {}, 0
        for n, k in sizes.items():
            self.at[n] = self.rows
            self.rows += self.up(k)

    @staticmethod
    def up(n: int) -> int:
        return -(-n // 8) * 8

    @staticmethod
    def pad(t: torch.Tensor) -> torch.Tensor:
        """``t`` with rows of zeros up to a multiple of eight."""
        more = RowPack.up(t.shape[0]) - t.shape[0]
        return torch.cat([t, t.new_zeros((more,) + tuple(t.shape[1:]))]) if more else t.contiguous()

    def pack(self, parts: Dict[str, torch.Tensor]) -> torch.Tensor:
        return torch.cat([self.pad(parts[n]) for n in self.sizes])

    def cols(self, product: torch.Tensor, name: str, padded: bool = False) -> torch.Tensor:
        """A part's columns of ``product [n, rows]`` (a view); ``padded``: up to the next multiple of eight."""
        k = self.sizes[name]
        return product[:, self.at[name]:self.at[name] + (self.up(k) if padded else k)]


class PagedModel:
    """Base class: ``cfg`` must have ``vocab_size``, ``max_position_embeddings``, ``bos_token_id`` and ``eos_token_id``."""
    architecture = ""
    continues_prompts = False          # whether a prompt pass may start behind cached tokens
    rewinds = True                     # whether a decoded token can be taken back by decoding another one at its position

    def __init__(self, weights, device, dtype):
        self.cfg = weights.cfg
        self.device, self.dtype = device, dtype
        self.weights = weights.to(device, dtype)

    def kv_shapes(self) -> List[Tuple[int, int, int]]:
        """(kv heads, key size, value size) of every layer's cache, in elements as stored."""
        raise NotImplementedError

    def state_shapes(self) -> List[Dict[str, Tuple[tuple, torch.dtype]]]:
        """What each layer keeps per sequence besides pages: name -> (shape, dtype).  The engine holds one slot of it per page-table
        row; a pass whose first token stands at position 0 takes the slot's content as zero.  Entries past the layers' are the model's own."""
        return [{} for _ in self.kv_shapes()]

    def kept_tokens(self) -> int:
        """How many of a sequence's first tokens stay readable whatever :meth:`cache_window` says."""
        return 0

    def cache_window(self) -> Optional[int]:
        """How many of the latest tokens any layer can still read (None: all of them).  Pages that lie behind go back to the
        pool while the sequence runs."""
        return None

    def pick_splits(self, rows: int, max_len: int) -> int:
        """Split count of the decode pass's attention (part of the key of its CUDA graph)."""
        raise NotImplementedError

    def prompt_pass(self, kv, page_table: torch.Tensor, batch: PromptBatch, hidden: bool = False) -> torch.Tensor:
        """Runs the batch, fills its pages; fp32 logits of the wanted places, or every position's final hidden state."""
        raise NotImplementedError

    def decode_pass(self, kv, page_table: torch.Tensor, meta: torch.Tensor, nsplit: int) -> torch.Tensor:
        """One token per row.  ``meta [B, 4]`` int32: token id, position, page-table row, cached length; logits ``[B, V]``."""
        raise NotImplementedError


@dataclass(frozen=True)
class ModelEntry:
    name: str
    config: type                       # has from_dict(json object)
    weights: type                      # has from_state_dict(cfg, tensors) and to(device, dtype)
    model: type                        # a PagedModel


_MODELS: Dict[str, ModelEntry] = {}
_DEFAULT = "llama"


def register_model(config: type, weights: type, model: type, *names: str) -> None:
    for n in names:
        _MODELS[n.lower()] = ModelEntry(names[0], config, weights, model)


def _ensure_builtin():
    from . import budorax, gelutar, kifusun, llama_paged, tifepel  # noqa: F401  (they register themselves)


def known_models() -> List[str]:
    _ensure_builtin()
    return sorted({e.name for e in _MODELS.values()})


def resolve_architecture(config: dict) -> ModelEntry:
    """The entry for a parsed ``config.json``: by ``architecture``, then the Hugging Face keys.  A directory that names no
    design is read as Llama, which is what the engine served first."""
    _ensure_builtin()
    own = config.get("architecture")
    if own is not None:
        if str(own).lower() not in _MODELS:
            raise ValueError(f"no model is registered for architecture {own!r} (known: {', '.join(known_models())})")
        return _MODELS[str(own).lower()]
    for n in list(config.get("architectures") or []) + [config.get("model_type")]:
        if n is not None and str(n).lower() in _MODELS:
            return _MODELS[str(n).lower()]
    return _MODELS[_DEFAULT]


def entry_of(cfg) -> ModelEntry:
    """The entry whose configuration class ``cfg`` is."""
    _ensure_builtin()
    for e in _MODELS.values():
        if type(cfg) is e.config:
            return e
    raise ValueError(f"no model is registered for a {type(cfg).__name__}")


def read_config(model_dir: str) -> Optional[dict]:
    path = os.path.join(model_dir, "config.json")
    if not os.path.exists(path):
        return None
    with open(path, encoding="utf-8") as f:
        return json.load(f)
