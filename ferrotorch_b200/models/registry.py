"""Registry of decoder families: which class loads the model of a directory, chosen by its ``config.json``.

A family registers a predicate on the configuration and the class that serves it.  The class offers
``from_pretrained(path, dtype, device)``, ``tiny_random(dtype, device)``, ``config`` (with ``vocab_size``, ``max_position_embeddings`` or ``None``),
``make_paged_cache`` and ``paged_forward``: what :class:`~ferrotorch_b200.models.serving.PagedStepper` and the server need."""
from __future__ import annotations

import importlib
import json
import os
from dataclasses import dataclass
from typing import Callable


@dataclass(frozen=True)
class CausalLMFamily:
    name: str
    matches: Callable[[dict], bool]
    model: str                    # "module:class"

    def model_class(self):
        mod, cls = self.model.split(":")
        return getattr(importlib.import_module(mod), cls)


_FAMILIES: list[CausalLMFamily] = []


def register_causal_lm(family: CausalLMFamily) -> None:
    """Later registrations are asked first."""
    _FAMILIES.insert(0, family)


def list_causal_lms() -> list[str]:
    return sorted(f.name for f in _FAMILIES)


def family_named(name: str) -> CausalLMFamily:
    for fam in _FAMILIES:
        if fam.name == name:
            return fam
    raise ValueError("no decoder family %r (known: %s)" % (name, ", ".join(list_causal_lms())))


def family_of(cfg: dict | str) -> CausalLMFamily:
    """The family of a configuration: a dict, a ``config.json`` or a directory that holds one."""
    if isinstance(cfg, str):
        with open(os.path.join(cfg, "config.json") if os.path.isdir(cfg) else cfg) as f:
            cfg = json.load(f)
    for fam in _FAMILIES:
        if fam.matches(cfg):
            return fam
    raise ValueError("no registered decoder family for this configuration (known: %s)" % ", ".join(list_causal_lms()))


def load_causal_lm(path: str, dtype=None, device="cpu"):
    """The model of a directory, as an instance of its family's class (``dtype`` default: bfloat16)."""
    import torch

    return family_of(path).model_class().from_pretrained(path, dtype=dtype or torch.bfloat16, device=device).eval()


def _is_llama(cfg: dict) -> bool:
    # Llama-shaped Hugging Face configurations, named so or not
    archs = cfg.get("architectures") or []
    return "LlamaForCausalLM" in archs or cfg.get("model_type") == "llama" or (not archs and "hidden_size" in cfg and "num_attention_heads" in cfg)


register_causal_lm(CausalLMFamily("llama", _is_llama, "ferrotorch_b200.models.llama:LlamaForCausalLM"))
register_causal_lm(CausalLMFamily("bopudra", lambda c: c.get("architecture") == "Bopudra", "ferrotorch_b200.models.bopudra:BopudraForCausalLM"))
register_causal_lm(CausalLMFamily("zolorax", lambda c: c.get("architecture") == "Zolorax", "ferrotorch_b200.models.zolorax:ZoloraxForCausalLM"))
register_causal_lm(CausalLMFamily("tenalorn", lambda c: c.get("architecture") == "Tenalorn", "ferrotorch_b200.models.tenalorn:TenalornForCausalLM"))
register_causal_lm(CausalLMFamily("mogelix", lambda c: c.get("architecture") == "Mogelix", "ferrotorch_b200.models.mogelix:MogelixForCausalLM"))
