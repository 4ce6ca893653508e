"""``BuguzenConfig``: the Buguzen decoder's config.json.

The class is the Python name of the host's ``BuguzenConfig`` (``csrc/host/config_buguzen.cpp``): keys ``architecture``
("Buguzen"), ``vocab``, ``width``, ``norm.eps``, ``token_side``, ``loop`` and ``layers`` - a list whose entries name a mixer (``type``
"attention", differential; "attention_2", whose values are its keys; or "lightning", linear attention with a fixed decay per head;
sizes and constants under ``mixer``) and a feed-forward (``mlp``: dense, or null).
"""
from __future__ import annotations

from .base import ModelConfig


class BuguzenConfig(ModelConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "BuguzenConfig":
        d = dict(d)
        d.setdefault("architecture", "Buguzen")
        return super().from_dict(d)
