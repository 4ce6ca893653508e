"""``ZifelornConfig``: the Zifelorn decoder's config.json.

The class is the Python name of the host's ``ZifelornConfig`` (``csrc/host/config_zifelorn.cpp``): keys ``architecture``
("Zifelorn"), ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``logit_scale`` and ``layers`` - a list whose entries name
a mixer (``type`` "latent_attention", which may read an earlier layer's latents through ``kv_from``, or "rglru", a block around
the real-gated linear recurrent unit; sizes and constants under ``mixer``) and a feed-forward (``mlp``: dense, experts, or null).
"""
from __future__ import annotations

from .base import ModelConfig


class ZifelornConfig(ModelConfig):
    @classmethod
    def from_dict(cls, d: dict) -> "ZifelornConfig":
        d = dict(d)
        d.setdefault("architecture", "Zifelorn")
        return super().from_dict(d)
