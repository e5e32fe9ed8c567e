"""The model families this library serves, by what config.json says: how a checkpoint folder becomes a model shape,
weights on the device, a cache and lanes (the reference has one family per loader, monoserve/runtime/config.py:46-66 and
monoserve/runtime/checkpoint.py:99-196).

    model = load(folder)                                    # config, weights
    kv = model.cache(n_pages, page_size, slots)
    lane_class(model.cfg)(fab, 0, model.cfg, model.weights, kv, ...)
"""
import json
import os


class _MoE:
    """Qwen3-MoE and GLM-4.5 MoE (monoserve_b200/model.py)."""

    @staticmethod
    def matches(config):
        return config.get("model_type") in ("qwen3_moe", "glm4_moe")

    @staticmethod
    def owns(cfg):
        return getattr(cfg, "model_type", None) in (None, "qwen3_moe", "glm4_moe")

    @staticmethod
    def load(folder, config, dtype):
        if dtype != "bfloat16":
            raise NotImplementedError(f"{config['model_type']} runs in bfloat16")
        from monoserve_b200.checkpoint import read_checkpoint
        from monoserve_b200.model import ModelWeights
        cfg, w = read_checkpoint(folder)
        return cfg, ModelWeights(cfg, w)

    @staticmethod
    def cache(cfg, n_pages, page_size, slots):
        from monoserve_b200.model import KVCache
        return KVCache(cfg, n_pages, page_size)

    @staticmethod
    def lane():
        from monoserve_b200.model import ModelLane
        return ModelLane


class _LayerList:
    """Decoders whose configuration lists a mixer per layer: Sinotar, Teganex (monoserve_b200/layer_list.py)."""

    @staticmethod
    def matches(config):
        from monoserve_b200.layer_list import DESIGNS
        return config.get("architecture") in DESIGNS

    @staticmethod
    def owns(cfg):
        return getattr(cfg, "model_type", None) in ("sinotar", "teganex")

    @staticmethod
    def load(folder, config, dtype):
        from monoserve_b200.layer_list import Weights, read_config, read_tensors
        cfg = read_config(config, dtype)
        return cfg, Weights(cfg, read_tensors(folder))

    @staticmethod
    def cache(cfg, n_pages, page_size, slots):
        from monoserve_b200.layer_list import LayerListCache
        return LayerListCache(cfg, n_pages, page_size, slots)

    @staticmethod
    def lane():
        from monoserve_b200.layer_list import LayerListLane
        return LayerListLane


FAMILIES = (_MoE, _LayerList)


def lane_class(cfg, default=None):
    """The lane class of a model shape; `default` stands in for the MoE decoders' class."""
    family = next(f for f in FAMILIES if f.owns(cfg))
    return default if default is not None and family is _MoE else family.lane()


class Model:
    def __init__(self, family, cfg, weights):
        self.family, self.cfg, self.weights = family, cfg, weights

    def cache(self, n_pages, page_size=16, slots=8):
        return self.family.cache(self.cfg, n_pages, page_size, slots)


def load(folder, dtype="bfloat16"):
    """The model of a checkpoint folder (config.json and safetensors), its weights on the device."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    for family in FAMILIES:
        if family.matches(config):
            return Model(family, *family.load(folder, config, dtype))
    raise NotImplementedError(f"no model family for {config.get('model_type') or config.get('architecture')}")
