"""Model classes.  :func:`model_class` picks the one a configuration names, as every loader of the package does."""
from __future__ import annotations


def model_class(cfg):
    """The model class of a :class:`blaze_b200.config.ModelConfig`."""
    if cfg.architecture == "Sevevik":
        from .sevevik import Sevevik
        return Sevevik
    if cfg.architecture == "Niletar":
        from .niletar import Niletar
        return Niletar
    if cfg.architecture == "Rapisun":
        from .rapisun import Rapisun
        return Rapisun
    if cfg.architecture == "Medodra":
        from .medodra import Medodra
        return Medodra
    from .qwen3 import Model
    return Model
