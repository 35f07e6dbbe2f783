"""Engine-mode decoders: layer arithmetic over flat ragged batches and paged caches, by model family."""
from .config import ModelConfig
from .weights import init_reference_order
from .transformer import EngineTransformerLM
from . import registry
from .registry import ModelFamily, build_model, family_of, init_weights, resolve_config
from .nabalix import NabalixConfig, NabalixLM
from .taminex import TaminexConfig, TaminexLM
from .meresun import MeresunConfig, MeresunLM
from .sodonex import SodonexConfig, SodonexLM

registry.register(ModelFamily(registry.DEFAULT_FAMILY, ModelConfig, EngineTransformerLM, init_reference_order))

__all__ = ["ModelConfig", "init_reference_order", "EngineTransformerLM", "ModelFamily", "build_model", "family_of",
           "init_weights", "resolve_config", "NabalixConfig", "NabalixLM", "TaminexConfig", "TaminexLM",
           "MeresunConfig", "MeresunLM", "SodonexConfig", "SodonexLM"]
