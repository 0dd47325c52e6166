from .schema import ConfigError, LayerSpec, ModelSpec, PartSpec, RunEntry
from .registry import (architecture_of, known_architectures, model_spec_from_config,
                       model_spec_from_dir, read_config_json, register_architecture)
from . import qwen3 as _qwen3
from .qwen3 import Qwen3Config
from . import mugizen as _mugizen
from . import vivesun as _vivesun
from . import beralix as _beralix
from . import nefipel as _nefipel
from . import pubulix as _pubulix
from . import difavik as _difavik

register_architecture(_qwen3.ARCHITECTURE, _qwen3.spec_from_config, replace=True)
register_architecture(_mugizen.ARCHITECTURE, _mugizen.spec_from_config, replace=True)
register_architecture(_vivesun.ARCHITECTURE, _vivesun.spec_from_config, replace=True)
register_architecture(_beralix.ARCHITECTURE, _beralix.spec_from_config, replace=True)
register_architecture(_nefipel.ARCHITECTURE, _nefipel.spec_from_config, replace=True)
register_architecture(_pubulix.ARCHITECTURE, _pubulix.spec_from_config, replace=True)
register_architecture(_difavik.ARCHITECTURE, _difavik.spec_from_config, replace=True)

__all__ = [
    "ConfigError", "LayerSpec", "ModelSpec", "PartSpec", "RunEntry", "Qwen3Config",
    "architecture_of", "known_architectures", "model_spec_from_config", "model_spec_from_dir",
    "read_config_json", "register_architecture",
]
