from .registry import (  # noqa: F401
    Architecture,
    ConfigError,
    architecture_name,
    lookup,
    parse_config,
    read_config_json,
    register_architecture,
    registered_architectures,
)
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry  # noqa: F401
from .qwen2_moe import Qwen2MoeConfig  # noqa: F401  (registers the architecture)
from .supevik import SupevikConfig  # noqa: F401  (registers the architecture)
from .fogapel import FogapelConfig  # noqa: F401  (registers the architecture)
from .zosipel import ZosipelConfig  # noqa: F401  (registers the architecture)
from .divadra import DivadraConfig  # noqa: F401  (registers the architecture)
from .ditazen import DitazenConfig  # noqa: F401  (registers the architecture)
from .kulanex import KulanexConfig  # noqa: F401  (registers the architecture)
