from .config import DufitarConfig, DufitarLayerConfig  # noqa: F401
from .loader import load_dufitar_weights, load_model_dir  # noqa: F401
from .model import DufitarModel  # noqa: F401
