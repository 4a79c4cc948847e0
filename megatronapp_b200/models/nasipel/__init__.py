from .config import NasipelConfig, NasipelLayerConfig  # noqa: F401
from .loader import load_model_dir, load_nasipel_weights  # noqa: F401
from .model import NasipelModel  # noqa: F401
