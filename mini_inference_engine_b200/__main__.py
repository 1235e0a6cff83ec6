"""``python -m mini_inference_engine_b200``."""

import sys

from .cli import main

sys.exit(main())
