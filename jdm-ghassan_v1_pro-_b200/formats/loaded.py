"""What every model loader returns."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import numpy as np


@dataclass
class LoadedModel:
    cfg: object                           # ModelConfig or LayerListConfig
    named: Dict[str, np.ndarray]          # tensors by parameter name: fp32 arrays, or stored-type tensors of a folder
    moe_bias: List[np.ndarray]
    tokenizer: Optional[object]
    metadata: dict
    tensor_types: Dict[str, int]
    raw: Optional[object] = None          # the open GGUF file, when its stored bytes can be used as they are
