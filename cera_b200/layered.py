"""Host side of cera_cuda_model_create_layered: a decoder given as a list of layer descriptions.

The model object is CudaModel's: forward, forward_prefill, generate_greedy, snapshot and the rest are inherited."""
import ctypes as C
import enum
import os

from ._lib import LayerDesc, LayeredConfig, check, lib
from .model import CudaModel
from .safetensors import SafetensorsFile
from .types import BF16, F32

DTYPES = {"bfloat16": BF16, "float32": F32}


class Mixer(enum.IntEnum):
    LATENT_ATTENTION = 1
    MINGRU = 2
    ATTENTION = 3
    RGLRU = 4
    SSM = 5


class Ff(enum.IntEnum):
    NONE = 0
    MOE = 1
    GATED = 2


class LayeredModel(CudaModel):
    def __init__(self, layers, dtype="bfloat16", device=0, **cfg):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r} is not one of {sorted(DTYPES)}")
        self.cfg = LayeredConfig(n_layers=len(layers), dtype=DTYPES[dtype], device=device, **cfg)
        self.layers = list(layers)
        self.tp = (0, 1)
        self.handle = C.c_void_p()
        arr = (LayerDesc * len(layers))(*layers)
        check(lib.cera_cuda_model_create_layered(C.byref(self.cfg), arr, C.byref(self.handle)))

    def add_tensor(self, role, layer, ggml_type, rows, cols, data, expert=None):
        if expert is None:
            return super().add_tensor(role, layer, ggml_type, rows, cols, data)
        ptr, nbytes, keep = self._raw(data)
        check(lib.cera_cuda_model_add_expert_tensor(self.handle, int(role), layer, expert, ggml_type, rows, cols, C.c_void_p(ptr), nbytes))
        del keep

    def load(self, folder, roles):
        """Give the model every tensor of `roles` - (name, role, layer, expert or None) - from folder/model.safetensors, and finalize."""
        with SafetensorsFile(os.path.join(folder, "model.safetensors")) as f:
            for name, role, layer, expert in roles:
                rows, cols, kind, data = f.get(name)
                self.add_tensor(role, layer, kind, rows, cols, data, expert=expert)
                del data
        self.finalize()
