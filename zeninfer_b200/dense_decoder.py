"""What the bfloat16 decoders share: a model folder's tensors as resident matrices and vectors, and the logits of a block's rows."""
from __future__ import annotations

import json
import os

import numpy as np

from . import blocks
from .backend import Backend
from .decoder import Decoder
from .safetensors import SafetensorsFile


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


class DenseDecoder(Decoder):
    """A model class sets Config (with from_dict), supplies `_end` beside what Decoder asks for, and leaves `final_norm`, `head` and,
    after a block, `_prefill_buffers()["last"]`.  `tensor(name)` returns a tensor of the model: uint16 bfloat16 bit patterns or
    fp32, in its own shape."""

    PREFILL_MIN = 2
    Config: type

    def _init_dense(self, backend: Backend, cfg, tensor, dtype: str, max_positions: int, device=None) -> None:
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}")
        self.cfg, self.exact, self._tensor = cfg, dtype == "float32", tensor
        self._init_runtime(backend, cfg.vocab, max_positions, device)
        self.handles: list[int] = []
        self.layers: list[dict] = []
        self._pf = None

    @classmethod
    def load(cls, backend: Backend, path: str, **kwargs):
        """A folder with config.json and model.safetensors."""
        with open(os.path.join(path, "config.json")) as f:
            cfg = cls.Config.from_dict(json.load(f))
        with SafetensorsFile(os.path.join(path, "model.safetensors")) as st:
            return cls(backend, cfg, st.array, **kwargs)      # uploads complete before the mapping closes

    # ---- tensors ----
    def _fetch(self, name: str, shape: tuple[int, ...] | None = None) -> np.ndarray:
        a = self._tensor(name)
        if shape is not None and tuple(a.shape) != shape:
            raise ValueError(f"{name}: shape {tuple(a.shape)}, expected {shape}")
        return a

    def _bits(self, name: str, shape: tuple[int, ...]) -> np.ndarray:
        a = self._fetch(name, shape)
        return a if a.dtype == np.uint16 else blocks.to_bf16(a)

    def _upload(self, bits: np.ndarray) -> int:
        bits = np.ascontiguousarray(bits)
        h = self.be.dev_upload("BF16", bits.view(np.uint8), bits.shape[0], bits.shape[1])
        self.handles.append(h)
        return h

    def _matrix(self, *parts: tuple[str, int], columns: int | None = None) -> int:
        """The named tensors' rows, stacked, as one resident bf16 matrix."""
        arrays = [self._bits(name, (rows, self.cfg.width if columns is None else columns)) for name, rows in parts]
        return self._upload(arrays[0] if len(arrays) == 1 else np.concatenate(arrays))

    def _values(self, name: str, shape: tuple[int, ...]) -> np.ndarray:
        a = self._fetch(name, shape)
        return np.array(blocks.from_bf16(a) if a.dtype == np.uint16 else a, np.float32)

    def _vector(self, name: str, shape: tuple[int, ...]):
        return self.torch.from_numpy(self._values(name, shape)).to(self.dev)

    # ---- logits ----
    def _logit_act(self) -> dict:
        return {}

    def _block_logits(self, rows: list[int]):
        torch, st, W = self.torch, self.stream.cuda_stream, self.cfg.width
        ld = round_up(W, 8)
        x = self._prefill_buffers()["last"][torch.tensor(rows, device=self.dev)]
        view = torch.zeros((len(rows), ld), dtype=torch.float32 if self.exact else torch.bfloat16, device=self.dev)
        out = torch.zeros((len(rows), self.vocab), dtype=torch.float32, device=self.dev)
        self.be.dev_sublayer_end_rows(self._end(dict(x=x), out_norm=self.final_norm), len(rows), view.data_ptr(), ld, not self.exact, st)
        self.be.dev_dense_gemm(self.head, view.data_ptr(), ld, len(rows), out.data_ptr(), self.vocab, st, exact=self.exact, **self._logit_act())
        self.stream.synchronize()      # x and view may go once the launches that read them have run
        return out

    def close(self) -> None:
        super().close()
        for h in self.handles:
            self.be.dev_free(h)
        self.handles.clear()
