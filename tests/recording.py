"""The drivers of the bf16-weight designs on CPU tensors, with the library replaced by a recorder."""

import pytest
import torch

from quickdraw_b200 import _lib, hybrid, mixers


class AsIfOnGpu(torch.Tensor):
    is_cuda = property(lambda self: True)


@pytest.fixture
def recorder(monkeypatch):
    """The drivers on CPU tensors with the library replaced by a recorder of (name, arguments)."""
    seen = []

    def record(name, *args):
        declared = _lib.HYBRID_LIBRARIES[_lib.HYBRID_OWNER[name]][name]
        assert len(args) == len(declared), (name, len(args), len(declared))
        seen.append((name, args))

    class Properties:
        multi_processor_count = 148

    for module in (hybrid, mixers):
        monkeypatch.setattr(module, "call_hybrid", record)
        monkeypatch.setattr(module, "stream_of", lambda t: None)
    monkeypatch.setattr(mixers, "size_hybrid", lambda name, *args: 4096)
    monkeypatch.setattr(torch.cuda, "get_device_properties", lambda device: Properties)
    return seen
