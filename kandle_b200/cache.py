"""What the layers of a hybrid decoder keep between steps, for a batch of sequences at one position.

  LatentRows    latent attention: one row (normed latent, rotated shared key part) per token,
                [B, maxS, width]; several layers may read the same rows
  KeyValueRows  grouped-query attention: a key row (after norm and rotation) and a value row per token
                and key head, [B, G, maxS, size]; several layers may read the same rows
  DeltaState    gated delta rule: the fp32 state matrix of every head and the last inputs of the short
                convolution; fixed size, carried from token to token
  WkvState      WKV recurrence: the fp32 state matrix of every head and the last token's input row

`SequenceCache` owns one such object per layer that has one of its own, the write position shared by
all layers, and the reset that hands the memory to the next request.
"""
from __future__ import annotations

import ctypes

from . import core, lib
from .core import Tensor
from .model_utils.pedorax import ChannelDeltaSpec, LatentAttentionSpec
from .model_utils.vogozen import HeadDeltaSpec, WindowAttentionSpec, WkvSpec


def _fill_zero(t: Tensor) -> None:
    lib.call("kd_fill", ctypes.byref(t._handle.c()), ctypes.c_double(0.0))


class LatentRows:
    """Rows are padded to a multiple of 16 numbers (zeros): whole 32-byte pieces for the bf16 kernels."""

    def __init__(self, spec: LatentAttentionSpec, batch: int, max_seq_len: int, dtype: str, hidden: int):
        self.width = (spec.kvRank + spec.rotDim + 15) // 16 * 16
        self.rows = core.zeros((batch, max_seq_len, self.width), dtype)

    def reset(self) -> None:
        pass                      # rows at and past the write position are never read

    def carried(self) -> list:
        return []

    def numbers_per_token(self) -> int:
        return self.width


class KeyValueRows:
    """All positions are kept, also those behind a window: another layer may read the same rows through a longer one.
    Reused memory must hold finite numbers, which rows of an earlier request are (kd_window_attention)."""

    def __init__(self, spec: WindowAttentionSpec, batch: int, max_seq_len: int, dtype: str, hidden: int):
        qd, vd = ctypes.c_int(0), ctypes.c_int(0)
        lib.call("kd_attention_head_sizes", lib.DTYPES[dtype][0], spec.dim, spec.vdim, ctypes.byref(qd), ctypes.byref(vd))
        self.heads, self.q_size, self.v_size = spec.kvHeads, qd.value, vd.value
        self.keys = core.zeros((batch, spec.kvHeads, max_seq_len, self.q_size), dtype)
        self.values = core.zeros((batch, spec.kvHeads, max_seq_len, self.v_size), dtype)

    def reset(self) -> None:
        pass                      # rows past the write position get no weight

    def carried(self) -> list:
        return []

    def numbers_per_token(self) -> int:
        return self.heads * (self.q_size + self.v_size)


def _state_matrices(batch: int, heads: int, dim: int, vdim: int) -> Tensor:
    r, c = ctypes.c_int(0), ctypes.c_int(0)
    lib.call("kd_delta_state_shape", dim, vdim, ctypes.byref(r), ctypes.byref(c))
    return core.zeros((batch, heads, r.value, c.value), "float32")


class DeltaState:
    def __init__(self, spec: ChannelDeltaSpec | HeadDeltaSpec, batch: int, max_seq_len: int, dtype: str, hidden: int):
        self.state = _state_matrices(batch, spec.heads, spec.dim, spec.vdim)
        self.history = core.zeros((batch, max(spec.taps - 1, 1), spec.channels), dtype)

    def reset(self) -> None:
        _fill_zero(self.state)
        _fill_zero(self.history)

    def carried(self) -> list:
        return [self.state, self.history]


class WkvState:
    def __init__(self, spec: WkvSpec, batch: int, max_seq_len: int, dtype: str, hidden: int):
        self.state = _state_matrices(batch, spec.heads, spec.dim, spec.dim)
        self.last = core.zeros((batch, hidden), dtype)

    def reset(self) -> None:
        _fill_zero(self.state)
        _fill_zero(self.last)

    def carried(self) -> list:
        return [self.state, self.last]


_KEPT = {LatentAttentionSpec: LatentRows, WindowAttentionSpec: KeyValueRows, ChannelDeltaSpec: DeltaState, HeadDeltaSpec: DeltaState, WkvSpec: WkvState}


class SequenceCache:
    def __init__(self, layers, batch: int, max_seq_len: int, dtype: str, hidden: int):
        self.batch, self.max_seq_len, self._number = batch, max_seq_len, 2 if dtype == "bfloat16" else 4
        self.pos = 0
        self._of = []
        for layer in layers:
            m = layer.mixer
            src = getattr(m, "kvFrom", None)
            self._of.append(_KEPT[type(m)](m, batch, max_seq_len, dtype, hidden) if src is None else self._of[src])
        self._own = list({id(x): x for x in self._of}.values())

    def of(self, layer: int):
        return self._of[layer]

    def reset(self) -> None:
        """Position 0 and zero recurrent state: the sequences are over, new ones may use their place."""
        for x in self._own:
            x.reset()
        self.pos = 0

    def room(self, tokens: int) -> None:
        if self.pos + tokens > self.max_seq_len:
            raise ValueError(f"Cache overflow: trying to write to position {self.pos}-{self.pos + tokens}, but maxSeqLen is {self.max_seq_len}")

    def snapshot(self) -> list:
        """Copies of everything that a step overwrites in place (a cache row can simply be written again)."""
        return [(t, t.clone()) for x in self._own for t in x.carried()]

    @staticmethod
    def restore(saved: list) -> None:
        for t, copy in saved:
            core.copy_(t, copy)
            copy.dispose()

    def bytes_per_token(self) -> int:
        return sum(x.numbers_per_token() * self._number for x in self._own if hasattr(x, "numbers_per_token"))

    def state_bytes(self) -> int:
        """Recurrent state per sequence."""
        return sum(t.numel // self.batch * (2 if t.dtype == "bfloat16" else 4) for x in self._own for t in x.carried())
