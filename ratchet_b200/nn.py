"""Thin graph builders over ``Tensor``, restating ratchet-nn (crates/ratchet-nn/src) so the model
graphs of the reference can be scheduled on the CUDA device exactly as written there.

Modules are duck-typed over the tensor class: anything with ratchet's ``Tensor`` method names works
(the tests run the same modules over a CPU-oracle tensor to get the reference result).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from . import capi


class Linear:
    """ratchet-nn/src/linear.rs:10-24: ``w.gemm(x, bias.cast(x.dt), false, true, true)`` = x W^T + b."""

    def __init__(self, w, b=None):
        self.w = w
        self.b = b

    def schedule(self, x):
        b = self.b.cast(x.dt()) if self.b is not None else None
        return self.w.gemm(x, b, False, True, True)


class Embedding:
    """ratchet-nn/src/embedding.rs:15-25: view to 1-D ids, index_select rows, view back."""

    def __init__(self, weight):
        self.weight = weight

    def schedule(self, ids):
        out_shape = list(ids.shape()) + [self.weight.shape()[-1]]
        n = 1
        for s in ids.shape():
            n *= s
        flat = ids.view([n])
        return self.weight.index_select(flat, 0).view(out_shape)


class LayerNorm:
    """ratchet-nn/src/norm.rs:37-43: upcast to f32, normalise, cast back."""

    def __init__(self, weight, bias, eps: float):
        self.weight, self.bias, self.eps = weight, bias, eps

    def schedule(self, x):
        return x.full().layer_norm(self.weight, self.bias, self.eps).cast(x.dt())


class RMSNorm:
    """ratchet-nn/src/norm.rs:63-69."""

    def __init__(self, weight, eps: float):
        self.weight, self.eps = weight, eps

    def schedule(self, x):
        return x.full().rms_norm(self.weight, self.eps).cast(x.dt())


class RotaryEmbedding:
    """ratchet-nn/src/rope.rs:24-45 (half-split pairs; ``traditional`` and ``scale`` are carried but,
    as in the reference, unused by the op)."""

    def __init__(self, dim: int, traditional: bool, base: float, scale: float):
        self.dim, self.traditional, self.base, self.scale = dim, traditional, base, scale

    def schedule(self, x, offset: int):
        return x.rope(self.dim, self.base, offset)


@dataclass
class KVEntry:
    """ratchet-nn/src/kv_cache.rs:4-19."""
    k_cache: object
    v_cache: object
    entries: int = 0


@dataclass
class KVCache:
    """ratchet-nn/src/kv_cache.rs:21-54."""
    layers: List[KVEntry] = field(default_factory=list)

    def __getitem__(self, i: int) -> KVEntry:
        return self.layers[i]

    def update(self, offset: int) -> None:
        for e in self.layers:
            e.entries += offset

    def entries(self, layer: int) -> int:
        return self.layers[layer].entries

    def reset(self) -> None:
        for e in self.layers:
            e.entries = 0


# ---------------------------------------------------------------------------------------- models with a 32-bit residual stream
class StreamNorm:
    """LayerNorm / RMSNorm of an f32 tensor (or of a column window of its rows) into the operand dtype of the matrix product that
    follows."""

    def __init__(self, kind: int, weight, eps: float, dt: int, shift=None):
        self.kind, self.weight, self.eps, self.dt, self.shift = kind, weight, eps, dt, shift

    def schedule(self, x, col: int = 0, gate=None, gate_col: int = 0):
        return x.norm_rows(self.kind, self.weight, self.eps, self.dt, col=col, gate=gate, gate_col=gate_col, shift=self.shift)


class PostNorm:
    """x + LayerNorm(y) * scale + shift for a sublayer output y: x are stream rows, f32 values followed by their copy in the operand
    dtype `dt` (f32: no copy).  A factor per channel behind the norm is folded into scale and shift."""

    def __init__(self, scale, shift, eps: float, dt: int):
        self.scale, self.shift, self.eps, self.dt = scale, shift, eps, dt

    def schedule(self, x, y):
        return x.post_norm(y, self.scale, self.shift, self.eps)

    def operand(self, x):
        """(tensor, first column) of the stream as the operand of a matrix product."""
        return (x, 0) if self.dt == capi.F32 else (x.bitcast(self.dt), 2 * self.scale.shape()[0])


class GatedMLP:
    """x + alpha * W_down (act(W_gate h) * W_up h), gate and up rows stacked in one weight."""

    def __init__(self, gate_up, down, act: str):
        self.gate_up, self.down, self.act = gate_up, down, act

    def schedule(self, h, resid, alpha: float):
        return self.down.linear(self.gate_up.linear(h).glu(self.act), resid=resid, alpha=alpha, dt=capi.F32)


class SquaredReluMLP:
    """W_down max(W_up h, 0)^2 as an f32 sublayer output; h at column `col` of wider rows."""

    def __init__(self, up, down):
        self.up, self.down = up, down

    def schedule(self, h, col: int = 0):
        return self.down.linear(self.up.linear(h, x_col=col, act="relu_squared"), dt=capi.F32)


class RotaryTable:
    """Frequencies of interleaved rotary pairs (plain or YaRN) on the device, and the factor on cos and sin."""

    def __init__(self, freqs, magnitude: float):
        self.freqs, self.magnitude = freqs, magnitude


class SequenceState:
    """What one sequence keeps between steps: per layer run one tensor - a recurrent state f32 [heads, dim, vdim], a ring of
    latents [rows, latent + rotated] or a ring of keys and values [rows, kv_heads * (dim + vdim)] - and the number of tokens seen.  The counterpart of ``KVCache`` for models whose layers
    keep different things."""

    def __init__(self, runs):
        self.runs = runs
        self.position = 0
        self.stack = None                  # the fused decode step bound to these tensors, once one has been made

    def reset(self) -> None:
        """Back to an empty sequence.  Recurrent states start at zero; ring rows are read only once written."""
        for t in self.runs:
            if t.rank() == 3:
                n = 4
                for s in t.shape():
                    n *= s
                t.dev.check(t.dev._lib.rcu_memset(t.dev.handle, t.data_ptr(), 0, n))
        self.position = 0
