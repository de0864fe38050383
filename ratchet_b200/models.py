"""Models by configuration: config.json names an architecture, the registry maps it to a class that reads the
configuration, loads the weights, makes and resets sequence states, runs blocks of tokens through the lazy graph and single
tokens through the fused decode step.

A served model offers: ``vocab``; ``new_state(max_tokens)``; ``prefill(tokens, state, want)`` -> f32 logits of the wanted places;
``decode(state, token=None)`` -> f32 logits buffer and next-token buffer on the device (token None: the arg-max of the step
before).  Both advance ``state.position``."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import numpy as np

from . import capi
from .callers import Dadezen, GroupedMixer, LatentMixer, LightningMixer, LoopEntry, Mefesun, ParallelLayer, PostNormLayer
from .capi import ERR_INVALID_ARG, ERR_UNSUPPORTED, RatchetCudaError
from .decoder import StackDecoder
from .device import Device
from .nn import Embedding, GatedMLP, PostNorm, RotaryTable, SequenceState, SquaredReluMLP, StreamNorm
from .safetensors import SafetensorsFile
from .tensor import Tensor

DTYPES = {"bfloat16": capi.BF16, "float32": capi.F32}
REGISTRY: Dict[str, type] = {}

CHUNK = 128                   # tokens of a linear-attention chunk: the decay tables hold this many powers


def register(architecture: str):
    def wrap(cls):
        REGISTRY[architecture] = cls
        return cls
    return wrap


def load_model(path: str, dev: Device, dtype: str = "bfloat16"):
    """The model of a folder with config.json and model.safetensors."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    arch = config.get("architecture")
    if arch not in REGISTRY:
        raise RatchetCudaError(ERR_UNSUPPORTED, f"no model class for architecture {arch!r} (known: {', '.join(sorted(REGISTRY))})")
    return REGISTRY[arch](config, SafetensorsFile(os.path.join(path, "model.safetensors")), dev, dtype)


# ---------------------------------------------------------------------------------------- configuration
@dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    factor: float = 0.0       # > 0: YaRN
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    @staticmethod
    def read(c: dict) -> "RotaryConfig":
        s = c.get("scaling")
        if not s:
            return RotaryConfig(int(c["dims"]), float(c["base"]))
        return RotaryConfig(int(c["dims"]), float(c["base"]), float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"]))


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    rot: RotaryConfig
    scale: float
    window: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: object             # LightningConfig or LatentConfig
    mlp: bool


@dataclass(frozen=True)
class DadezenConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float
    layers: Tuple[LayerConfig, ...]
    loop: Optional[Tuple[int, int, int]] = None      # start, stop, times

    @staticmethod
    def read(c: dict) -> "DadezenConfig":
        layers = []
        for i, e in enumerate(c["layers"]):
            m = e["mixer"]
            if e["type"] == "lightning":
                mixer = LightningConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), tuple(float(d) for d in m["decay"]))
                if len(mixer.decay) != mixer.heads:
                    raise RatchetCudaError(ERR_INVALID_ARG, f"layer {i}: {len(mixer.decay)} decays for {mixer.heads} heads")
            elif e["type"] == "latent_attention":
                mixer = LatentConfig(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), RotaryConfig.read(m["rot"]), float(m["scale"]),
                                     int(m["mask"]["size"]))
            else:
                raise RatchetCudaError(ERR_UNSUPPORTED, f"layer {i}: mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise RatchetCudaError(ERR_UNSUPPORTED, f"layer {i}: feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(mixer, bool(mlp)))
        loop = c.get("loop")
        return DadezenConfig(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), float(c["residual_mult"]), tuple(layers),
                             (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass) in execution order; pass is None outside the loop."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        if not 0 <= start < stop <= n or times < 1:
            raise RatchetCudaError(ERR_INVALID_ARG, f"loop {self.loop} over {n} layers")
        return ([(i, None) for i in range(start)] + [(i, t) for t in range(times) for i in range(start, stop)] +
                [(i, None) for i in range(stop, n)])


@dataclass(frozen=True)
class GroupedConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: RotaryConfig
    scale: float
    chunk: int                # 0: every earlier position is seen


@dataclass(frozen=True)
class MefesunConfig:
    width: int
    vocab: int
    eps: float
    softcap: Optional[float]
    layers: Tuple[LayerConfig, ...]
    weights_of: Tuple[int, ...]          # per layer: the layer whose tensors it uses (itself, unless they are shared)

    @staticmethod
    def read(c: dict) -> "MefesunConfig":
        layers, shared = [], []
        for i, e in enumerate(c["layers"]):
            m = e["mixer"]
            if e["type"] != "attention":
                raise RatchetCudaError(ERR_UNSUPPORTED, f"layer {i}: mixer {e['type']!r}")
            mask = m.get("mask")
            mixer = GroupedConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), RotaryConfig.read(m["rot"]), float(m["scale"]),
                                  int(mask["size"]) if mask else 0)
            if mixer.kv_heads < 1 or mixer.heads % mixer.kv_heads or mixer.rot.dims > mixer.dim or mixer.chunk < (1 if mask else 0):
                raise RatchetCudaError(ERR_INVALID_ARG, f"layer {i}: {mixer}")
            mlp = e.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise RatchetCudaError(ERR_UNSUPPORTED, f"layer {i}: feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(mixer, bool(mlp)))
            shared.append(e.get("weights_of"))
        order = []
        for i in range(len(layers)):
            j, steps = i, 0
            while shared[j] is not None:
                j, steps = int(shared[j]), steps + 1
                if not 0 <= j < len(layers) or steps > len(layers):
                    raise RatchetCudaError(ERR_INVALID_ARG, f"layer {i}: weights of layer {j}")
            if layers[j] != layers[i]:
                raise RatchetCudaError(ERR_INVALID_ARG, f"layer {i} uses the weights of layer {j}, whose sizes are others")
            order.append(j)
        cap = c.get("logit_softcap")
        if cap is not None and not float(cap) > 0:
            raise RatchetCudaError(ERR_INVALID_ARG, f"logit_softcap {cap}")
        return MefesunConfig(int(c["width"]), int(c["vocab"]), float(c["norm"]["eps"]), None if cap is None else float(cap), tuple(layers), tuple(order))


# ---------------------------------------------------------------------------------------- models
class _Weights:
    """Device tensors from a safetensors file: matrices in the model's dtype, rows of several matrices stacked into one;
    vectors (norm scales, biases) in f32."""

    def __init__(self, file: SafetensorsFile, dev: Device, dt: int):
        self.file, self.dev, self.dt = file, dev, dt

    def matrix(self, *names: str) -> Tensor:
        cols = {self.file.shape(n)[1:] for n in names}
        if any(len(self.file.shape(n)) != 2 for n in names) or len(cols) != 1:
            raise RatchetCudaError(ERR_INVALID_ARG, f"{', '.join(names)}: matrices of one width expected")
        parts = []
        for n in names:
            kind, raw = self.file.raw(n)
            if self.dt == capi.BF16:
                parts.append(raw if kind == "BF16" else capi.to_bf16(self.file.f32(n)))
            else:
                parts.append(self.file.f32(n))
        return Tensor.from_data(parts[0] if len(parts) == 1 else np.concatenate(parts), device=self.dev, dt=self.dt)

    def vector(self, *names: str, dt: int = capi.F32) -> Tensor:
        v = np.concatenate([self.file.f32(n).reshape(-1) for n in names])
        return Tensor.from_data(capi.to_bf16(v), device=self.dev, dt=dt) if dt == capi.BF16 else self.const(v)

    def const(self, a: np.ndarray) -> Tensor:
        return Tensor.from_data(np.ascontiguousarray(a, np.float32), device=self.dev)


class DecoderModel:
    """What the served decoders share: ``graph`` (a caller with ``schedule(ids, state, want, streams)``) runs blocks of tokens,
    ``_stack(state)`` makes the fused step over a state's tensors, which runs single ones."""

    def __init__(self, cfg, dev: Device, dtype: str):
        if dtype not in DTYPES:
            raise RatchetCudaError(ERR_UNSUPPORTED, f"dtype {dtype!r} (bfloat16 or float32)")
        self.dev, self.dt, self.cfg, self.vocab = dev, DTYPES[dtype], cfg, cfg.vocab

    @staticmethod
    def _check(file: SafetensorsFile, name: str, shape) -> None:
        if file.shape(name) != tuple(shape):
            raise RatchetCudaError(ERR_INVALID_ARG, f"{name} is {file.shape(name)}, expected {tuple(shape)}")

    def prefill(self, tokens: Sequence[int], state: SequenceState, want: Sequence[int] = (), streams: Optional[list] = None) -> np.ndarray:
        ids = Tensor.from_data(np.asarray(tokens, np.int32), device=self.dev)
        places = Tensor.from_data(np.asarray(want, np.int32), device=self.dev) if len(want) else None
        out = self.graph.schedule(ids, state, places, streams).resolve()
        state.position += len(tokens)
        return out.to_numpy() if places is not None else np.empty((0, self.vocab), np.float32)

    def decode(self, state: SequenceState, token: Optional[int] = None):
        if state.stack is None:
            state.stack = self._stack(state)
        state.stack.position = state.position
        if token is None:
            state.stack.step_device()
        else:
            state.stack.step(token)
        state.position += 1
        return state.stack.logits, state.stack.token


@register("Dadezen")
class DadezenModel(DecoderModel):
    def __init__(self, config: dict, file: SafetensorsFile, dev: Device, dtype: str = "bfloat16"):
        super().__init__(DadezenConfig.read(config), dev, dtype)
        c, w = self.cfg, _Weights(file, dev, self.dt)
        self._check(file, "embed", (c.vocab, c.width))
        self._check(file, "head", (c.vocab, c.width))
        layers = [self._layer(w, i, lc) for i, lc in enumerate(c.layers)]
        entry, self._steps = None, []
        if c.loop:
            self._check(file, "loop.step", (c.loop[2], c.width))
            self._check(file, "loop.in", (c.width, 2 * c.width))
            self._steps = [w.const(v) for v in file.f32("loop.step")]
            entry = LoopEntry(w.matrix("loop.in"), self._steps)
        norm = StreamNorm(capi.LAYER_NORM, w.vector("final.norm"), c.eps, self.dt)
        self.graph = Dadezen(Embedding(w.matrix("embed")), layers, c.runs(), c.loop[0] if c.loop else None, entry, norm, w.matrix("head"))

    def _layer(self, w: _Weights, i: int, lc: LayerConfig) -> ParallelLayer:
        c, m, p, f = self.cfg, lc.mixer, f"l{i}.", w.file
        norm = lambda kind, name: StreamNorm(kind, w.vector(name), c.eps, self.dt)
        x = p + "mix."
        if isinstance(m, LightningConfig):
            H, D, E = m.heads, m.dim, m.vdim
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                self._check(f, x + n, (rows, c.width))
            self._check(f, x + "o", (c.width, H * E))
            powers = np.power(np.array(m.decay, np.float64)[:, None], np.arange(CHUNK + 1)[None, :])
            mixer = LightningMixer(w.matrix(x + "q", x + "k", x + "v", x + "g"), w.const(np.array(m.decay)), w.const(powers),
                                   norm(capi.RMS_NORM, x + "norm"), w.matrix(x + "o"), H, D, E)
        else:
            H, D, R, E = m.heads, m.dim, m.rot_dim, m.vdim
            q_rank, kv_rank = f.shape(x + "dq")[0], f.shape(x + "dkv.norm")[0]
            self._check(f, x + "dkv", (kv_rank + R, c.width))
            self._check(f, x + "uq", (H * (D + R), q_rank))
            self._check(f, x + "uk", (H * D, kv_rank))
            self._check(f, x + "uv", (H * E, kv_rank))
            self._check(f, x + "o", (c.width, H * E))
            r = m.rot
            if r.dims > R:
                raise RatchetCudaError(ERR_INVALID_ARG, f"layer {i}: {r.dims} rotated of {R} features")
            table, magnitude = capi.rotary_frequencies(r.dims, r.base, r.factor, r.original, r.fast, r.slow)
            mixer = LatentMixer(w.matrix(x + "dq", x + "dkv"), norm(capi.RMS_NORM, x + "dq.norm"), w.matrix(x + "uq"), norm(capi.RMS_NORM, x + "dkv.norm"),
                                w.matrix(x + "uk", x + "uv"), RotaryTable(w.const(table), magnitude), w.matrix(x + "o"), H, D, R, E, m.window, m.scale)
        norm2 = mlp = None
        if lc.mlp:
            ff = f.shape(p + "mlp.gate")[0]
            self._check(f, p + "mlp.up", (ff, c.width))
            self._check(f, p + "mlp.down", (c.width, ff))
            norm2, mlp = norm(capi.LAYER_NORM, p + "norm2"), GatedMLP(w.matrix(p + "mlp.gate", p + "mlp.up"), w.matrix(p + "mlp.down"), "gelu")
        return ParallelLayer(norm(capi.LAYER_NORM, p + "norm1"), mixer, norm2, mlp, c.residual_mult)

    # ------------------------------------------------------------------ sequence state
    def new_state(self, max_tokens: Optional[int] = None) -> SequenceState:
        """State tensors of one sequence of at most `max_tokens` tokens.  A latent ring holds the window (no more than the
        sequence), whatever the length of the prompt."""
        tensors = []
        for i, _ in self.graph.runs:
            m = self.cfg.layers[i].mixer
            if isinstance(m, LightningConfig):
                tensors.append(Tensor.zeros((m.heads, m.dim, m.vdim), capi.F32, self.dev))
            else:
                rows = m.window if max_tokens is None else min(m.window, max_tokens)
                mixer = self.graph.layers[i].mixer
                tensors.append(Tensor.zeros((rows, mixer.ukv.shape()[1] + m.rot_dim), self.dt, self.dev))
        return SequenceState(tensors)

    # ------------------------------------------------------------------ single tokens
    def _stack(self, state: SequenceState) -> StackDecoder:
        c, g = self.cfg, self.graph
        runs = []
        for k, (i, t) in enumerate(g.runs):
            m, layer = c.layers[i].mixer, g.layers[i]
            r = capi.rcu_stack_run()
            mx = layer.mixer
            r.heads, r.dim, r.vdim = m.heads, m.dim, m.vdim
            r.norm1, r.out, r.mix_norm, r.state = layer.norm1.weight.data_ptr(), mx.out.data_ptr(), 0, state.runs[k].data_ptr()
            if layer.mlp is not None:
                r.ff = layer.mlp.down.shape()[1]
                r.norm2, r.gate_up, r.down = layer.norm2.weight.data_ptr(), layer.mlp.gate_up.data_ptr(), layer.mlp.down.data_ptr()
            if isinstance(m, LightningConfig):
                r.mixer, r.mix_in, r.mix_norm, r.decay = capi.MIXER_LIGHTNING, mx.proj.data_ptr(), mx.norm.weight.data_ptr(), mx.decay.data_ptr()
            else:
                r.mixer, r.mix_in, r.mix_norm, r.kv_norm = capi.MIXER_LATENT, mx.low.data_ptr(), mx.q_norm.weight.data_ptr(), mx.kv_norm.weight.data_ptr()
                r.q_rank, r.kv_rank, r.rot_dim, r.rot_pairs = mx.uq.shape()[1], mx.ukv.shape()[1], m.rot_dim, m.rot.dims // 2
                r.window, r.ring_rows, r.scale, r.rot_magnitude = m.window, state.runs[k].shape()[0], m.scale, mx.rot.magnitude
                r.uq, r.ukv, r.freqs = mx.uq.data_ptr(), mx.ukv.data_ptr(), mx.rot.freqs.data_ptr()
            if t is not None and i == g.first:
                r.enter, r.enter_bias = g.entry.w.data_ptr(), self._steps[t].data_ptr()
            runs.append(r)
        cfg = capi.rcu_stack_config(c.width, c.vocab, len(runs), c.eps, c.residual_mult, 0.0, self.dt, capi.LAYER_PARALLEL, None)
        return StackDecoder(self.dev, cfg, runs, g.embedding.weight.data_ptr(), g.norm.weight.data_ptr(), g.head.data_ptr(), (g, state.runs))


@register("Mefesun")
class MefesunModel(DecoderModel):
    def __init__(self, config: dict, file: SafetensorsFile, dev: Device, dtype: str = "bfloat16"):
        super().__init__(MefesunConfig.read(config), dev, dtype)
        c, w = self.cfg, _Weights(file, dev, self.dt)
        self._check(file, "embed", (c.vocab, c.width))
        self._rotary: Dict[RotaryConfig, RotaryTable] = {}
        layers = [self._layer(w, i, lc) if c.weights_of[i] == i else None for i, lc in enumerate(c.layers)]
        embed = w.matrix("embed")
        norm = StreamNorm(capi.LAYER_NORM, w.vector("final.norm"), c.eps, self.dt, shift=w.vector("final.norm.b"))
        self.graph = Mefesun(Embedding(embed), layers, list(c.weights_of), norm, embed, self.dt, c.softcap)

    def _rot(self, w: _Weights, r: RotaryConfig) -> RotaryTable:
        if r not in self._rotary:
            table, magnitude = capi.rotary_frequencies(r.dims, r.base, r.factor, r.original, r.fast, r.slow)
            self._rotary[r] = RotaryTable(w.const(table), magnitude)
        return self._rotary[r]

    def _layer(self, w: _Weights, i: int, lc: LayerConfig) -> PostNormLayer:
        c, m, p, f = self.cfg, lc.mixer, f"l{i}.", w.file
        H, G, D, E = m.heads, m.kv_heads, m.dim, m.vdim
        x = p + "mix."
        for n, rows in (("q", H * D), ("k", G * D), ("v", G * E)):
            self._check(f, x + n, (rows, c.width))
            self._check(f, x + n + ".b", (rows,))
        for n, shape in (("o", (c.width, H * E)), ("o.b", (c.width,)), ("q.norm", (D,)), ("k.norm", (D,)), ("sink", (H,))):
            self._check(f, x + n, shape)

        def norm(k: str) -> PostNorm:
            for n in (f"norm{k}", f"norm{k}.b", f"ls{k}"):
                self._check(f, p + n, (c.width,))
            ls = f.f32(f"{p}ls{k}")
            return PostNorm(w.const(f.f32(f"{p}norm{k}") * ls), w.const(f.f32(f"{p}norm{k}.b") * ls), c.eps, self.dt)

        biases = (x + "q.b", x + "k.b", x + "v.b")
        mixer = GroupedMixer(w.matrix(x + "q", x + "k", x + "v"), w.vector(*biases, dt=self.dt), w.vector(*biases), w.vector(x + "q.norm"), w.vector(x + "k.norm"),
                             self._rot(w, m.rot), w.vector(x + "sink"), w.matrix(x + "o"), w.vector(x + "o.b"), c.eps, H, G, D, E, m.scale, chunk=m.chunk)
        norm2 = mlp = None
        if lc.mlp:
            ff = f.shape(p + "mlp.up")[0]
            self._check(f, p + "mlp.up", (ff, c.width))
            self._check(f, p + "mlp.down", (c.width, ff))
            norm2, mlp = norm("2"), SquaredReluMLP(w.matrix(p + "mlp.up"), w.matrix(p + "mlp.down"))
        return PostNormLayer(norm("1"), mixer, norm2, mlp)

    def new_state(self, max_tokens: Optional[int] = None) -> SequenceState:
        """A ring of keys and values per layer run: the chunk's positions, no more than the sequence's."""
        tensors = []
        for lc in self.cfg.layers:
            m = lc.mixer
            sizes = [n for n in (m.chunk, max_tokens) if n]
            if not sizes:
                raise RatchetCudaError(ERR_INVALID_ARG, "a layer that sees every position needs the most tokens a sequence may hold")
            tensors.append(Tensor.zeros((min(sizes), m.kv_heads * (m.dim + m.vdim)), self.dt, self.dev))
        return SequenceState(tensors)

    def _stack(self, state: SequenceState) -> StackDecoder:
        c, g = self.cfg, self.graph
        runs = []
        for k, i in enumerate(g.order):
            layer, r = g.layers[i], capi.rcu_stack_run()
            mx = layer.mixer
            r.mixer, r.heads, r.kv_heads, r.dim, r.vdim = capi.MIXER_GROUPED, mx.heads, mx.kv_heads, mx.dim, mx.vdim
            r.rot_pairs, r.rot_magnitude, r.freqs = mx.rot.freqs.shape()[1], mx.rot.magnitude, mx.rot.freqs.data_ptr()
            r.window, r.chunk, r.scale, r.ring_rows, r.state = mx.window, mx.chunk, mx.scale, state.runs[k].shape()[0], state.runs[k].data_ptr()
            r.mix_in, r.mix_bias, r.mix_norm, r.kv_norm = mx.qkv.data_ptr(), mx.qkv_bias_f32.data_ptr(), mx.q_norm.data_ptr(), mx.k_norm.data_ptr()
            r.sink, r.out, r.out_bias = mx.sink.data_ptr(), mx.out.data_ptr(), mx.out_bias.data_ptr()
            r.norm1, r.norm1_shift = layer.norm1.scale.data_ptr(), layer.norm1.shift.data_ptr()
            if layer.mlp is not None:
                r.ff = layer.mlp.down.shape()[1]
                r.norm2, r.norm2_shift = layer.norm2.scale.data_ptr(), layer.norm2.shift.data_ptr()
                r.gate_up, r.down = layer.mlp.up.data_ptr(), layer.mlp.down.data_ptr()
            runs.append(r)
        cfg = capi.rcu_stack_config(c.width, c.vocab, len(runs), c.eps, 0.0, c.softcap or 0.0, self.dt, capi.LAYER_POST_NORM, g.norm.shift.data_ptr())
        return StackDecoder(self.dev, cfg, runs, g.embedding.weight.data_ptr(), g.norm.weight.data_ptr(), g.head.data_ptr(), (g, state.runs))
