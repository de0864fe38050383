"""The callers of the hot path, restated from ratchet-models so the benchmark configurations can be
scheduled through the lazy ``Tensor`` API exactly as the reference schedules them:

* Phi-3 decoder (crates/ratchet-models/src/phi3/{attn,mlp,model}.rs),
* the Phi-2 MLP block inside its parallel-residual layer (phi2/mlp.rs:13-15, phi2/model.rs:78-89),
* the Whisper encoder (whisper/{encoder,residual_block,mha,mlp}.rs);

and two decoders the reference does not have: Dadezen - parallel layers over linear attention and windowed latent
attention, with a loop of layers that runs several times - and Mefesun - norms on the sublayers' outputs, grouped heads
that attend inside chunks of positions, layers that share weights.

They only call ``Tensor`` builder methods, as ``Module::schedule`` does in the reference; no device
code lives here.
"""
from __future__ import annotations

from typing import List, Optional

from . import capi
from .nn import GatedMLP, PostNorm, RotaryTable, SequenceState, SquaredReluMLP, StreamNorm
from .nn import KVCache, KVEntry, LayerNorm, Linear, RMSNorm, RotaryEmbedding, Embedding


# ---------------------------------------------------------------------------------------- Phi-3
class Phi3SelfAttention:
    """phi3/attn.rs:88-159."""

    def __init__(self, qkv: Linear, o: Linear, rope: RotaryEmbedding, n_heads: int, n_kv_heads: int, softmax_scale):
        self.qkv, self.o, self.rope = qkv, o, rope
        self.n_heads, self.n_kv_heads, self.softmax_scale = n_heads, n_kv_heads, softmax_scale

    def schedule(self, x, mask=None, cache: Optional[KVEntry] = None):
        batch, q_len, n_state = x.shape()
        hdim = n_state // self.n_heads
        kv_x_hdim = self.n_kv_heads * hdim
        qkv = self.qkv.schedule(x)
        return self.o.schedule(self.attend(qkv, batch, q_len, n_state, mask, cache))

    def attend(self, qkv, batch, q_len, n_state, mask=None, cache: Optional[KVEntry] = None):
        """Everything between the fused qkv projection and the output projection (attn.rs:95-157)."""
        hdim = n_state // self.n_heads
        kv_x_hdim = self.n_kv_heads * hdim
        query_pos = self.n_heads * hdim
        key_pos = query_pos + kv_x_hdim
        value_pos = key_pos + kv_x_hdim
        q = qkv.slice([(0, batch), (0, q_len), (0, query_pos)])
        k = qkv.slice([(0, batch), (0, q_len), (query_pos, key_pos)])
        v = qkv.slice([(0, batch), (0, q_len), (key_pos, value_pos)])
        q = q.view([batch, q_len, self.n_heads, hdim]).permute([0, 2, 1, 3])
        k = k.view([batch, q_len, self.n_kv_heads, hdim]).permute([0, 2, 1, 3])
        v = v.view([batch, q_len, self.n_kv_heads, hdim]).permute([0, 2, 1, 3])
        offset = cache.entries if cache is not None else 0
        q_dt = q.dt()
        q = self.rope.schedule(q.full(), offset).cast(q_dt)
        k = self.rope.schedule(k.full(), offset).cast(q_dt)
        if cache is not None:
            k = cache.k_cache.cache(k, 2, offset)
            v = cache.v_cache.cache(v, 2, offset)
        attn = q.full().matmul(k.full(), False, True).mul(self.softmax_scale).cast(q_dt)
        if mask is not None:
            attn = attn.add(mask.cast(attn.dt()))
        w = attn.full().softmax(3).cast(v.dt())
        wv = w.matmul(v, False, False).permute([0, 2, 1, 3])
        return wv.view([batch, q_len, n_state])


class Phi3MLP:
    """phi3/mlp.rs:31-39: fused gate_up projection, up * silu(gate), down projection."""

    def __init__(self, up_proj: Linear, down_proj: Linear):
        self.up_proj, self.down_proj = up_proj, down_proj

    def schedule(self, x):
        input_dt = x.dt()
        up_states = self.up_proj.schedule(x)
        a, b, c = up_states.shape()
        gate = up_states.slice([(0, a), (0, b), (0, c // 2)])
        up = up_states.slice([(0, a), (0, b), (c // 2, c)])
        up = up.mul(gate.full().silu().cast(input_dt))
        return self.down_proj.schedule(up)


class Phi3DecoderLayer:
    """phi3/model.rs:103-118."""

    def __init__(self, input_norm: RMSNorm, self_attn: Phi3SelfAttention, ffn_norm: RMSNorm, mlp: Phi3MLP):
        self.input_norm, self.self_attn, self.ffn_norm, self.mlp = input_norm, self_attn, ffn_norm, mlp

    def schedule(self, x, mask=None, cache: Optional[KVEntry] = None):
        residual = x
        xs = self.input_norm.schedule(x)
        attn_output = self.self_attn.schedule(xs, mask, cache)
        xs = residual.add(attn_output)
        residual = xs
        xs = self.ffn_norm.schedule(xs)
        xs = self.mlp.schedule(xs)
        return residual.add(xs)


class Phi3:
    """phi3/model.rs:134-156 (decode only: no mask is generated for seq_len <= 1, as there)."""

    def __init__(self, embedding: Embedding, layers: List[Phi3DecoderLayer], ln_post: RMSNorm, lm_head: Linear, kv_cache: KVCache):
        self.embedding, self.layers, self.ln_post, self.lm_head, self.kv_cache = embedding, layers, ln_post, lm_head, kv_cache

    def schedule(self, ids, mask=None):
        x = self.embedding.schedule(ids)
        _, seq_len, n_state = x.shape()
        for i, layer in enumerate(self.layers):
            x = layer.schedule(x, mask, self.kv_cache[i])
        x = self.ln_post.schedule(x)
        x = x.slice([(0, 1), (seq_len - 1, seq_len), (0, n_state)])
        return self.lm_head.schedule(x)


# ---------------------------------------------------------------------------------------- Phi-2
class Phi2MLPBlock:
    """LayerNorm -> fc1 -> gelu -> fc2 -> + x: the MLP arm of phi2/model.rs:78-89 with phi2/mlp.rs:13-15."""

    def __init__(self, ln: LayerNorm, fc1: Linear, fc2: Linear):
        self.ln, self.fc1, self.fc2 = ln, fc1, fc2

    def schedule(self, x):
        h = self.ln.schedule(x)
        return self.fc2.schedule(self.fc1.schedule(h).gelu()).add(x)


# ---------------------------------------------------------------------------------------- Whisper
class WhisperMHA:
    """whisper/mha.rs:57-127; ``dk`` is the [1] tensor holding head_dim^-0.25."""

    def __init__(self, q: Linear, k: Linear, v: Linear, o: Linear, n_heads: int, dk):
        self.q, self.k, self.v, self.o, self.n_heads, self.dk = q, k, v, o, n_heads, dk

    def schedule(self, x):
        q = self.q.schedule(x)
        k = self.k.schedule(x)
        v = self.v.schedule(x)
        bs, n_ctx, n_state = q.shape()
        q_dt = q.dt()
        hdim = n_state // self.n_heads
        q = q.view([bs, n_ctx, self.n_heads, hdim]).permute([0, 2, 1, 3]).mul(self.dk)
        k = k.view([bs, n_ctx, self.n_heads, hdim]).permute([0, 2, 3, 1]).mul(self.dk)
        v = v.view([bs, n_ctx, self.n_heads, hdim]).permute([0, 2, 1, 3])
        qk = q.matmul(k, False, False).full()
        w = qk.softmax(3).cast(q_dt)
        wv = w.matmul(v, False, False).permute([0, 2, 1, 3]).view([bs, n_ctx, n_state])
        return self.o.schedule(wv)


class WhisperMLP:
    """whisper/mlp.rs:18-22."""

    def __init__(self, l1: Linear, l2: Linear):
        self.l1, self.l2 = l1, l2

    def schedule(self, x):
        return self.l2.schedule(self.l1.schedule(x).full().gelu().cast(x.dt()))


class WhisperBlock:
    """whisper/residual_block.rs:30-51 without cross attention (encoder)."""

    def __init__(self, attn_ln: LayerNorm, attn: WhisperMHA, mlp_ln: LayerNorm, mlp: WhisperMLP):
        self.attn_ln, self.attn, self.mlp_ln, self.mlp = attn_ln, attn, mlp_ln, mlp

    def schedule(self, x):
        attn = x.add(self.attn.schedule(self.attn_ln.schedule(x)))
        return self.mlp.schedule(self.mlp_ln.schedule(attn)).add(attn)


class WhisperEncoder:
    """whisper/encoder.rs:49-55,108-122: conv stem in f32 (conv1d k3 s1 -> gelu -> conv1d k3 s2 -> gelu,
    permute, + positional embedding), cast to the activation dtype, blocks, final LayerNorm."""

    def __init__(self, conv1_w, conv1_b, conv2_w, conv2_b, pos_embed, blocks: List[WhisperBlock], ln_post: LayerNorm, activation_dt: int):
        self.conv1_w, self.conv1_b, self.conv2_w, self.conv2_b = conv1_w, conv1_b, conv2_w, conv2_b
        self.pos_embed, self.blocks, self.ln_post, self.activation_dt = pos_embed, blocks, ln_post, activation_dt

    def schedule(self, mel):
        x = mel.full().conv1d(self.conv1_w, self.conv1_b, 1, 1).gelu()
        x = x.conv1d(self.conv2_w, self.conv2_b, 2, 1).gelu()
        x = x.permute([0, 2, 1]).add(self.pos_embed.full())
        x = x.cast(self.activation_dt)
        for blk in self.blocks:
            x = blk.schedule(x)
        return self.ln_post.schedule(x)


# ---------------------------------------------------------------------------------------- Dadezen
class LightningMixer:
    """Linear attention with a fixed decay per head; the output, RMS-normed over all heads and gated, goes through the output
    projection into the residual stream.  ``proj`` stacks the q, k, v and gate rows; ``decay`` [heads] serves single tokens, its
    powers ``decay_pow`` [heads, n] blocks."""

    def __init__(self, proj, decay, decay_pow, norm: StreamNorm, out, heads: int, dim: int, vdim: int):
        self.proj, self.decay, self.decay_pow, self.norm, self.out = proj, decay, decay_pow, norm, out
        self.heads, self.dim, self.vdim = heads, dim, vdim

    def schedule(self, h, resid, alpha: float, state, position: int):
        qkv = self.heads * (2 * self.dim + self.vdim)
        rows = self.proj.linear(h, act="silu", act_cols=qkv)
        y = self.norm.schedule(rows.lightning(self.decay_pow, state), gate=rows, gate_col=qkv)
        return self.out.linear(y, resid=resid, alpha=alpha, dt=capi.F32)


class LatentMixer:
    """Sliding-window attention whose keys and values are linear images of a cached latent; one rotated key part is shared
    by the heads.  ``low`` stacks the query-latent, latent and rotated-key rows, ``ukv`` the key and value rows."""

    def __init__(self, low, q_norm: StreamNorm, uq, kv_norm: StreamNorm, ukv, rot: RotaryTable, out, heads: int, dim: int, rot_dim: int,
                 vdim: int, window: int, scale: float):
        self.low, self.q_norm, self.uq, self.kv_norm, self.ukv, self.rot, self.out = low, q_norm, uq, kv_norm, ukv, rot, out
        self.heads, self.dim, self.rot_dim, self.vdim, self.window, self.scale = heads, dim, rot_dim, vdim, window, scale

    def schedule(self, h, resid, alpha: float, ring, position: int):
        tokens = h.shape()[0]
        q_rank, kv_rank = self.uq.shape()[1], self.ukv.shape()[1]
        low = self.low.linear(h, dt=capi.F32)
        q = self.uq.linear(self.q_norm.schedule(low)).view([tokens, self.heads, self.dim + self.rot_dim])
        q = q.rotary(self.rot.freqs, self.rot.magnitude, position, first=self.dim)
        rows = tokens + min(position, self.window - 1)
        seen = low.latent_append(self.kv_norm.weight, self.kv_norm.eps, self.rot.freqs, self.rot.magnitude, position, ring, rows, col=q_rank)
        o = q.window_attention(self.ukv.linear(seen), seen, kv_rank, self.vdim, self.window, self.scale)
        return self.out.linear(o, resid=resid, alpha=alpha, dt=capi.F32)


class ParallelLayer:
    """x + alpha * (mixer(norm1 x) + mlp(norm2 x)), both branches from the same x; no mlp: the mixer alone."""

    def __init__(self, norm1: StreamNorm, mixer, norm2: Optional[StreamNorm], mlp: Optional[GatedMLP], alpha: float):
        self.norm1, self.mixer, self.norm2, self.mlp, self.alpha = norm1, mixer, norm2, mlp, alpha

    def schedule(self, x, state, position: int):
        y = self.mixer.schedule(self.norm1.schedule(x), x, self.alpha, state, position)
        return y if self.mlp is None else self.mlp.schedule(self.norm2.schedule(x), y, self.alpha)


class LoopEntry:
    """x <- W [x; x0] + step, before the first layer of a pass."""

    def __init__(self, w, steps: List):
        self.w, self.steps = w, steps

    def schedule(self, x, x0, t: int):
        both = type(x).cat([x.cast(x0.dt()), x0], 1)
        return self.w.linear(both, bias=self.steps[t], dt=capi.F32)


class Dadezen:
    """``runs``: (layer index, pass or None) in execution order; ``first``: the layer a pass begins with."""

    def __init__(self, embedding: Embedding, layers: List[ParallelLayer], runs, first: Optional[int], entry: Optional[LoopEntry],
                 norm: StreamNorm, head):
        self.embedding, self.layers, self.runs, self.first, self.entry, self.norm, self.head = embedding, layers, runs, first, entry, norm, head

    def schedule(self, ids, state: SequenceState, want=None, streams: Optional[list] = None):
        """ids: a block of token ids, following `state.position` earlier ones.  Logits f32 [len(want), vocab] of the places in
        the i32 tensor `want`, or - without one - the residual stream (which still runs every layer)."""
        x0 = self.embedding.schedule(ids)
        x = x0.full()
        for k, (i, t) in enumerate(self.runs):
            if t is not None and i == self.first:
                x = self.entry.schedule(x, x0, t)
            x = self.layers[i].schedule(x, state.runs[k], state.position)
            if streams is not None:
                streams.append(x)
        if want is None:
            return x
        return self.head.linear(self.norm.schedule(x.index_select(want, 0)), dt=capi.F32)


# ---------------------------------------------------------------------------------------- Mefesun
class GroupedMixer:
    """Softmax attention of grouped heads inside chunks of positions (or a window, or over everything), with a norm per head, rotation and
    a sink.  ``qkv`` stacks the query, key and value rows (``qkv_bias`` in the operands' dtype for a block's product, ``qkv_bias_f32``
    for the fused step, which adds it in f32), ``out`` maps to an f32 sublayer output."""

    def __init__(self, qkv, qkv_bias, qkv_bias_f32, q_norm, k_norm, rot: RotaryTable, sink, out, out_bias, eps: float, heads: int, kv_heads: int, dim: int,
                 vdim: int, scale: float, window: int = 0, chunk: int = 0):
        self.qkv, self.qkv_bias, self.qkv_bias_f32, self.q_norm, self.k_norm = qkv, qkv_bias, qkv_bias_f32, q_norm, k_norm
        self.rot, self.sink, self.out, self.out_bias = rot, sink, out, out_bias
        self.eps, self.heads, self.kv_heads, self.dim, self.vdim, self.scale, self.window, self.chunk = eps, heads, kv_heads, dim, vdim, scale, window, chunk

    def seen_before(self, position: int) -> int:
        """Cached positions that a token at `position` sees."""
        if self.chunk:
            return position % self.chunk
        return min(position, self.window - 1) if self.window else position

    def schedule(self, h, col: int, angles, ring, position: int):
        tokens = h.shape()[0]
        rows = self.qkv.linear(h, bias=self.qkv_bias, x_col=col)
        q = rows.norm_rotary(self.heads, self.q_norm, self.eps, angles)
        old = self.seen_before(position)
        keep = min(tokens, self.seen_before(position + tokens))         # rows that later tokens can see
        kv = rows.kv_append(self.kv_heads, self.k_norm, self.eps, angles, position, keep, ring, old + tokens, col=self.heads * self.dim)
        o = q.grouped_attention(kv, self.kv_heads, self.vdim, self.scale, self.sink, self.window, self.chunk, position - old)
        return self.out.linear(o, bias=self.out_bias, dt=capi.F32)


class PostNormLayer:
    """x <- x + norm1(mixer x), x <- x + norm2(mlp x) on stream rows; no mlp: the mixer alone."""

    def __init__(self, norm1: PostNorm, mixer: GroupedMixer, norm2: Optional[PostNorm], mlp: Optional[SquaredReluMLP]):
        self.norm1, self.mixer, self.norm2, self.mlp = norm1, mixer, norm2, mlp

    def schedule(self, x, angles, state, position: int):
        x = self.norm1.schedule(x, self.mixer.schedule(*self.norm1.operand(x), angles, state, position))
        return x if self.mlp is None else self.norm2.schedule(x, self.mlp.schedule(*self.norm2.operand(x)))


class Mefesun:
    """``order``: the layer of every run (layers that share weights appear more than once)."""

    def __init__(self, embedding: Embedding, layers: List[PostNormLayer], order: List[int], norm: StreamNorm, head, dt: int, softcap: Optional[float]):
        self.embedding, self.layers, self.order, self.norm, self.head, self.dt, self.softcap = embedding, layers, order, norm, head, dt, softcap

    def schedule(self, ids, state: SequenceState, want=None, streams: Optional[list] = None):
        """As ``Dadezen.schedule``; ``streams`` receives stream rows (their first `width` columns are the residual stream)."""
        x = self.embedding.schedule(ids).stream_rows(self.dt)
        angles = {}                                  # once per frequency table: every layer turns by the same angles
        for k, i in enumerate(self.order):
            rot = self.layers[i].mixer.rot
            if rot not in angles:
                angles[rot] = rot.freqs.rotary_angles(rot.magnitude, state.position, ids.shape()[0])
            x = self.layers[i].schedule(x, angles[rot], state.runs[k], state.position)
            if streams is not None:
                streams.append(x)
        if want is None:
            return x
        h = self.norm.schedule(x.index_select(want, 0))
        return self.head.linear(h, dt=capi.F32, act="softcap" if self.softcap else None, act_param=self.softcap or 0.0)
