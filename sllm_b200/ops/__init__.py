"""The operations a step is made of, each a hand-written sm_100a kernel.

Tensors must lie on a CUDA device and be contiguous; there is no CPU path and no
library model code behind these functions.  Matrix products of the bfloat16
path with many rows go to cuBLAS (as the reference's engine does,
kernels/cuda/kernels.cu:752-767); everything else, and every product of the
float32 path, runs in this package's own kernels.
"""

from __future__ import annotations

import functools
import os

import torch

from ._lib import KernelError, KernelTimes, call, launches, lib  # noqa: F401

F32, BF16 = 0, 1


def _dt(t: torch.Tensor) -> int:
    if t.dtype == torch.float32:
        return F32
    if t.dtype == torch.bfloat16:
        return BF16
    raise KernelError(f"unsupported dtype {t.dtype}; the kernels take float32 and bfloat16")


def _dtc(dtype: torch.dtype) -> int:
    if dtype == torch.float32:
        return F32
    if dtype == torch.bfloat16:
        return BF16
    raise KernelError(f"unsupported dtype {dtype}; the kernels take float32 and bfloat16")


def _chk(*tensors) -> None:
    for t in tensors:
        if t is not None and not (t.is_cuda and t.is_contiguous()):
            if not t.is_cuda:
                raise KernelError("the kernels run on a CUDA device only; got a tensor on " + str(t.device))
            raise KernelError("the kernels take contiguous tensors")


def _p(t):
    return None if t is None else t.data_ptr()


# the raw handle of the current stream: torch's quick accessor where this torch has it (the public
# `current_stream()` builds a Stream object, several microseconds a launch)
_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


_current_device = getattr(torch._C, "_cuda_getDevice", None)      # (torch.cuda.current_device() checks initialisation each time)


def _stream():
    if _raw_stream is not None:
        return _raw_stream(_current_device() if _current_device is not None else torch.cuda.current_device())
    return torch.cuda.current_stream().cuda_stream


def embed_gather(table: torch.Tensor, ids: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    """float32 ``[T, H]`` rows of ``table`` (``[V, H]``) at int32 ``ids``, times ``scale``."""
    _chk(table, ids)
    T, (V, H) = ids.numel(), table.shape
    out = torch.empty((T, H), dtype=torch.float32, device=table.device)
    call("sllm_embed_gather", _p(table), _dt(table), _p(ids), _p(out), T, H, V, float(scale), _stream())
    return out


# ---- a stream of several copies ------------------------------------------------------------------------

MAX_STREAMS = 16


def embed_streams(table, step, scale: float, copies, pair_table=None, before=None, pairs=None) -> torch.Tensor:
    """float32 ``[T, copies, H]`` (``[T, H]`` where ``copies`` is None), every copy the row of ``table`` at the step's token ids times
    ``scale``; with ``pairs`` (`config.plan.TokenPairs`) plus the row of ``pair_table`` ``[buckets + 1, H]`` that the token and the
    one before it name (the last row at position 0).  The token before a portion's first is the request's row of ``before`` (float32
    ``[slots, 1]``), which then receives the portion's last token."""
    _chk(table, pair_table, before, step.token_ids)
    T, (V, H) = step.token_ids.numel(), table.shape
    if pairs is not None and (pair_table is None or tuple(pair_table.shape) != (pairs.buckets + 1, H) or pair_table.dtype != table.dtype or
                              before is None or before.dtype != torch.float32):
        raise KernelError("embed_streams: pairs of tokens need their table [buckets + 1, H] and the tokens before, float32 [slots, 1]")
    out = torch.empty((T, H) if copies is None else (T, int(copies), H), dtype=torch.float32, device=table.device)
    call("sllm_embed_streams", _p(table), _dt(table), _p(step.token_ids), _p(out), T, H, V, float(scale), int(copies or 1), _p(pair_table),
         *((int(pairs.buckets), int(pairs.mul_prev), int(pairs.mul_cur)) if pairs is not None else (0, 0, 0)), _p(step.positions),
         _p(step.seq_of_token), _p(step.q_start), _p(step.state_slots), _p(before), _stream())
    return out


def streams_step(streams, term, mix, share, into, gain, eps: float, out_dtype, rows=None):
    """One sublayer's border in a stream of several copies ``[T, s, W]`` (float32): with ``term`` (float32 ``[T, W]`` or a stack of
    partial sums), every new stream r = sum over the old s of ``mix[s, r]`` times stream s, plus ``share[r]`` times the term, in place;
    then the RMS norm (``gain`` float32 ``[W]``) of sum over s of ``into[s]`` times stream s, in ``out_dtype`` (``gain`` None: no
    norm, nothing returned).  ``rows`` (int32): only these rows are computed, ``[len(rows), W]``, and no stream is written."""
    _chk(streams, term, mix, share, into, gain, rows)
    T, s, W = streams.shape
    if streams.dtype != torch.float32 or (term is not None and (tuple(term.shape[-2:]) != (T, W) or tuple(mix.shape) != (s, s) or share.numel() != s)) or \
            (gain is not None and (gain.numel() != W or into.numel() != s)):
        raise KernelError("streams_step: float32 streams [T, s, W], a term that fits them, s x s and s weights")
    R = T if rows is None else rows.numel()
    h = torch.empty((R, W), dtype=out_dtype, device=streams.device) if gain is not None else None
    call("sllm_streams_step", _p(streams), *_term(term), _p(mix), _p(share), _p(into), _p(gain), float(eps), _p(rows), _p(h),
         _dtc(out_dtype) if h is not None else F32, R, T, s, W, _stream())
    return h


# ---- a stream with sinusoidal positions, a norm in groups, a token shift ----------------------------

def add_sinusoid_(stream: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """``stream[t, 2i] += sin(p_t f_i)``, ``stream[t, 2i+1] += cos(p_t f_i)`` in place; the angle is a float32 product."""
    _chk(stream, positions, inv_freq)
    T, W = stream.shape
    if stream.dtype != torch.float32 or inv_freq.dtype != torch.float32 or inv_freq.numel() != W // 2:
        raise KernelError("add_sinusoid_: a float32 stream of even width and width/2 float32 frequencies")
    call("sllm_add_sinusoid", _p(stream), _p(positions), _p(inv_freq), T, W, _stream())
    return stream


def _term(t):
    """(pointer, parts, stride) of a pending term: float32 ``[T, W]`` or a stack of partial sums ``[parts, T, W]``."""
    if t is None:
        return None, 0, 0
    if t.dtype != torch.float32:
        raise KernelError("a pending term of the stream is float32")
    return (_p(t), t.shape[0], t.shape[1] * t.shape[2]) if t.dim() == 3 else (_p(t), 1, 0)


def add_group_ssq(stream: torch.Tensor, terms, groups: int, eps: float, want_rinv: bool = True):
    """Add up to two pending ``terms`` into the float32 ``stream`` in place and return, per row and group of
    ``width / groups`` consecutive channels, ``1 / sqrt(mean square + eps)`` as float32 ``[T, groups]`` (None if
    not wanted: a plain addition)."""
    terms = [t for t in (terms or ()) if t is not None]
    if len(terms) > 2:
        raise KernelError("add_group_ssq: at most two pending terms")
    _chk(stream, *terms)
    T, W = stream.shape
    if stream.dtype != torch.float32:
        raise KernelError("add_group_ssq: the stream is float32")
    for t in terms:
        if tuple(t.shape[-2:]) != (T, W):
            raise KernelError(f"add_group_ssq: a term {tuple(t.shape)} does not fit the stream {(T, W)}")
    rinv = torch.empty((T, groups), dtype=torch.float32, device=stream.device) if want_rinv else None
    d0 = _term(terms[0] if terms else None)
    d1 = _term(terms[1] if len(terms) > 1 else None)
    call("sllm_add_group_ssq", _p(stream), *d0, *d1, _p(rinv), T, W, int(groups), float(eps), _stream())
    return rinv


def group_norm_shift(stream, rinv, gain, out_dtype, *, groups: int | None = None, eps: float = 0.0, mix=None, state=None,
                     step=None, want_plain: bool = True):
    """The norm in groups applied: ``h = stream * rinv[group] * gain`` in ``out_dtype``; with ``rinv`` None the kernel
    takes the reciprocal roots itself (``groups``, ``eps``), so a stream with nothing pending needs one kernel.  With
    ``mix``: also the mixer's input ``hs = h + (h_prev - h) * mix``, ``h_prev`` the same request's row before (for the
    first token of its portion, the request's row of ``state`` ``[slots, W]``, which then receives the portion's last
    ``h``).  Returns ``h``, or ``(h, hs)`` (``h`` None if not wanted)."""
    _chk(stream, rinv, gain, mix, state)
    T, W = stream.shape
    groups = int(rinv.shape[1] if rinv is not None else groups)
    h = torch.empty((T, W), dtype=out_dtype, device=stream.device) if (want_plain or mix is None) else None
    if mix is None:
        call("sllm_group_norm_shift", _p(stream), _p(rinv), _p(gain), None, None, None, None, None, _p(h), None,
             _dtc(out_dtype), T, W, groups, float(eps), _stream())
        return h
    hs = torch.empty((T, W), dtype=out_dtype, device=stream.device)
    call("sllm_group_norm_shift", _p(stream), _p(rinv), _p(gain), _p(mix), _p(state), _p(step.seq_of_token), _p(step.q_start),
         _p(step.state_slots), _p(h), _p(hs), _dtc(out_dtype), T, W, groups, float(eps), _stream())
    return h, hs


ACTIVATIONS = {"silu": 0, "gelu_tanh": 1}


def act_mul(gu: torch.Tensor, interleave: int, out_dtype: torch.dtype, act: str) -> torch.Tensor:
    """``act(gate) * up`` of ``gu [T, 2I]`` whose columns alternate between gate and up in blocks of
    ``interleave`` (``interleave == I``: all gates, then all ups); ``act`` is ``silu`` or ``gelu_tanh``."""
    _chk(gu)
    T, two_i = gu.shape
    I = two_i // 2
    out = torch.empty((T, I), dtype=out_dtype, device=gu.device)
    call("sllm_act_mul", _p(gu), _dt(gu), _p(out), _dtc(out_dtype), T, I, int(interleave), ACTIVATIONS[act], _stream())
    return out


def linear_act_mul(x, w_gate_up, bias, interleave: int, out_dtype, act: str) -> torch.Tensor:
    """``act(x Wg^T + bg) * (x Wu^T + bu)`` with gate and up rows (and biases) alternating in one matrix in blocks of
    ``interleave``.  SiLU without biases: `linear_silu_mul`'s kernels.  The tanh form of GELU, bfloat16, blocks of 8: the
    activation leaves with the product's tile (up to 32 tokens the streaming kernel, prompt portions the CTA-pair
    product).  Otherwise the product with its bias, then `act_mul`."""
    if act == "silu" and bias is None:
        return linear_silu_mul(x, w_gate_up, interleave, out_dtype)
    if (act == "gelu_tanh" and interleave == 8 and x.is_cuda and x.dtype == torch.bfloat16 and out_dtype == torch.bfloat16
            and w_gate_up.shape[0] % 16 == 0 and _GATED_FUSED):
        M, K = x.shape
        N = w_gate_up.shape[0]
        if stream_supports(M, N, K):
            return linear_stream(x, w_gate_up, bias, out_dtype, act=act)
        if M > TCGEN05_MIN_ROWS and _PAIR_GEMM != "off" and pair_supports(M, N, K):
            return gemm_pair(x, w_gate_up, bias, out_dtype, act=act)
    return act_mul(linear(x, w_gate_up, bias, x.dtype), interleave, out_dtype, act)


_GATED_FUSED = os.environ.get("SLLM_GATED_FUSED", "1") != "0"      # 0: the product, then the activation kernel


def tanh_cols(x: torch.Tensor, col0: int, n: int, out_dtype: torch.dtype) -> torch.Tensor:
    """``tanh(x[:, col0:col0+n])`` of a float32 product, in ``out_dtype``."""
    _chk(x)
    T, ld = x.shape
    if x.dtype != torch.float32:
        raise KernelError("tanh_cols: a float32 product")
    out = torch.empty((T, n), dtype=out_dtype, device=x.device)
    call("sllm_tanh_cols", _p(x), ld, int(col0), int(n), _p(out), _dtc(out_dtype), T, _stream())
    return out


# ---- the generalized delta rule -----------------------------------------------------------------------

def delta_rule_supports(dk: int, dv: int) -> bool:
    return 1 <= dk <= 256 and dv >= 1


def delta_rule(proj, offs, decay, a_bias, state, step, heads: int, dk: int, dv: int) -> torch.Tensor:
    """The recurrence over the step's tokens, request by request in token order, from and into the
    requests' rows of ``state`` (float32 ``[slots, heads, dk, dv]``).  ``proj`` is a float32 product ``[T, ld]``
    whose columns ``offs = (r, k, v, a)`` hold receptance, key, value and removal logits; ``decay`` float32
    ``[T, heads*dk]`` holds decay logits; ``a_bias`` float32 ``[heads*dk]``.  Returns ``o`` float32 ``[T, heads*dv]``."""
    _chk(proj, decay, a_bias, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or decay.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("delta_rule: everything that enters the recurrence is float32")
    if tuple(decay.shape) != (T, heads * dk) or tuple(state.shape[1:]) != (heads, dk, dv):
        raise KernelError(f"delta_rule: decay {tuple(decay.shape)} or state {tuple(state.shape)} does not fit {heads} heads of {dk}x{dv}")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=proj.device)
    off_r, off_k, off_v, off_a = (int(o) for o in offs)
    call("sllm_delta_rule", _p(proj), ld, off_r, off_k, off_v, off_a, _p(decay), _p(a_bias), _p(state), _p(step.q_start),
         _p(step.state_slots), _p(out), step.num_seqs, heads, dk, dv, int(step.max_q_len), _stream())
    return out


GATE_ACTS = {"sigmoid": 0, "silu": 1, "none": 2}


def delta_out(o, gain, proj, off_g: int, eps: float, heads: int, dv: int, out_dtype, gate_act: str = "sigmoid", out=None,
              out_off: int = 0, step=None, max_len: int = 0) -> torch.Tensor:
    """Each head's ``o`` over its root mean square, times ``gain`` (``[heads*dv]``; None: ones), times ``sigmoid`` (or ``silu``) of
    the gate logits (columns ``off_g`` of ``proj``), in ``out_dtype``; with ``gate_act`` ``none`` there is no gate and
    ``proj`` may be None.  ``out``: a wider tensor whose columns ``out_off ..`` receive the result.  ``max_len`` > 0 (with ``step``):
    rows of requests that bring more tokens are left alone."""
    if gate_act == "none":
        proj, off_g = o, 0
    _chk(o, gain, proj, out)
    T = o.shape[0]
    if out is None:
        out = torch.empty((T, heads * dv), dtype=out_dtype, device=o.device)
    call("sllm_delta_out", _p(o), _p(gain), _p(proj), proj.shape[1], int(off_g), float(eps), _p(out), _dtc(out.dtype), T, heads, dv,
         GATE_ACTS[gate_act], out.shape[1], int(out_off), _p(step.seq_of_token) if max_len else None, _p(step.q_start) if max_len else None,
         int(max_len), _stream())
    return out


def forget_gate_attention(proj, offs, f_bias, lower, state, step, heads: int, dk: int, dv: int) -> torch.Tensor:
    """S <- diag(f) S + (1 - f) v^T; o = S^T silu(q) with f = lower + (1 - lower) sigmoid(z + f_bias) per key channel, over the
    step's tokens from and into ``state`` (float32 ``[slots, heads, dk, dv]``).  ``proj`` float32 ``[T, ld]`` holds q, the
    gate's logits z and v at columns ``offs``; ``f_bias`` and ``lower`` float32 ``[heads*dk]``.  Returns ``o`` float32
    ``[T, heads*dv]``."""
    _chk(proj, f_bias, lower, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or state.dtype != torch.float32 or f_bias.dtype != torch.float32 or lower.dtype != torch.float32:
        raise KernelError("forget_gate_attention: everything that enters the recurrence is float32")
    if tuple(state.shape[1:]) != (heads, dk, dv) or f_bias.numel() != heads * dk or lower.numel() != heads * dk:
        raise KernelError(f"forget_gate_attention: state {tuple(state.shape)} or the gate's vectors do not fit {heads} heads of {dk}x{dv}")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=proj.device)
    off_q, off_f, off_v = (int(o) for o in offs)
    call("sllm_forget_gate_attention", _p(proj), ld, off_q, off_f, off_v, _p(f_bias), _p(lower), _p(state), _p(step.q_start),
         _p(step.state_slots), _p(out), step.num_seqs, heads, dk, dv, int(step.max_q_len), _stream())
    return out


def add_rows_(stream, rows, vec) -> None:
    """``stream += rows + vec`` in place: ``rows`` float32 ``[T, W]`` or None, ``vec`` float32 ``[W]`` or None."""
    _chk(stream, rows, vec)
    T, W = stream.shape
    if stream.dtype != torch.float32 or (rows is not None and (rows.dtype != torch.float32 or tuple(rows.shape) != (T, W))) or \
            (vec is not None and (vec.dtype != torch.float32 or vec.numel() != W)):
        raise KernelError("add_rows_: the stream, the rows and the vector are float32 of the stream's width")
    call("sllm_add_rows", _p(stream), _p(rows), _p(vec), T, W, _stream())


def norm_pair(stream, gain_a, gain_b, eps: float, out_dtype):
    """Two RMS norms of the same float32 rows: ``(x / rms(x) * gain_a, x / rms(x) * gain_b)`` in ``out_dtype`` (the second
    None when ``gain_b`` is None)."""
    _chk(stream, gain_a, gain_b)
    T, W = stream.shape
    if stream.dtype != torch.float32 or gain_a.dtype != torch.float32 or (gain_b is not None and gain_b.dtype != torch.float32):
        raise KernelError("norm_pair: the stream and the gains are float32")
    a = torch.empty((T, W), dtype=out_dtype, device=stream.device)
    b = torch.empty((T, W), dtype=out_dtype, device=stream.device) if gain_b is not None else None
    call("sllm_norm_pair", _p(stream), _p(gain_a), _p(gain_b), float(eps), _p(a), _p(b), _dtc(out_dtype), T, W, _stream())
    return a, b


def gated_delta_rule(qkv, offs, gates, off_b: int, off_dt: int, a_log, dt_bias, state, step, heads: int, key_heads: int,
                     dk: int, dv: int, q_scale: float) -> torch.Tensor:
    """The gated delta rule over the step's tokens, request by request in token order, from and into the requests' rows
    of ``state`` (float32 ``[slots, heads, dk, dv]``): S <- g S; w = beta (v - S^T k); S <- S + k w^T; o = S^T q, with k
    and q made unit vectors per head here (q also times ``q_scale``), beta = sigmoid(b) and g = exp(-exp(A) softplus(a +
    dt)) one number per head.  ``qkv`` float32 ``[T, ld]`` holds q, k (``key_heads`` heads of ``dk``) and v (``heads`` of
    ``dv``) at columns ``offs``; ``gates`` float32 ``[T, ldg]`` the logits b and a at columns ``off_b + h``, ``off_dt + h``.
    Returns ``o`` float32 ``[T, heads*dv]``."""
    _chk(qkv, gates, a_log, dt_bias, state)
    T, ld = qkv.shape
    if qkv.dtype != torch.float32 or gates.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("gated_delta_rule: everything that enters the recurrence is float32")
    if tuple(state.shape[1:]) != (heads, dk, dv):
        raise KernelError(f"gated_delta_rule: state {tuple(state.shape)} does not fit {heads} heads of {dk}x{dv}")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=qkv.device)
    off_q, off_k, off_v = (int(o) for o in offs)
    call("sllm_gated_delta_rule", _p(qkv), ld, off_q, off_k, off_v, _p(gates), gates.shape[1], int(off_b), int(off_dt), _p(a_log),
         _p(dt_bias), _p(state), _p(step.q_start), _p(step.state_slots), _p(out), step.num_seqs, heads, key_heads, dk, dv,
         float(q_scale), int(step.max_q_len), _stream())
    return out


def gated_linear_attention(proj, offs, z, state, step, heads: int, dk: int, dv: int, q_scale: float, tau: float) -> torch.Tensor:
    """S <- diag(alpha) S + k v^T; o = S^T (q * q_scale) with alpha = sigmoid(z)^(1/tau) per key channel, over the step's
    tokens from and into ``state`` (float32 ``[slots, heads, dk, dv]``).  ``proj`` float32 ``[T, ld]`` holds q, k, v at
    columns ``offs``; ``z`` float32 ``[T, heads*dk]``.  Returns ``o`` float32 ``[T, heads*dv]``."""
    _chk(proj, z, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or z.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("gated_linear_attention: everything that enters the recurrence is float32")
    if tuple(z.shape) != (T, heads * dk) or tuple(state.shape[1:]) != (heads, dk, dv):
        raise KernelError(f"gated_linear_attention: z {tuple(z.shape)} or state {tuple(state.shape)} does not fit {heads} heads of {dk}x{dv}")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=proj.device)
    off_q, off_k, off_v = (int(o) for o in offs)
    call("sllm_gated_linear_attention", _p(proj), ld, off_q, off_k, off_v, _p(z), _p(state), _p(step.q_start), _p(step.state_slots),
         _p(out), step.num_seqs, heads, dk, dv, float(q_scale), 1.0 / float(tau), int(step.max_q_len), _stream())
    return out


# ---- two mixers side by side: normed, rotated attention heads; short convolutions; the normed mean ---------------

def qk_norm_rope_kv_write(qkv, q_gain, k_gain, eps: float, positions, table, rotary_dim: int, nq: int, nkv: int, dim: int,
                          vdim: int, slot_mapping, k_cache, v_cache, out_dtype, q_mul=None, col_off: int = 0) -> torch.Tensor:
    """From a float32 product ``[T, (nq+nkv)*dim + nkv*vdim]``: every query and key head over its root mean square times
    its gain (``[dim]``, shared by the heads), then rotated; values as they are.  The queries come back ``[T, nq*D]`` in
    ``out_dtype`` with D the cache's head size (>= dim and vdim; zeros beyond); keys and values go to ``slot_mapping`` in
    the pages (not written when ``slot_mapping`` is None: the product may then end behind the queries' columns).  With both gains None the heads are not normed; ``q_mul``
    (float32 ``[nq]``) multiplies each query head.  ``col_off``: the column of ``qkv`` at which q|k|v start (a product that
    holds other projections too)."""
    _chk(qkv, q_gain, k_gain, q_mul, positions, table, slot_mapping, k_cache, v_cache)
    T, ld = qkv.shape
    num_pages, nkv_c, page_size, D = k_cache.shape
    if qkv.dtype != torch.float32 or nkv_c != nkv or k_cache.dtype != out_dtype or tuple(v_cache.shape) != tuple(k_cache.shape):
        raise KernelError("qk_norm_rope_kv_write: a float32 product and a cache of the compute dtype [pages, nkv, page_size, D]")
    max_pos = 0
    if rotary_dim:
        if table is None or table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rotary_dim // 2):
            raise KernelError("qk_norm_rope_kv_write: rotary table must be float32 [positions, 2, rotary_dim/2]")
        max_pos = table.shape[0]
    q = torch.empty((T, nq * D), dtype=out_dtype, device=qkv.device)
    if col_off < 0 or col_off + nq * dim + (nkv * (dim + vdim) if slot_mapping is not None else 0) > ld:
        raise KernelError("qk_norm_rope_kv_write: q|k|v lie outside the product's columns")
    call("sllm_qk_norm_rope_kv_write", _p(qkv) + 4 * int(col_off), ld, _p(q_gain), _p(k_gain), _p(q_mul), float(eps), _p(positions), _p(table), int(rotary_dim),
         max_pos, nq, nkv, dim, vdim, D, _p(slot_mapping), page_size, num_pages, _p(k_cache), _p(v_cache), _p(q),
         _dtc(out_dtype), T, _stream())
    return q


def whole_norm_kv_write(qkv, bias, q_gain, k_gain, eps: float, positions, q_temp, nq: int, nkv: int, dim: int, vdim: int, slot_mapping,
                        k_cache, v_cache, out_dtype) -> torch.Tensor:
    """From a float32 product ``[T, nq*dim (+ nkv*(dim + vdim))]`` (or a stack of partial sums) plus ``bias``: all query rows over
    their common root mean square times ``q_gain`` ``[nq*dim]``, times 1 + coef ln(floor((p + 1) / every) + 1) with ``q_temp`` =
    (coef, every) (None: 1); the key rows likewise with ``k_gain`` ``[nkv*dim]``; values as they are.  The queries come back ``[T,
    nq*D]`` in ``out_dtype`` with D the cache's head size (zeros beyond dim); keys and values go to ``slot_mapping`` in the pages (None: the
    product holds queries alone)."""
    _chk(qkv, bias, q_gain, k_gain, positions, slot_mapping, k_cache, v_cache)
    T, ld = qkv.shape[-2:]
    num_pages, nkv_c, page_size, D = k_cache.shape
    want = nq * dim + (nkv * (dim + vdim) if slot_mapping is not None else 0)
    if nkv_c != nkv or k_cache.dtype != out_dtype or tuple(v_cache.shape) != tuple(k_cache.shape) or ld < want or \
            (bias is not None and bias.numel() != ld) or q_gain.numel() != nq * dim or (slot_mapping is not None and k_gain.numel() != nkv * dim):
        raise KernelError(f"whole_norm_kv_write: a product of {want} columns, gains of the projections' sizes and a cache of the compute dtype")
    q = torch.empty((T, nq * D), dtype=out_dtype, device=qkv.device)
    coef, every = q_temp if q_temp is not None else (0.0, 1)
    call("sllm_whole_norm_kv_write", *_term(qkv), ld, _p(bias), _p(q_gain), _p(k_gain), float(eps), _p(positions), float(coef), int(every), nq, nkv,
         dim, vdim, D, _p(slot_mapping), page_size, num_pages, _p(k_cache), _p(v_cache), _p(q), _dtc(out_dtype), T, _stream())
    return q


def norm_cols(x, off: int, n: int, gain, eps: float, out_dtype) -> torch.Tensor:
    """Columns ``off .. off+n`` of a float32 product over their root mean square, times ``gain``, in ``out_dtype``."""
    _chk(x, gain)
    T, ld = x.shape
    if x.dtype != torch.float32 or gain.dtype != torch.float32 or gain.numel() != n:
        raise KernelError("norm_cols: a float32 product and a float32 gain of as many values as columns")
    out = torch.empty((T, n), dtype=out_dtype, device=x.device)
    call("sllm_norm_cols", _p(x), ld, int(off), int(n), _p(gain), float(eps), _p(out), _dtc(out_dtype), T, _stream())
    return out


def short_conv_add(x, weight, state, step, out_dtype) -> torch.Tensor:
    """``x + conv(x)``: the float32 rows ``x [T, C]`` plus their causal convolution over time per channel (``weight`` float32
    ``[C, taps]``, the current token's tap last; the inputs before a request's portion from its row of ``state`` ``[slots, C,
    taps-1]``, which then receives the portion's last ones), in ``out_dtype``."""
    _chk(x, weight, state)
    T, C = x.shape
    taps = weight.shape[1]
    if x.dtype != torch.float32 or weight.dtype != torch.float32 or tuple(weight.shape) != (C, taps) or \
            (taps > 1 and tuple(state.shape[1:]) != (C, taps - 1)):
        raise KernelError("short_conv_add: float32 input and taps [C, taps], and a state [slots, C, taps-1]")
    out = torch.empty((T, C), dtype=out_dtype, device=x.device)
    call("sllm_short_conv", _p(x), C, 0, _p(weight), None, taps, _p(state) if taps > 1 else None, _p(step.seq_of_token), _p(step.q_start),
         _p(step.state_slots), _p(out), _dtc(out_dtype), 1, T, step.num_seqs, C, _stream())
    if taps > 1:
        launches["own"] += 1          # the state's kernel
    return out


def short_conv_silu(x, off: int, weight, state, step, bias=None) -> torch.Tensor:
    """``silu`` of a causal convolution over time (plus ``bias`` float32 ``[C]``), per channel, of columns ``off .. off+C`` of the float32 product ``x``:
    ``weight`` float32 ``[C, taps]`` with the current token's tap last; the ``taps - 1`` inputs before a request's portion
    come from its row of ``state`` (float32 ``[slots, C, taps-1]``, zeros at a sequence's start), which then receives the
    portion's last ones.  float32 ``[T, C]``."""
    _chk(x, weight, state, bias)
    T, ld = x.shape
    C, taps = weight.shape
    if x.dtype != torch.float32 or weight.dtype != torch.float32 or (taps > 1 and tuple(state.shape[1:]) != (C, taps - 1)) or \
            (bias is not None and (bias.dtype != torch.float32 or bias.numel() != C)):
        raise KernelError("short_conv_silu: float32 input, taps and bias, and a state [slots, C, taps-1]")
    out = torch.empty((T, C), dtype=torch.float32, device=x.device)
    call("sllm_short_conv_silu", _p(x), ld, int(off), _p(weight), _p(bias), taps, _p(state) if taps > 1 else None, _p(step.seq_of_token),
         _p(step.q_start), _p(step.state_slots), _p(out), T, step.num_seqs, C, _stream())
    if taps > 1:
        launches["own"] += 1          # the state's kernel
    return out


def norm_mean_add_(stream, a, gain_a, b, gain_b, eps: float) -> None:
    """``stream += (a / rms(a) * gain_a + b / rms(b) * gain_b) / 2`` row by row, all float32."""
    _chk(stream, a, gain_a, b, gain_b)
    T, W = stream.shape
    if any(t.dtype != torch.float32 for t in (stream, a, b, gain_a, gain_b)) or tuple(a.shape) != (T, W) or tuple(b.shape) != (T, W):
        raise KernelError("norm_mean_add_: float32 [T, W] terms for a float32 stream")
    call("sllm_norm_mean_add", _p(stream), _p(a), _p(gain_a), _p(b), _p(gain_b), float(eps), T, W, _stream())


# ---- a mixture of experts ----------------------------------------------------------------------------------

def moe_route(logits, correction, groups: int, keep: int, top: int, scale: float):
    """The router's choice from float32 logits ``[T, E]``: (dense weights float32 ``[T, E]`` with zeros for the experts not
    chosen, indices int32 ``[T, top]``, weights float32 ``[T, top]``).  Scores are sigmoids; the choice goes by score +
    ``correction`` within the ``keep`` best of ``groups`` groups (a group's score: its two largest choice scores);
    the weights are the chosen scores times ``scale``."""
    _chk(logits, correction)
    T, E = logits.shape
    if logits.dtype != torch.float32:
        raise KernelError("moe_route: the router's logits are float32")
    dense = torch.empty((T, E), dtype=torch.float32, device=logits.device)
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    wts = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    call("sllm_moe_route", _p(logits), _p(correction), T, E, int(groups), int(keep), int(top), float(scale), _p(dense), _p(idx),
         _p(wts), _stream())
    return dense, idx, wts


def moe_act(up, dense, ff: int, out_dtype) -> torch.Tensor:
    """``gelu(up) * weight`` for the routed experts' columns (expert e's at ``e*ff``, weight ``dense[t, e]``) and
    ``gelu(up)`` for the columns after them; the exact gelu, float32 arithmetic, ``out_dtype`` out."""
    _chk(up, dense)
    T, N = up.shape
    E = dense.shape[1]
    out = torch.empty((T, N), dtype=out_dtype, device=up.device)
    call("sllm_moe_act", _p(up), _dt(up), _p(dense), _p(out), _dtc(out_dtype), T, N, E, int(ff), _stream())
    return out


def moe_route_top_softmax(logits, top: int, scale: float = 1.0, experts: "int | None" = None, gated: int = 0):
    """The ``top`` largest of the float32 router logits ``[T, E]`` win (the lower index on a tie); their weights are the
    softmax over the winners alone, times ``scale``.  (dense weights float32 ``[T, E]`` with zeros elsewhere, indices int32 ``[T, top]`` by
    falling logit, weights float32 ``[T, top]``).  ``experts``: only so many of the logits' columns are experts; ``gated`` (0 or 1):
    the column behind them is the logit of an expert every token uses, and the dense weights ``[T, E + gated]`` end with its sigmoid."""
    _chk(logits)
    T, ld = logits.shape
    E = int(experts or ld)
    if gated not in (0, 1) or E + gated > ld:
        raise KernelError(f"moe_route_top_softmax: {E} experts and {gated} gate columns in rows of {ld} logits")
    if logits.dtype != torch.float32:
        raise KernelError("moe_route_top_softmax: the router's logits are float32")
    dense = torch.empty((T, E + gated), dtype=torch.float32, device=logits.device)
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    wts = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    call("sllm_moe_route_top_softmax", _p(logits), ld, T, E, int(gated), int(top), float(scale), _p(dense), _p(idx), _p(wts), _stream())
    return dense, idx, wts


def gated_clamp_act(gu, interleave: int, limit: float, out_dtype, *, alpha: float = 1.702, dense=None, ff: int | None = None,
                    act: str = "clamped_swish", tail: int = 0):
    """``g' sigmoid(alpha g') (u' + 1)`` with ``g' = min(g, limit)`` and ``u' = clamp(u, -limit, limit)`` of ``gu [T, 2N]``
    whose columns alternate between gate and up in blocks of ``interleave``.  With ``dense`` (float32 ``[T, E]``, the
    routing weights of E experts of ``ff`` columns each, N = E ff): also times the token's weight of the column's expert;
    the columns of an expert a token does not use are not read.  ``act`` ``silu``: ``g sigmoid(g) u`` instead (``limit`` and
    ``alpha`` unused).  ``tail``: so many columns behind the experts' belong to one more expert, with the last of the weights."""
    _chk(gu, dense)
    T, two_n = gu.shape
    N = two_n // 2
    E = dense.shape[1] if dense is not None else 0
    out = torch.empty((T, N), dtype=out_dtype, device=gu.device)
    call("sllm_gated_clamp_act", _p(gu), _dt(gu), _p(dense), _p(out), _dtc(out_dtype), T, N, E, int(ff if dense is not None else N), int(tail),
         int(interleave), float(limit), float(alpha), {"clamped_swish": 0, "silu": 1}[act], _stream())
    return out


# ---- sublayers between two norms; an element-wise gated recurrence ---------------------------------------------------

def post_add_norm(stream, term, post_gain, post_eps: float, pre_gain, pre_eps: float, out_dtype=torch.float32):
    """``stream += term / rms(term) * post_gain`` (skipped when ``term`` is None; ``term`` float32 ``[T, W]`` or a stack of
    partial sums ``[parts, T, W]``), then ``stream / rms(stream) * pre_gain`` in ``out_dtype`` (None when ``pre_gain`` is
    None).  Gains float32 ``[W]``; everything float32."""
    _chk(stream, term, post_gain, pre_gain)
    T, W = stream.shape
    if stream.dtype != torch.float32 or (term is not None and tuple(term.shape[-2:]) != (T, W)):
        raise KernelError("post_add_norm: a float32 stream [T, W] and a term that fits it")
    h = torch.empty((T, W), dtype=out_dtype, device=stream.device) if pre_gain is not None else None
    call("sllm_post_add_norm", _p(stream), *_term(term), _p(post_gain), float(post_eps), _p(pre_gain), float(pre_eps), _p(h),
         _dtc(out_dtype), T, W, _stream())
    return h


def post_add_copy(stream, term, post_gain, post_eps: float, out_dtype=None):
    """``stream += term / rms(term) * post_gain`` (skipped when ``term`` is None), for a reader that takes the stream as it is:
    returns the stream in ``out_dtype`` (the stream itself where that is float32, None where ``out_dtype`` is None)."""
    _chk(stream, term, post_gain)
    T, W = stream.shape
    if stream.dtype != torch.float32 or (term is not None and tuple(term.shape[-2:]) != (T, W)):
        raise KernelError("post_add_copy: a float32 stream [T, W] and a term that fits it")
    h = None
    if out_dtype is not None and out_dtype != torch.float32:
        h = torch.empty((T, W), dtype=out_dtype, device=stream.device)
    if term is not None or h is not None:
        call("sllm_post_add_norm", _p(stream), *_term(term), _p(post_gain), float(post_eps), None, 0.0, _p(h),
             _dtc(out_dtype) if h is not None else F32, T, W, _stream())
    return stream if out_dtype == torch.float32 else h


def softcap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(x / cap)`` in place on a float32 tensor."""
    _chk(x)
    if x.dtype != torch.float32:
        raise KernelError("softcap_: float32 values")
    call("sllm_softcap", _p(x), x.numel(), float(cap), _stream())
    return x


def post_add_norm_conv(stream, term, post_gain, post_eps: float, pre_gain, pre_eps: float, weight, state, step, out_dtype):
    """`post_add_norm` and `short_conv_add` of its result in one launch, for a step in which every request brings ONE token:
    the normed row stays in the CTA, ``out = h + conv(h)`` reads the request's row of ``state`` (float32 ``[slots, W, taps-1]``)
    and moves it on.  ``weight`` float32 ``[W, taps]``.  Returns ``out`` ``[T, W]`` in ``out_dtype``."""
    _chk(stream, term, post_gain, pre_gain, weight, state)
    T, W = stream.shape
    taps = weight.shape[1]
    if T != step.num_seqs:
        raise KernelError(f"post_add_norm_conv: {T} tokens of {step.num_seqs} requests; this form takes one token a request")
    if stream.dtype != torch.float32 or (term is not None and tuple(term.shape[-2:]) != (T, W)) or weight.dtype != torch.float32 or \
            tuple(weight.shape) != (W, taps) or (taps > 1 and (state.dtype != torch.float32 or tuple(state.shape[1:]) != (W, taps - 1))):
        raise KernelError("post_add_norm_conv: a float32 stream [T, W], a term that fits it, taps [W, taps] and a state [slots, W, taps-1]")
    out = torch.empty((T, W), dtype=out_dtype, device=stream.device)
    call("sllm_post_add_norm_conv", _p(stream), *_term(term), _p(post_gain), float(post_eps), _p(pre_gain), float(pre_eps), _p(weight),
         taps, _p(state) if taps > 1 else None, _p(step.seq_of_token), _p(step.state_slots), _p(out), _dtc(out_dtype), T, W, _stream())
    return out


def mingru_scan(proj, offs, state, step, width: int, out_dtype) -> torch.Tensor:
    """``S <- (1 - z) S + z c`` element by element over the step's tokens, request by request in token order, from and into
    ``state`` (float32 ``[slots, width]``), with z = sigmoid(a), c = b + 1/2 where b >= 0 and sigmoid(b) elsewhere, read out
    as ``S * silu(g)``; a, b, g are the float32 columns ``offs = (a, b, g)`` of ``proj [T, ld]``.  ``[T, width]``."""
    _chk(proj, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or state.dtype != torch.float32 or tuple(state.shape[1:]) != (width,):
        raise KernelError("mingru_scan: a float32 product and a state [slots, width]")
    out = torch.empty((T, width), dtype=out_dtype, device=proj.device)
    oz, ox, og = (int(o) for o in offs)
    call("sllm_mingru_scan", _p(proj), ld, oz, ox, og, _p(state), _p(step.q_start), _p(step.state_slots), _p(out), _dtc(out_dtype),
         T, step.num_seqs, int(width), _stream())
    return out


def decay_linear_attention(proj, offs, decay, state, step, heads: int, dk: int, dv: int) -> torch.Tensor:
    """S <- decay_h S + k v^T; o = S^T q with q, k, v each through silu, over the step's tokens from and into ``state``
    (float32 ``[slots, heads, dk, dv]``).  ``proj`` float32 ``[T, ld]`` holds q, k, v at columns ``offs``; ``decay`` float32
    ``[heads]``.  Returns ``o`` float32 ``[T, heads*dv]``."""
    _chk(proj, decay, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or decay.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("decay_linear_attention: everything that enters the recurrence is float32")
    if tuple(decay.shape) != (heads,) or tuple(state.shape[1:]) != (heads, dk, dv):
        raise KernelError(f"decay_linear_attention: decay {tuple(decay.shape)} or state {tuple(state.shape)} does not fit {heads} heads of {dk}x{dv}")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=proj.device)
    off_q, off_k, off_v = (int(o) for o in offs)
    call("sllm_decay_linear_attention", _p(proj), ld, off_q, off_k, off_v, _p(decay), _p(state), _p(step.q_start),
         _p(step.state_slots), _p(out), step.num_seqs, heads, dk, dv, int(step.max_q_len), _stream())
    return out


def retention(proj, offs, decay, table, rotary_dim: int, k_scale: float, state, step, heads: int, dk: int, dv: int,
              max_len: int = 0) -> torch.Tensor:
    """S <- decay_h S + k v^T; o = S^T q over the step's tokens from and into ``state`` (float32 ``[slots, heads, dk, dv]``), with
    q and k rotated by position over their first ``rotary_dim`` channels (channel i with i + rotary_dim/2; ``table`` float32
    ``[positions, 2, rotary_dim/2]``, None: no rotation) and k then times ``k_scale``.  ``proj`` float32 ``[T, ld]`` holds q, k, v
    at columns ``offs``; ``decay`` float32 ``[heads]``.  Returns ``o`` float32 ``[T, heads*dv]``.  ``max_len`` > 0: requests that bring
    more tokens are left alone (neither their states nor their rows are touched)."""
    _chk(proj, decay, table, state)
    T, ld = proj.shape
    if proj.dtype != torch.float32 or decay.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("retention: everything that enters the recurrence is float32")
    if tuple(decay.shape) != (heads,) or tuple(state.shape[1:]) != (heads, dk, dv):
        raise KernelError(f"retention: decay {tuple(decay.shape)} or state {tuple(state.shape)} does not fit {heads} heads of {dk}x{dv}")
    rot = int(rotary_dim) if table is not None else 0
    if rot and (table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rot // 2)):
        raise KernelError("retention: rotary table must be float32 [positions, 2, rotary_dim/2]")
    out = torch.empty((T, heads * dv), dtype=torch.float32, device=proj.device)
    off_q, off_k, off_v = (int(o) for o in offs)
    call("sllm_retention", _p(proj), ld, off_q, off_k, off_v, _p(decay), _p(step.positions), _p(table), rot, table.shape[0] if rot else 0,
         float(k_scale), _p(state), _p(step.q_start), _p(step.state_slots), _p(out), step.num_seqs, heads, dk, dv, int(step.max_q_len),
         int(max_len), _stream())
    return out


RETENTION_CHUNK = 64           # tokens per chunk of the chunked form (its kernels')
# Portions of at least so many tokens take it (0: none does).  In a graph, one portion at 32 heads of 64 x 64, us: 64 tokens 19 token by
# token and 25 in chunks, 128 tokens 31 and 26, 2,048 tokens 525 and 81.
RETENTION_CHUNKED_FROM = int(os.environ.get("SLLM_RETENTION_CHUNKED_FROM", "96"))


@functools.lru_cache(maxsize=4096)
def retention_chunked_supports(dk: int, dv: int) -> bool:
    return bool(lib().sllm_retention_chunked_supports(int(dk), int(dv)))


def portion_chunks(q_lens, ctx_lens, min_len: int, device):
    """The step's long portions cut into chunks of `RETENTION_CHUNK` tokens: (first tokens, their positions, lengths, chunks; requests,
    their first chunk, how many, requests) on the device, or None where no portion has ``min_len`` tokens."""
    t0, pos, n, seq, first, count = [], [], [], [], [], []
    start = 0
    for s, (q, ctx) in enumerate(zip(q_lens, ctx_lens)):
        if q >= min_len:
            seq.append(s)
            first.append(len(t0))
            for a in range(0, q, RETENTION_CHUNK):
                t0.append(start + a)
                pos.append(ctx - q + a)
                n.append(min(RETENTION_CHUNK, q - a))
            count.append(len(t0) - first[-1])
        start += q
    if not seq:
        return None
    t = torch.tensor(t0 + pos + n + seq + first + count, dtype=torch.int32).to(device, non_blocking=True)
    C, R = len(t0), len(seq)
    o = 3 * C
    return t[:C], t[C:2 * C], t[2 * C:o], C, t[o:o + R], t[o + R:o + 2 * R], t[o + 2 * R:], R


def retention_chunked(proj, offs, off_g: int, decay, table, rotary_dim: int, k_scale: float, eps: float, state, step, chunks, heads: int,
                      dk: int, dv: int, out) -> None:
    """Retention, the heads' norm and the silu gate (columns ``off_g`` of ``proj``) for the requests that ``chunks`` (see
    `portion_chunks`) cuts, a chunk of tokens at a time; their rows of ``out`` ``[T, heads*dv]`` and their states are written, others
    left alone."""
    _chk(proj, decay, table, state, out)
    if proj.dtype != torch.float32 or decay.dtype != torch.float32 or state.dtype != torch.float32:
        raise KernelError("retention_chunked: everything that enters the recurrence is float32")
    if tuple(decay.shape) != (heads,) or tuple(state.shape[1:]) != (heads, dk, dv) or tuple(out.shape) != (proj.shape[0], heads * dv):
        raise KernelError(f"retention_chunked: decay {tuple(decay.shape)}, state {tuple(state.shape)} or output {tuple(out.shape)} does not fit "
                          f"{heads} heads of {dk}x{dv}")
    rot = int(rotary_dim) if table is not None else 0
    if rot and (table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rot // 2)):
        raise KernelError("retention_chunked: rotary table must be float32 [positions, 2, rotary_dim/2]")
    t0, pos, n, C, seq, first, count, R = chunks
    scratch = torch.empty((C, heads, dk, dv), dtype=torch.float32, device=proj.device)
    off_q, off_k, off_v = (int(o) for o in offs)
    call("sllm_retention_chunked", _p(proj), proj.shape[1], off_q, off_k, off_v, int(off_g), _p(decay), _p(table), rot,
         table.shape[0] if rot else 0, float(k_scale), float(eps), _p(state), _p(step.state_slots), _p(t0), _p(pos), _p(n), C, _p(seq), _p(first),
         _p(count), R, _p(scratch), _p(out), _dtc(out.dtype), out.shape[1], heads, dk, dv, _stream())
    launches["own"] += 2           # the three kernels of the entry point


def retention_gated(proj, offs, off_g: int, decay, table, rotary_dim: int, k_scale: float, eps: float, state, step, heads: int, dk: int,
                    dv: int, out_dtype) -> torch.Tensor:
    """`retention` and what follows it in a layer: each head's output over its root mean square, times silu of columns ``off_g`` of
    ``proj``, ``[T, heads*dv]`` in ``out_dtype``.  Long prompt portions run in chunks (heads of up to 128 x 128), single tokens and short
    portions token by token; a step may hold both."""
    chunks, longest = None, 0
    if RETENTION_CHUNKED_FROM > 0 and step.max_q_len >= RETENTION_CHUNKED_FROM and step.q_lens and retention_chunked_supports(dk, dv):
        if "retention" not in step.attn_tiles:
            step.attn_tiles["retention"] = portion_chunks(step.q_lens, step.ctx_lens, RETENTION_CHUNKED_FROM, proj.device)
        chunks, longest = step.attn_tiles["retention"], RETENTION_CHUNKED_FROM - 1
    if chunks is None:
        o = retention(proj, offs, decay, table, rotary_dim, k_scale, state, step, heads, dk, dv)
        return delta_out(o, None, proj, off_g, eps, heads, dv, out_dtype, "silu")
    out = torch.empty((proj.shape[0], heads * dv), dtype=out_dtype, device=proj.device)
    retention_chunked(proj, offs, off_g, decay, table, rotary_dim, k_scale, eps, state, step, chunks, heads, dk, dv, out)
    if chunks[7] < step.num_seqs:
        o = retention(proj, offs, decay, table, rotary_dim, k_scale, state, step, heads, dk, dv, max_len=longest)
        delta_out(o, None, proj, off_g, eps, heads, dv, out_dtype, "silu", out=out, step=step, max_len=longest)
    return out


# ---- a state-space recurrence: one decay per token and head ------------------------------------------------

# Portions of at least so many tokens run in chunks (0: none does), shorter ones token by token.  In a graph, one portion at 64 heads of 128 x 64,
# us: 64 tokens 20 token by token and 34 in chunks, 128 tokens 36 and 35, 256 tokens 68 and 45, 2,048 tokens 520 and 199; four of 512: 304 and 225.
STATE_SPACE_CHUNKED_FROM = int(os.environ.get("SLLM_STATE_SPACE_CHUNKED_FROM", "128"))


@functools.lru_cache(maxsize=4096)
def state_space_chunked_supports(n: int, dv: int) -> bool:
    return bool(lib().sllm_state_space_chunked_supports(int(n), int(dv)))


def _state_space_args(xbc, proj, off_dt, dt_bias, a_log, skip, state, heads, groups, n, dv, what):
    _chk(xbc, proj, dt_bias, a_log, skip, state)
    if any(t.dtype != torch.float32 for t in (xbc, proj, dt_bias, a_log, skip, state)):
        raise KernelError(f"{what}: everything that enters the recurrence is float32")
    if tuple(state.shape[1:]) != (heads, n, dv) or xbc.shape[1] != heads * dv + 2 * groups * n or heads % groups or off_dt + heads > proj.shape[1]:
        raise KernelError(f"{what}: state {tuple(state.shape)} or inputs {tuple(xbc.shape)} do not fit {heads} heads of {n}x{dv} in {groups} groups")


def state_space_walk(xbc, proj, off_dt: int, dt_bias, a_log, skip, state, step, heads: int, groups: int, n: int, dv: int, max_len: int = 0, out=None):
    """`state_space` token by token.  ``max_len`` > 0: requests that bring more tokens are left alone (neither their states nor
    their rows of ``out`` are touched)."""
    _state_space_args(xbc, proj, off_dt, dt_bias, a_log, skip, state, heads, groups, n, dv, "state_space")
    if out is None:
        out = torch.empty((xbc.shape[0], heads * dv), dtype=torch.float32, device=xbc.device)
    call("sllm_state_space", _p(xbc), xbc.shape[1], _p(proj), proj.shape[1], int(off_dt), _p(dt_bias), _p(a_log), _p(skip), _p(state),
         _p(step.q_start), _p(step.state_slots), _p(out), step.num_seqs, heads, groups, n, dv, int(step.max_q_len), int(max_len), _stream())
    return out


def state_space_chunked(xbc, proj, off_dt: int, dt_bias, a_log, skip, state, step, chunks, heads: int, groups: int, n: int, dv: int, out) -> None:
    """`state_space` for the requests that ``chunks`` (see `portion_chunks`) cuts, a chunk of tokens at a time; their rows of ``out`` and
    their states are written, others left alone."""
    _state_space_args(xbc, proj, off_dt, dt_bias, a_log, skip, state, heads, groups, n, dv, "state_space_chunked")
    t0, _, count, C, seq, first, runs, R = chunks
    scratch = torch.empty((C, heads, n, dv), dtype=torch.float32, device=xbc.device)
    keeps = torch.empty((C, heads), dtype=torch.float32, device=xbc.device)
    scores = torch.empty((C, groups, RETENTION_CHUNK, RETENTION_CHUNK), dtype=torch.float32, device=xbc.device)
    call("sllm_state_space_chunked", _p(xbc), xbc.shape[1], _p(proj), proj.shape[1], int(off_dt), _p(dt_bias), _p(a_log), _p(skip), _p(state),
         _p(step.state_slots), _p(t0), _p(count), C, _p(seq), _p(first), _p(runs), R, _p(scratch), _p(scores), _p(keeps), _p(out), heads, groups, n, dv, _stream())
    launches["own"] += 2           # the three kernels of the entry point


@functools.lru_cache(maxsize=4096)
def state_space_token_supports(n: int, dv: int) -> bool:
    return bool(lib().sllm_state_space_token_supports(int(n), int(dv)))


def state_space_token(xbc, proj, off_dt: int, dt_bias, a_log, skip, state, step, heads: int, groups: int, n: int, dv: int) -> torch.Tensor:
    """`state_space` for a step in which every request brings ONE token: the states stream through registers once."""
    _state_space_args(xbc, proj, off_dt, dt_bias, a_log, skip, state, heads, groups, n, dv, "state_space_token")
    if xbc.shape[0] != step.num_seqs:
        raise KernelError(f"state_space_token: {xbc.shape[0]} tokens of {step.num_seqs} requests; this form takes one token a request")
    out = torch.empty((xbc.shape[0], heads * dv), dtype=torch.float32, device=xbc.device)
    call("sllm_state_space_token", _p(xbc), xbc.shape[1], _p(proj), proj.shape[1], int(off_dt), _p(dt_bias), _p(a_log), _p(skip), _p(state),
         _p(step.state_slots), _p(out), step.num_seqs, heads, groups, n, dv, _stream())
    return out


def state_space(xbc, proj, off_dt: int, dt_bias, a_log, skip, state, step, heads: int, groups: int, n: int, dv: int) -> torch.Tensor:
    """The state-space recurrence over the step's tokens, request by request in token order, from and into the requests' rows of
    ``state`` (float32 ``[slots, heads, n, dv]``): S <- exp(-exp(a_log_h) dt) S + dt B x^T; y = S^T C + skip_h x, with dt = softplus of
    column ``off_dt + h`` of the float32 product ``proj`` plus ``dt_bias[h]``.  ``xbc`` float32 ``[T, heads*dv + 2*groups*n]`` holds x (head
    by head), B and C (group by group; head h uses group h // (heads / groups)).  Returns y float32 ``[T, heads*dv]``.  Long prompt
    portions run in chunks (states of up to 128 x 128), short ones and single tokens beside them token by token; where every request
    brings one token a form of its own streams the states."""
    if xbc.shape[0] == step.num_seqs and state_space_token_supports(n, dv):
        return state_space_token(xbc, proj, off_dt, dt_bias, a_log, skip, state, step, heads, groups, n, dv)
    chunks, longest = None, 0
    if STATE_SPACE_CHUNKED_FROM > 0 and step.max_q_len >= STATE_SPACE_CHUNKED_FROM and step.q_lens and state_space_chunked_supports(n, dv):
        key = ("chunks", STATE_SPACE_CHUNKED_FROM)
        if key not in step.attn_tiles:
            step.attn_tiles[key] = portion_chunks(step.q_lens, step.ctx_lens, STATE_SPACE_CHUNKED_FROM, xbc.device)
        chunks, longest = step.attn_tiles[key], STATE_SPACE_CHUNKED_FROM - 1
    args = (xbc, proj, off_dt, dt_bias, a_log, skip, state, step)
    if chunks is None:
        return state_space_walk(*args, heads, groups, n, dv)
    out = torch.empty((xbc.shape[0], heads * dv), dtype=torch.float32, device=xbc.device)
    state_space_chunked(*args, chunks, heads, groups, n, dv, out)
    if chunks[7] < step.num_seqs:
        state_space_walk(*args, heads, groups, n, dv, max_len=longest, out=out)
    return out


def gated_group_norm(y, gate, off_g: int, gain, eps: float, groups: int, out_dtype) -> torch.Tensor:
    """``v = y * silu(gate[:, off_g ..])``, its channels in ``groups`` equal parts each over its own root mean square, times ``gain``, in
    ``out_dtype``; ``y`` float32 ``[T, n]``, ``gate`` a float32 product."""
    _chk(y, gate, gain)
    T, n = y.shape
    if y.dtype != torch.float32 or gate.dtype != torch.float32 or gain.numel() != n or n % groups or off_g + n > gate.shape[1]:
        raise KernelError("gated_group_norm: float32 rows, gates and a gain of their width, in equal parts")
    out = torch.empty((T, n), dtype=out_dtype, device=y.device)
    call("sllm_gated_group_norm", _p(y), _p(gate), gate.shape[1], int(off_g), _p(gain), float(eps), int(groups), _p(out), _dtc(out_dtype), T, n, _stream())
    return out


# ---- latent attention ------------------------------------------------------------------------------------

def latent_rope_write(proj, off: int, rank: int, tail: int, rotary_dim: int, gain, eps: float, positions, table, slot_mapping,
                      cache, queries=None):
    """`latent_write` with ``tail`` more columns behind the latent: a key part all heads share, not normed, its first
    ``rotary_dim`` channels rotated by position (``table`` float32 ``[positions, 2, rotary_dim/2]``).  Rows of the cache
    ``[pages, 1, page_size, D]`` receive latent, tail and zeros up to D.  ``queries`` = (column, gain): also `norm_cols` of as many
    columns as the gain has values, in the cache's dtype, by the same launch; they are returned."""
    _chk(proj, gain, positions, table, slot_mapping, cache)
    q_off, q_gain = queries if queries is not None else (0, None)
    q = torch.empty((proj.shape[0], q_gain.numel()), dtype=cache.dtype, device=proj.device) if q_gain is not None else None
    D = cache.shape[3]
    if proj.dtype != torch.float32 or cache.shape[1] != 1 or D < rank + tail:
        raise KernelError("latent_rope_write: a float32 product and a cache [pages, 1, page_size, D >= rank + tail]")
    max_pos = 0
    if rotary_dim:
        if table is None or table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rotary_dim // 2):
            raise KernelError("latent_rope_write: rotary table must be float32 [positions, 2, rotary_dim/2]")
        max_pos = table.shape[0]
    call("sllm_latent_rope_write", _p(proj), proj.shape[1], int(off), int(rank), int(tail), int(rotary_dim), _p(gain), float(eps),
         _p(positions), _p(table), max_pos, _p(slot_mapping), _p(cache), _dt(cache), D, int(q_off),
         q_gain.numel() if q_gain is not None else 0, _p(q_gain), _p(q), proj.shape[0], _stream())
    return q


def rope_cols_(out, ooff: int, ostride: int, x, xoff: int, xstride: int, n: int, rotary_dim: int, positions, table, heads: int) -> None:
    """Per head h: the ``n`` columns ``x[t, xoff + h*xstride ..]`` of a float32 product, the first ``rotary_dim`` of them
    rotated by position, written to ``out[t, h*ostride + ooff ..]``; what lies between ``ooff + n`` and the head's next
    ``ostride`` is zeroed."""
    _chk(out, x, positions, table)
    if x.dtype != torch.float32:
        raise KernelError("rope_cols_: a float32 product")
    max_pos = table.shape[0] if rotary_dim else 0
    call("sllm_rope_cols", _p(x), x.shape[1], int(xoff), int(xstride), int(n), int(rotary_dim), _p(positions), _p(table), max_pos,
         _p(out), _dt(out), out.shape[1], int(ooff), int(ostride), x.shape[0], int(heads), _stream())


def latent_write(proj, off: int, rank: int, gain, eps: float, slot_mapping, cache) -> None:
    """Columns ``off .. off+rank`` of the float32 product, over their root mean square, times ``gain``: each
    token's latent, written to its place in the paged ``cache`` ``[pages, 1, page_size, rank]`` (skipped where the
    slot is -1)."""
    _chk(proj, gain, slot_mapping, cache)
    if proj.dtype != torch.float32 or cache.shape[1] != 1 or cache.shape[3] != rank:
        raise KernelError("latent_write: a float32 product and a cache [pages, 1, page_size, rank]")
    call("sllm_latent_write", _p(proj), proj.shape[1], int(off), int(rank), _p(gain), float(eps), _p(slot_mapping), _p(cache),
         _dt(cache), proj.shape[0], _stream())


def head_linear(x, xoff: int, w, out_dtype, *, gate=None, goff: int = 0, gate_elem: bool = False, xstride: int | None = None,
                ostride: int | None = None) -> torch.Tensor:
    """A product per head: ``out[t, h, :] = w[h] @ x[t, xoff + h*xstride : .. + din]`` with ``w [H, dout, din]`` (heads
    ``xstride`` apart in x, ``din`` by default), times ``sigmoid(gate[t, goff + h])`` if ``gate`` (a float32 product) is
    given, or, with ``gate_elem``, times ``sigmoid(gate[t, goff + h*dout + n])`` element by element.  ``[T, H*ostride]`` in
    ``out_dtype`` (``ostride`` >= dout, dout by default; the columns between are left for the caller to fill)."""
    _chk(x, w, gate)
    T, ldx = x.shape
    H, dout, din = w.shape
    xs, os_ = int(xstride or din), int(ostride or dout)
    out = torch.empty((T, H * os_), dtype=out_dtype, device=x.device)
    call("sllm_head_linear_strided", _p(x), _dt(x), ldx, int(xoff), xs, _p(w), _dt(w), _p(out), _dtc(out_dtype), H * os_, os_,
         _p(gate), gate.shape[1] if gate is not None else 0, int(goff), 1 if gate_elem else 0, T, H, din, dout, _stream())
    return out


def add_rmsnorm(residual: torch.Tensor, delta, weight: torch.Tensor, eps: float,
                out_dtype: torch.dtype) -> torch.Tensor:
    """``residual += delta`` (in place, if delta is given; a 3-d delta is a stack of
    partial sums) and return ``rmsnorm(residual) * weight`` in ``out_dtype``."""
    _chk(residual, delta, weight)
    rows, H = residual.shape
    if residual.dtype != torch.float32 or weight.dtype != torch.float32:
        raise KernelError("add_rmsnorm: the residual stream and the gain are float32")
    parts, stride = 1, 0
    if delta is not None:
        if delta.dim() == 3:
            parts, stride = delta.shape[0], delta.shape[1] * delta.shape[2]
        if tuple(delta.shape[-2:]) != (rows, H):
            raise KernelError(f"add_rmsnorm: delta {tuple(delta.shape)} does not fit residual {(rows, H)}")
    out = torch.empty((rows, H), dtype=out_dtype, device=residual.device)
    call("sllm_add_rmsnorm", _p(residual), _p(delta), _dt(delta) if delta is not None else F32, parts, stride,
         _p(weight), float(eps), _p(out), _dtc(out_dtype), rows, H, _stream())
    return out


def gemm_f32(x: torch.Tensor, w: torch.Tensor, bias) -> torch.Tensor:
    """True float32 ``x @ w.T + bias``: CUDA-core FMA, fixed summation order."""
    _chk(x, w, bias)
    M, K = x.shape
    N, K2 = w.shape
    if K != K2:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    out = torch.empty((M, N), dtype=torch.float32, device=x.device)
    call("sllm_gemm_f32", _p(x), _p(w), _p(bias), _p(out), M, N, K, _stream())
    return out


TCGEN05_MIN_ROWS = 128    # below this a 128-row tile is mostly padding
PAIR_SILU_FROM_ROWS = 64  # from here on gate|up with its activation goes to the CTA-pair kernel (see `linear_silu_mul`)
STREAM_MAX_ROWS = 32      # beyond this the kernel's shared-memory reads of the activations bound it


@functools.lru_cache(maxsize=4096)
def stream_supports(M: int, N: int, K: int) -> bool:
    """Whether the weight-streaming kernel is the one for this product (it is not where the tensor-core form
    of the same job is the faster one: see `linear_tc_supports`)."""
    if not (M <= STREAM_MAX_ROWS and bool(lib().sllm_linear_stream_supports(int(M), int(N), int(K)))):
        return False
    return not linear_tc_supports(M, N, K)


PLAIN_ACTS = {None: 0, "relu2": 1, "token": 2, "gelu": 3}      # SLLM_ACT_* of the kernels: activations of a plain (ungated) result


class TokenColumns:
    """Columns ``off ..`` of a table with a row per token id (``table [V, ld]`` in the compute dtype), at the step's ``ids``
    (int32 ``[T]``): what the ``token`` activation multiplies by."""
    __slots__ = ("table", "ids", "off")

    def __init__(self, table, ids, off: int):
        self.table, self.ids, self.off = table, ids, int(off)

    def args(self):
        return _p(self.table), _p(self.ids), self.off, self.table.shape[1], self.table.shape[0]


_NO_TOKEN = (None, None, 0, 0, 0)


def linear_stream(x, w, bias, out_dtype, *, splits: int = 1, silu: bool = False, act: "str | None" = None):
    """The weight-streaming kernel for at most 64 tokens.  With ``splits`` > 1 the result is
    a float32 stack ``[splits', M, N]`` of partial sums (bias in the first) that the consumer
    adds; with ``silu`` the matrix is gate|up interleaved in blocks of 8 and the result is
    ``silu(gate) * up`` of width N/2; with ``act="gelu_tanh"`` it is ``gelu_tanh(gate + bias) * (up + bias)``
    (the bias interleaved like the rows)."""
    if act not in (None, "gelu_tanh") or (act and silu):
        raise KernelError(f"linear_stream: gated epilogue {act!r}")
    gated = silu or act is not None
    _chk(x, w, bias)
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    L = lib()
    real = L.sllm_linear_stream_splits(K, int(splits)) if splits > 1 else 1
    partial = None
    if real > 1:
        partial = torch.empty((real, M, N), dtype=torch.float32, device=x.device)
        out = None
    else:
        out = torch.empty((M, N // 2 if gated else N), dtype=out_dtype, device=x.device)
    call("sllm_linear_stream", _p(x), _p(w), _p(bias), _p(out), _dtc(out_dtype), _p(partial), M, N, K,
         real if real > 1 else 1, 1 if silu else 2 if act else 0, _stream())
    return partial if real > 1 else out


_tc_status: dict = {}      # device -> int32[1]: non-zero once a wait inside a tcgen05 kernel ran out
_tc_used = {"since_check": 0}


def _status_word(device) -> torch.Tensor:
    t = _tc_status.get(device)
    if t is None:
        t = _tc_status[device] = torch.zeros(1, dtype=torch.int32, device=device)
    return t


def status_word_launches() -> int:
    """Launches since the last check of kernels that report through the status word."""
    return _tc_used["since_check"]


def note_status_word_launches(n: int) -> None:
    """A replayed CUDA graph launched ``n`` such kernels (the capture counted them once)."""
    _tc_used["since_check"] += int(n)


def check_tcgen05_status() -> None:
    """Raise if a bounded wait inside a TMA-fed kernel (the tcgen05 product, the TMA attention) gave
    up since the last check (reads one int from each device that ran such a kernel; synchronises)."""
    if not _tc_used["since_check"]:
        return
    _tc_used["since_check"] = 0
    for dev, t in _tc_status.items():
        code = int(t.item())
        if code:
            t.zero_()
            who = {1: "gemm_tcgen05: the TMA producer", 2: "gemm_tcgen05: the MMA issuer", 3: "gemm_tcgen05: the epilogue",
                   11: "attention_tma: the producer", 12: "attention_tma: a compute warp",
                   41: "gemm_pair: the TMA producer", 42: "gemm_pair: the MMA issuer", 43: "gemm_pair: the epilogue",
                   31: "linear_tc: the TMA producer", 32: "linear_tc: the MMA issuer", 33: "linear_tc: the epilogue",
                   }.get(code, f"code {code}")
            raise KernelError(f"{who} on {dev}: a bounded wait ran out; the result is not valid")


@functools.lru_cache(maxsize=4096)
def tcgen05_supports(M: int, N: int, K: int) -> bool:
    return bool(lib().sllm_gemm_tcgen05_supports(int(M), int(N), int(K)))


def gemm_tcgen05(x, w, bias, out_dtype, *, silu: bool = False):
    """``x @ w.T (+ bias)`` on the tcgen05 tensor cores (TMA-fed, accumulator in tensor memory);
    with ``silu`` the matrix is gate|up interleaved in blocks of 8 and the bfloat16 result is
    ``silu(gate) * up`` of width N/2."""
    _chk(x, w, bias)
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise KernelError("gemm_tcgen05: bfloat16 operands only")
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    if silu:
        epi, out = 2, torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
    elif out_dtype == torch.float32:
        epi, out = 0, torch.empty((M, N), dtype=torch.float32, device=x.device)
    else:
        epi, out = 1, torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    call("sllm_gemm_tcgen05", _p(x), _p(w), _p(bias), _p(out), M, N, K, epi, _p(_status_word(x.device)), _stream())
    _tc_used["since_check"] += 1
    return out


# which products of prompt portions (more than 128 rows) run on this package's CTA-pair kernel: "all", "fused" (only
# gate|up with its SiLU epilogue; the plain products go to the library) or "off" (the one-CTA kernel for gate|up)
_PAIR_GEMM = os.environ.get("SLLM_PAIR_GEMM", "all")


@functools.lru_cache(maxsize=4096)
def pair_supports(M: int, N: int, K: int) -> bool:
    return bool(lib().sllm_gemm_pair_supports(int(M), int(N), int(K)))


@functools.lru_cache(maxsize=4096)
def pair_tiles_wide(M: int, N: int) -> bool:
    """Whether tiles of 256 x 512 serve an [M, N] result better than tiles of 256 x 256.  The pairs of SMs run
    the tiles in waves; a wide tile takes twice a narrow one's time and a quarter less traffic from L2, but its
    epilogue is not hidden behind the next tile's products.  So: wide where it needs no more time in waves and a
    pair has few tiles anyway (the attention and down projections of a prompt portion: one wave in place of one
    and a half), narrow where a pair walks many tiles (gate|up: sixteen each at 2,048 rows)."""
    pairs = max(num_sms() // 2, 1)
    mt = -(-M // 256)
    waves_narrow = -(-(mt * -(-N // 256)) // pairs)
    waves_wide = -(-(mt * -(-N // 512)) // pairs)
    return 2 * waves_wide <= waves_narrow and waves_narrow < 4


@functools.lru_cache(maxsize=4096)
def pair_wide_cols(M: int, N: int):
    """`pair_tiles_wide` for the epilogues that also have wide tiles of 448, 384 and 320 columns (float32 result,
    residual).  Measured, a wave of wide tiles takes time in proportion to 256 + its columns (the operands a pair
    pulls per k block) and a wave of 256-wide tiles as much as 384 such units (2,048 rows, K = 5,120, us a wave:
    48 / 50 / 55 / 63 at 320 / 384 / 448 / 512 columns, 30.5 at 256).  A narrower wide tile is taken where it
    beats both the 512-wide and the 256-wide tiles by that count: 2,048 x 3,584 (the attention and down
    projections of a 7B model) has 56 tiles of 512 for 74 pairs of SMs and 64 of 448 (58 -> 53 us and 232 -> 214
    with the residual epilogue); 1,024 x 5,120 goes from 77 us to 60 at 320 columns.
    False: 256 x 256; True: 256 x 512; else the width."""
    pairs = max(num_sms() // 2, 1)
    mt = -(-M // 256)
    waves_narrow = -(-(mt * -(-N // 256)) // pairs)
    if waves_narrow >= 4:
        return False
    best, best_cost = False, waves_narrow * 384
    if pair_tiles_wide(M, N):
        best, best_cost = True, min(best_cost, -(-(mt * -(-N // 512)) // pairs) * 768)
    for cols in (448, 384, 320):
        cost = -(-(mt * -(-N // cols)) // pairs) * (256 + cols)
        if cost < best_cost:
            best, best_cost = cols, cost
    return best


@functools.lru_cache(maxsize=4096)
def pair_tiles_slim(M: int, N: int) -> bool:
    """Whether tiles of 256 x 128 serve an [M, N] result better than tiles of 256 x 256: where the wider ones
    would leave at least half of the pairs of SMs without a tile (a prompt portion of 512 tokens times the
    q|k|v matrix: 36 tiles for 74 pairs; 30.6 -> 25.5 us).  The gain is small, since a pair is bound by the rate
    at which it pulls its operands and half the width moves three quarters of the bytes; where K is long enough
    the product is cut along K instead (`pair_splits`)."""
    pairs = max(num_sms() // 2, 1)
    return 2 * (-(-M // 256) * -(-N // 256)) <= pairs


PAIR_SPLIT_MAX = 8            # slices of K at most (each leaves a float32 copy of the result for the consumer to add)
PAIR_SPLIT_MIN_BLOCKS = 8     # 64-wide k blocks a slice has at least
PAIR_US_PER_K_BLOCK = 0.4     # a pair of SMs on one 256 x 256 tile, per 64-wide k block (measured: 116 us for K = 18,944)
PAIR_US_PER_ELEMENT = 2.4e-6  # one more float32 copy of the result for the next kernel to add, per element (whole portions
                              # of 192 to 1,024 tokens were timed with 0.5, 1.0 and 2.4: the last gave the best choices)
PAIR_SPLIT_GAIN = 0.85        # slices only where the whole path (slices, then a kernel that adds them) takes this share
PAIR_SPLIT_GAIN_WAVES = 0.8    # the same where the unsliced tiles are more than one wave


@functools.lru_cache(maxsize=4096)
def pair_splits(M: int, N: int, K: int) -> int:
    """Slices of K for the CTA-pair product of an [M, N] result with few 256 x 256 tiles: a pair of SMs pulls its
    operands through shared memory at a rate of its own, so a product whose tiles leave most pairs idle takes as
    long as its tiles' K, whatever the GPU could do (512 tokens times the down projection: 28 tiles for 74 pairs,
    116 us; the library's product 56).  With S slices a unit is (tile, slice), the units run in waves over the pairs
    and the time goes as waves / S; the slices' partial sums are a stack for the consumer to add (512 tokens, down:
    66 us in two slices).  The choice weighs that against the fused epilogues the unsliced product keeps: waves x K
    blocks for the products, a copy of the result per slice written and read, three copies for the residual
    epilogue's traffic (in a graph, measured: within 10 % of this at 192 to 1,024 tokens)."""
    pairs = max(num_sms() // 2, 1)
    tiles = -(-M // 256) * -(-N // 256)
    k_blocks = -(-K // 64)
    t_tile, t_copy = k_blocks * PAIR_US_PER_K_BLOCK, M * N * PAIR_US_PER_ELEMENT
    whole = -(-tiles // pairs) * t_tile + 3 * t_copy
    best, best_cost = 1, whole
    for s in range(2, PAIR_SPLIT_MAX + 1):
        if k_blocks // s < PAIR_SPLIT_MIN_BLOCKS:
            break
        cost = -(-tiles * s // pairs) / s * t_tile + (s + 2) * t_copy
        if cost < best_cost:
            best, best_cost = s, cost
    # (more than one wave of tiles: whole portions gained where the model promised a quarter (hidden 5,120, 1,024
    # tokens: 7.7 -> 7.3 ms for 8 layers) and not where it promised a fifth (hidden 3,584, 1,792 tokens))
    gain = PAIR_SPLIT_GAIN if tiles <= pairs else PAIR_SPLIT_GAIN_WAVES
    return best if best_cost <= gain * whole else 1


def gemm_pair(x, w, bias, out_dtype, *, silu: bool = False, wide: "bool | str | None" = None, scale: "RowScale | None" = None,
              residual=None, next_gain=None, splits: int = 1, act: "str | None" = None, token: "TokenColumns | None" = None):
    """The same product and epilogues as `gemm_tcgen05`, by pairs of CTAs on 256 x 256 tiles, on
    256 x 512 tiles (``wide=True``; by default where those fill the GPU at least as well; ``wide=448``, ``384`` or
    ``320``: tiles of that many columns, float32 result or residual epilogue, chosen by `pair_wide_cols` where
    they fill the pairs of SMs better) or on 256 x 128 tiles (``wide="slim"``; by default where the result has few tiles)
    (``tcgen05.mma`` with ``cta_group::2``: each CTA loads half of each operand).
    ``scale``: a norm still owed on ``x`` (`RowScale`).  ``residual`` (float32 ``[M, N]``): the product is added
    into it in place and None is returned; with ``next_gain`` the kernel also writes the next norm's input in the
    owed form and ``(xg, RowScale)`` comes back (the scale's eps left at 0 for the caller to set).
    ``splits`` > 1 (float32 result, no other epilogue): K in that many slices, the result a stack ``[splits', M, N]``
    of partial sums (bias in the first) for the consumer to add.  ``act="gelu_tanh"``: the gated epilogue
    ``gelu_tanh(gate + bias) * (up + bias)`` in place of ``silu``'s (rows and bias interleaved in blocks of 8); ``"relu2"``:
    bfloat16 ``max(v, 0)^2`` of the plain result; ``"gelu"``: its exact gelu; ``"token"``: bfloat16 ``gelu_tanh(v)`` times ``token``'s columns."""
    _chk(x, w, bias, residual, next_gain)
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise KernelError("gemm_pair: bfloat16 operands only")
    if act not in (None, "gelu_tanh", "relu2", "token", "gelu") or (act and silu):
        raise KernelError(f"gemm_pair: epilogue {act!r}")
    plain_act = act if act in ("relu2", "token", "gelu") else None
    gelu, silu = act == "gelu_tanh", silu or act == "gelu_tanh"
    if plain_act and (residual is not None or bias is not None or out_dtype != torch.bfloat16 or (token is not None) != (act == "token")):
        raise KernelError(f"gemm_pair: the {act} epilogue takes neither bias nor residual and gives bfloat16")
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    out = xg = ssq = None
    stride = 0
    plain_or_residual = not silu and (residual is not None or out_dtype == torch.float32)
    if wide is None:
        wide = False if splits > 1 else "slim" if pair_tiles_slim(M, N) else \
            False if act == "token" else pair_wide_cols(M, N) if plain_or_residual else pair_tiles_wide(M, N)
    code = 2 if wide == "slim" else 0 if wide is False else 1 if wide is True or wide == 512 else int(wide)
    if code > 2 and (code not in (448, 384, 320) or not plain_or_residual):
        raise KernelError(f"gemm_pair: tiles of {wide} columns (448, 384 or 320, and only with a float32 result or a residual)")
    if residual is not None:
        if silu or residual.dtype != torch.float32 or tuple(residual.shape) != (M, N):
            raise KernelError(f"gemm_pair: residual {tuple(residual.shape)} {residual.dtype} does not fit [{M}, {N}] float32")
        epi = 3
        if next_gain is not None:
            if next_gain.dtype != torch.float32 or next_gain.numel() != N:
                raise KernelError("gemm_pair: the next norm's gain is float32 of N values")
            parts = pair_parts(N, code)
            stride = (parts + 3) & ~3
            xg = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
            ssq = torch.empty((M, stride), dtype=torch.float32, device=x.device)
    elif silu:
        epi, out = 4 if gelu else 2, torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
    elif out_dtype == torch.float32:
        real = int(lib().sllm_gemm_pair_splits(K, int(splits))) if splits > 1 else 1
        epi, out = 0, torch.empty((real, M, N) if real > 1 else (M, N), dtype=torch.float32, device=x.device)
    else:
        epi, out = {None: 1, "relu2": 5, "token": 6, "gelu": 7}[plain_act], torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    if splits > 1 and (epi != 0 or scale is not None):
        raise KernelError("gemm_pair: slices of K leave float32 partial sums: no other epilogue, no owed norm")
    call("sllm_gemm_pair", _p(x), _p(w), _p(bias), _p(out), M, N, K, epi, code, int(splits),
         *(scale.args_with_stride() if scale is not None else (None, 0, 0, 0.0, 0)),
         _p(residual), _p(next_gain), _p(xg), _p(ssq), stride, *(token.args() if token is not None else _NO_TOKEN),
         _p(_status_word(x.device)), _stream())
    _tc_used["since_check"] += 1
    if residual is not None:
        return (xg, RowScale(ssq, pair_parts(N, code), 0.0, N)) if next_gain is not None else None
    return out


@functools.lru_cache(maxsize=256)
def pair_parts(N: int, form: int = 0) -> int:
    """Partial sums of squares per row that `gemm_pair`'s residual epilogue writes for N columns with tiles of the
    form ``form`` (the kernel's code: 0, 1, 2, or 448, 384, 320)."""
    return int(lib().sllm_gemm_pair_parts_of(int(N), int(form)))


LINEAR_TC_MAX_ROWS = 128  # the tokens are the tensor core's N side: one tile of at most 128
# Plain products go to it only where it beats the library: a reduction of at least this length with at
# most this many tokens (at 7B sizes, 64 tokens: down 29.3 against 30.7 us; qkv 11.6 against 9.2 us).
LINEAR_TC_SPLIT_MIN_K = 8192
LINEAR_TC_SPLIT_MAX_ROWS = 64


_LINEAR_TC = os.environ.get("SLLM_LINEAR_TCGEN05", "1") != "0"     # 0: 33..128 tokens on the library product


# From how many tokens on it takes a product over from the streaming kernel, by the matrix's size (in-graph
# times at 7B sizes, us, streaming kernel / this one).  A small matrix (q|k|v, o_proj: under 2^25 elements)
# stays with the streaming kernel as far as that goes (24 tokens: 9.1 / 10.1, 7.2 / 9.3).  A large one moves
# from 17 tokens on (24 tokens: gate|up 52.0 / 48.3, down 28.9 / 26.9; 16 tokens: 45.2 / 52.3, 24.3 / 26.3).
# A very wide one (the output head: at least four 128-row tiles an SM) moves from 9 on (16 tokens: 190.5 /
# 179.6; 32 tokens: 222.7 / 180.4; 8 tokens: 184.3 / 179.7, left where it is).
LINEAR_TC_LARGE = 1 << 25
LINEAR_TC_LARGE_FROM_ROWS = 17
LINEAR_TC_WIDE_TILES_PER_SM = 4
LINEAR_TC_WIDE_FROM_ROWS = 9


def _tc_from_rows(N: int, K: int) -> int:
    if N * K < LINEAR_TC_LARGE:
        return STREAM_MAX_ROWS + 1
    if -(-N // 128) >= LINEAR_TC_WIDE_TILES_PER_SM * num_sms():
        return LINEAR_TC_WIDE_FROM_ROWS
    return LINEAR_TC_LARGE_FROM_ROWS


@functools.lru_cache(maxsize=4096)
def linear_tc_takes(M: int, N: int, K: int) -> bool:
    """Whether the kernel runs these sizes at all."""
    return _LINEAR_TC and M <= LINEAR_TC_MAX_ROWS and bool(lib().sllm_linear_tc_supports(int(M), int(N), int(K)))


@functools.lru_cache(maxsize=4096)
def linear_tc_supports(M: int, N: int, K: int) -> bool:
    return linear_tc_takes(M, N, K) and M >= _tc_from_rows(N, K)


@functools.lru_cache(maxsize=4096)
def _tc_splits(N: int, K: int) -> int:
    """Slices of K so that (tiles of 128 rows) x slices comes to about one unit per SM, each slice
    at least eight 64-wide k blocks long."""
    tiles = -(-N // 128)
    return max(1, min(num_sms() // tiles, (K // 64) // 8))


def linear_tc(x, w, bias, out_dtype, *, splits: int = 1, silu: bool = False, act: "str | None" = None):
    """The weight-streaming product on the tcgen05 tensor cores for up to 128 tokens.  With
    ``splits`` > 1 the result is a float32 stack ``[splits', M, N]`` of partial sums (bias in the
    first) that the consumer adds; with ``silu`` the matrix is gate|up interleaved in blocks of 8
    and the bfloat16 result is ``silu(gate) * up`` of width N/2; with ``act="relu2"`` the bfloat16 result is ``max(v, 0)^2``, with
    ``"gelu"`` the exact gelu."""
    _chk(x, w, bias)
    if act not in (None, "relu2", "gelu") or (act and (silu or out_dtype != torch.bfloat16)):
        raise KernelError(f"linear_tc: epilogue {act!r}")
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise KernelError("linear_tc: bfloat16 operands only")
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    real = 1
    if silu:
        epi, out = 2, torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
    elif out_dtype == torch.float32:
        real = int(lib().sllm_linear_tc_splits(K, int(splits))) if splits > 1 else 1
        epi = 0
        out = torch.empty((real, M, N) if real > 1 else (M, N), dtype=torch.float32, device=x.device)
    else:
        epi, out = {None: 1, "relu2": 3, "gelu": 4}[act], torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    call("sllm_linear_tc", _p(x), _p(w), _p(bias), _p(out), M, N, K, real, epi, _p(_status_word(x.device)), _stream())
    _tc_used["since_check"] += 1
    return out


WS_MAX_COLS = 8192        # wider products have CTAs enough for the 128-row streaming kernel
WS_MAX_ROWS = 32          # one, two or four 8-token tiles (with fewer k blocks in flight the more tiles, so that two CTAs still share an SM)
# Four tiles (17..32 tokens, one k block in flight per group) stream slowly, so only where little streams and the
# fused epilogues save kernels: a short reduction, a matrix of at most 2^24 elements, and rows enough for one and a
# half CTAs an SM (q|k|v and o_proj at a hidden size of 3,584: decode at batch 24 and 32 +2.5 %; at hidden sizes of
# 1,536 and 2,048 the k-split kernel with its norm and rotary kernels stayed the faster, 2.05 against 2.21 ms a step).
WS_ROWS32_MAX_ELEMENTS = int(os.environ.get("SLLM_WS_ROWS32_MAX_ELEMENTS", str(1 << 24)))
WS_ROWS32_MAX_K = 4096
MAX_SCALE_PARTS_ROWS32 = 192   # the table of partial sums a four-tile consumer keeps (streams of up to 3,072 columns)


@functools.lru_cache(maxsize=4096)
def ws_supports(M: int, N: int, K: int) -> bool:
    """Whether the warp-split kernel is the one for this product.  With two token tiles (9..16 tokens) only where
    its 16-row CTAs fit the GPU at once: at N = 5120 (320 to 592 CTAs for 296 places) it falls behind the k-split
    kernel by more than the fused epilogues save (16 tokens, K = 27648: 64.3 against 49.2 us)."""
    return N <= WS_MAX_COLS and ws_takes(M, N, K) and _ws_tokens_ok(M, N, K)


@functools.lru_cache(maxsize=4096)
def ws_takes(M: int, N: int, K: int) -> bool:
    """Whether the kernel runs these sizes at all."""
    return M <= WS_MAX_ROWS and bool(lib().sllm_linear_ws_supports(int(M), int(N), int(K)))


def _ws_tokens_ok(M: int, N: int, K: int) -> bool:
    if M <= 8:
        return True
    if -(-N // 16) > 2 * num_sms():
        return False
    return M <= 16 or (N * K <= WS_ROWS32_MAX_ELEMENTS and K <= WS_ROWS32_MAX_K and 2 * -(-N // 16) >= 3 * num_sms())


class RowScale:
    """An RMSNorm still owed on an activation: the activation is bfloat16(stream * gain), ``ssq`` is float32
    ``[M, stride]`` (stride = ``parts`` rounded up to 4) with ``parts`` partial sums of squares of each row of
    the stream (``width`` wide), and whoever multiplies the activation by a matrix multiplies each row of the
    result by ``rsqrt(sum(ssq[row, :parts]) / width + eps)``: W (x g / rms) = (W (x g)) / rms."""
    __slots__ = ("ssq", "parts", "eps", "width")

    def __init__(self, ssq, parts: int, eps: float, width: int):
        self.ssq, self.parts, self.eps, self.width = ssq, int(parts), float(eps), int(width)

    def args(self):
        return _p(self.ssq), self.parts, self.eps, self.width

    def args_with_stride(self):
        return _p(self.ssq), self.parts, self.ssq.shape[1], self.eps, self.width


_NO_SCALE = (None, 0, 0.0, 0)
MAX_SCALE_PARTS = 608          # partial sums a consumer keeps in shared memory per row


def linear_ws(x, w, bias, out_dtype, residual=None, scale: RowScale | None = None, next_gain=None, act: "str | None" = None,
              token: "TokenColumns | None" = None):
    """The warp-split streaming kernel (at most 16 tokens): ``x @ w.T (+ bias)`` in ``out_dtype``,
    or, given ``residual`` (float32 ``[M, N]``), added into it in place (returns None).  ``scale``: a norm
    still owed on ``x`` (`RowScale`).  ``next_gain`` (with ``residual``): the gain of the norm that follows; the
    kernel then also writes that norm's input in the owed form and ``(xg, RowScale)`` is returned (the scale's
    eps is left at 0 for the caller to set).  ``act`` (without ``residual``): ``"relu2"``, the result's ``max(v, 0)^2``, ``"gelu"``, its exact gelu, or
    ``"token"``, ``gelu_tanh(v)`` times ``token``'s columns."""
    _chk(x, w, bias, residual, next_gain)
    M, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"linear: x {tuple(x.shape)} does not fit w {tuple(w.shape)}")
    out = None
    if residual is None:
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    elif residual.dtype != torch.float32 or tuple(residual.shape) != (M, N):
        raise KernelError(f"linear: residual {tuple(residual.shape)} {residual.dtype} does not fit [{M}, {N}] float32")
    xg = ssq = None
    parts = 0
    if next_gain is not None:
        if residual is None or next_gain.dtype != torch.float32 or next_gain.numel() != N:
            raise KernelError("linear_ws: the next norm's input needs the residual epilogue and a float32 gain of N values")
        parts = int(lib().sllm_linear_ws_parts(N, K))
        xg = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
        ssq = torch.empty((M, (parts + 3) & ~3), dtype=torch.float32, device=x.device)
    call("sllm_linear_ws", _p(x), _p(w), _p(bias), _p(out), _dtc(out_dtype), _p(residual), M, N, K,
         *(scale.args() if scale is not None else _NO_SCALE), _p(next_gain), _p(xg), _p(ssq),
         PLAIN_ACTS[act], *(token.args() if token is not None else _NO_TOKEN), _stream())
    if next_gain is not None:
        return xg, RowScale(ssq, parts, 0.0, N)
    return out


def _pair_rows(M: int) -> bool:
    return _PAIR_GEMM == "all" and M > TCGEN05_MIN_ROWS


def can_accumulate(x: torch.Tensor, w: torch.Tensor) -> bool:
    """Whether `linear_accumulate` has a kernel for these operands: few tokens (the warp-split streaming
    kernel) or a prompt portion (the CTA-pair product)."""
    if not (x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and x.is_cuda):
        return False
    M, K = x.shape
    N = w.shape[0]
    if ws_supports(M, N, K):
        return True
    # (a result of so few tiles that it is better cut along K leaves partial sums, which a norm kernel adds)
    return _pair_rows(M) and N % 4 == 0 and pair_supports(M, N, K) and pair_splits(M, N, K) == 1


def linear_accumulate(x, w, bias, residual) -> None:
    """``residual += x @ w.T (+ bias)`` in one kernel (see `can_accumulate`)."""
    if ws_supports(x.shape[0], w.shape[0], x.shape[1]):
        linear_ws(x, w, bias, torch.float32, residual=residual)
    else:
        gemm_pair(x, w, bias, torch.float32, residual=residual)


_NORM_FUSED = os.environ.get("SLLM_NORM_FUSED", "1") != "0"     # 0: every RMSNorm of a step is a kernel of its own


def can_accumulate_norm(x: torch.Tensor, w: torch.Tensor) -> bool:
    """Whether `linear_accumulate_norm` has a kernel for these operands."""
    if not (_NORM_FUSED and can_accumulate(x, w)):
        return False
    M, N = x.shape[0], w.shape[0]
    if ws_supports(M, N, x.shape[1]):
        return int(lib().sllm_linear_ws_parts(N, x.shape[1])) <= (MAX_SCALE_PARTS if M <= 16 else MAX_SCALE_PARTS_ROWS32)
    return N % 8 == 0


def linear_accumulate_norm(x, w, bias, residual, gain, eps: float):
    """``residual += x @ w.T (+ bias)`` and, from the same kernel, the input of the RMSNorm (``gain``, ``eps``)
    that follows, in the owed form: ``(bfloat16(residual * gain), RowScale)``."""
    if ws_supports(x.shape[0], w.shape[0], x.shape[1]):
        xg, scale = linear_ws(x, w, bias, torch.float32, residual=residual, next_gain=gain)
    else:
        xg, scale = gemm_pair(x, w, bias, torch.float32, residual=residual, next_gain=gain)
    scale.eps = float(eps)
    return xg, scale


def linear_scaled_supports(x: torch.Tensor, w: torch.Tensor) -> bool:
    """Whether `linear` takes ``x`` with a norm still owed (``scale=``): a prompt portion on the CTA-pair product."""
    M, K = x.shape
    return (x.is_cuda and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and _pair_rows(M)
            and pair_supports(M, w.shape[0], K))


def _stream_splits(N: int, K: int) -> int:
    ctas = -(-N // 128)
    return max(1, min(2 * num_sms() // ctas, K // 128, 16))


def linear(x: torch.Tensor, w: torch.Tensor, bias, out_dtype: torch.dtype, allow_partials: bool = False,
           scale: "RowScale | None" = None) -> torch.Tensor:
    """``x @ w.T (+ bias)``; ``w`` is ``[N, K]``.  float32 operands: this package's
    float32 kernel.  bfloat16 operands, float32 accumulation, result in ``out_dtype``: up
    to 64 rows the weight-streaming kernel (which, if ``allow_partials``, may return a
    float32 stack of partial sums ``[parts, M, N]`` for the consumer to add); beyond that
    the library product."""
    if x.dtype != w.dtype:
        raise KernelError(f"linear: x is {x.dtype}, w is {w.dtype}")
    if scale is not None:                       # a norm still owed on x (see `linear_scaled_supports`)
        if not linear_scaled_supports(x, w):
            raise KernelError("linear: no kernel takes this input with its norm still owed")
        return gemm_pair(x, w, bias, out_dtype, scale=scale)
    if x.dtype == torch.float32:
        if out_dtype != torch.float32:
            raise KernelError("linear: the float32 path keeps float32 results")
        return gemm_f32(x, w, bias)
    _chk(x, w, bias)
    if not x.is_cuda:
        raise KernelError("linear: CUDA only")
    M, K = x.shape
    N = w.shape[0]
    if ws_supports(M, N, K):
        return linear_ws(x, w, bias, out_dtype)
    if stream_supports(M, N, K):
        splits = _stream_splits(N, K) if (allow_partials and out_dtype == torch.float32) else 1
        return linear_stream(x, w, bias, out_dtype, splits=splits)
    if allow_partials and out_dtype == torch.float32 and M <= LINEAR_TC_SPLIT_MAX_ROWS and K >= LINEAR_TC_SPLIT_MIN_K \
            and linear_tc_supports(M, N, K):
        # a long reduction into few columns (the down projection): slices of K over all the SMs
        return linear_tc(x, w, bias, out_dtype, splits=_tc_splits(N, K))
    if N * K >= LINEAR_TC_LARGE and -(-N // 128) >= num_sms() and linear_tc_supports(M, N, K):
        return linear_tc(x, w, bias, out_dtype)      # a large matrix whose 128-row tiles are enough for every SM
    if _PAIR_GEMM == "all" and M > TCGEN05_MIN_ROWS and pair_supports(M, N, K):
        # prompt portions: pairs of CTAs on the tensor cores (tcgen05.mma with cta_group::2); a result of few tiles in
        # slices of K where the consumer adds partial sums
        if allow_partials and out_dtype == torch.float32 and pair_splits(M, N, K) > 1:
            return gemm_pair(x, w, bias, out_dtype, splits=pair_splits(M, N, K))
        return gemm_pair(x, w, bias, out_dtype)
    launches["library"] += 1
    if out_dtype == torch.float32:
        out = torch.mm(x, w.t(), out_dtype=torch.float32)
    else:
        out = torch.mm(x, w.t())
    if bias is not None:
        out += bias.to(out.dtype)
    return out


def plain_act(x, out_dtype, act: str, token: "TokenColumns | None" = None) -> torch.Tensor:
    """``act`` of ``x [T, N]`` (or of the sum of a stack of partial sums ``[parts, T, N]``) in ``out_dtype``: ``relu2`` is ``max(x, 0)^2``, ``gelu`` the exact (erf) gelu, ``token`` is ``gelu_tanh(x)`` times ``token``'s columns
    (a table of ``out_dtype``)."""
    _chk(x)
    T, N = x.shape[-2:]
    parts, stride = (x.shape[0], T * N) if x.dim() == 3 else (1, 0)
    if (act == "token") != (token is not None) or (token is not None and token.table.dtype != out_dtype):
        raise KernelError("plain_act: the token activation needs its table, of the result's dtype")
    out = torch.empty((T, N), dtype=out_dtype, device=x.device)
    call("sllm_plain_act", _p(x), _dt(x), parts, stride, _p(out), _dtc(out_dtype), T, N, PLAIN_ACTS[act], *(token.args() if token is not None else _NO_TOKEN),
         _stream())
    return out


_PLAIN_ACT_FUSED = os.environ.get("SLLM_PLAIN_ACT_FUSED", "1") != "0"      # 0: the product, then the activation kernel


def linear_plain_act(x, w, out_dtype, act: str, token: "TokenColumns | None" = None) -> torch.Tensor:
    """``act(x @ w.T)`` in ``out_dtype`` (see `plain_act`).  bfloat16: the activation leaves with the product's tile (the warp-split
    streaming product up to 16 tokens, the CTA-pair product of prompt portions; ``relu2`` and ``gelu`` of large matrices also on tensor memory).
    Otherwise the product in float32, cut along K where that is faster, then the activation kernel, which adds the slices.
    (In a graph, us: 8,448 x 2,048 and 8 tokens 8.3 in the warp-split form, 8.7 in four slices and a kernel, 17.5 in the streaming
    form unsliced; 16,512 x 4,096 and 8 tokens 29.3 / 26.6 / 36.8, on tensor memory 28.0; 32 tokens of the former 13.0 / 11.5 / 20.6,
    of the latter 27.6 on tensor memory and 35 in slices.)"""
    if _PLAIN_ACT_FUSED and x.is_cuda and x.dtype == torch.bfloat16 and out_dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and \
            x.shape[1] == w.shape[1]:
        M, K = x.shape
        N = w.shape[0]
        large = N * K >= LINEAR_TC_LARGE
        if ws_supports(M, N, K) or (M <= 16 and not large and ws_takes(M, N, K)):
            return linear_ws(x, w, None, out_dtype, act=act, token=token)
        if act in ("relu2", "gelu") and large and M >= LINEAR_TC_WIDE_FROM_ROWS and linear_tc_takes(M, N, K):
            return linear_tc(x, w, None, out_dtype, act=act)
        if _pair_rows(M) and pair_supports(M, N, K):
            return gemm_pair(x, w, None, out_dtype, act=act, token=token)
    return plain_act(linear(x, w, None, torch.float32, True), out_dtype, act, token)


def silu_mul(gu: torch.Tensor, interleave: int, out_dtype: torch.dtype) -> torch.Tensor:
    """``silu(gate) * up`` of ``gu [T, 2I]`` whose columns alternate between gate
    and up in blocks of ``interleave``."""
    _chk(gu)
    T, two_i = gu.shape
    I = two_i // 2
    out = torch.empty((T, I), dtype=out_dtype, device=gu.device)
    call("sllm_silu_mul", _p(gu), _dt(gu), _p(out), _dtc(out_dtype), T, I, int(interleave), _stream())
    return out


def silu_scaled_supports(x, w_gate_up, interleave: int, out_dtype) -> bool:
    """Whether `linear_silu_mul` takes an input whose norm is still owed (``scale``)."""
    M, K = x.shape
    N = w_gate_up.shape[0]
    if not (x.is_cuda and x.dtype == torch.bfloat16 and out_dtype == torch.bfloat16 and interleave == 8 and N % 16 == 0):
        return False
    return (M <= 32 and stream_supports(M, N, K)) or (M > TCGEN05_MIN_ROWS and _PAIR_GEMM != "off" and pair_supports(M, N, K))


def linear_silu_mul(x: torch.Tensor, w_gate_up: torch.Tensor, interleave: int, out_dtype: torch.dtype,
                    scale: RowScale | None = None) -> torch.Tensor:
    """``silu(x Wg^T) * (x Wu^T)`` with gate and up rows interleaved in one matrix.  ``scale``: a norm still
    owed on ``x`` (`RowScale`; see `silu_scaled_supports`)."""
    if scale is not None:
        if not silu_scaled_supports(x, w_gate_up, interleave, out_dtype):
            raise KernelError("linear_silu_mul: no kernel takes this input with its norm still owed")
        _chk(x, w_gate_up, scale.ssq)
        M, K = x.shape
        N = w_gate_up.shape[0]
        if M > 32:
            return gemm_pair(x, w_gate_up, None, out_dtype, silu=True, scale=scale)
        out = torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
        call("sllm_linear_stream_silu_scaled", _p(x), _p(w_gate_up), _p(out), M, N, K, *scale.args(), _stream())
        return out
    if x.dtype == torch.bfloat16 and out_dtype == torch.bfloat16 and interleave == 8 and x.is_cuda:
        M, K = x.shape
        N = w_gate_up.shape[0]
        if stream_supports(M, N, K):
            return linear_stream(x, w_gate_up, None, out_dtype, silu=True)
        if PAIR_SILU_FROM_ROWS <= M <= TCGEN05_MIN_ROWS and N % 16 == 0 and _PAIR_GEMM != "off" and pair_supports(M, N, K):
            # 64..128 tokens: still bound by reading W once, and the pair kernel's narrow tiles (two accumulators, the
            # epilogue under the next tile) stream it faster than `linear_tc`, whose accumulator is 128 columns wide there
            # (in a graph, 7B sizes, us: 64 tokens 51.0 against 53.4, 96 tokens 51.8 / 57.9, 128 tokens 53.1 / 61.9)
            return gemm_pair(x, w_gate_up, None, out_dtype, silu=True, wide=False)
        if N % 16 == 0 and linear_tc_supports(M, N, K):
            return linear_tc(x, w_gate_up, None, out_dtype, silu=True)
        if M > TCGEN05_MIN_ROWS and N % 16 == 0 and _PAIR_GEMM != "off" and pair_supports(M, N, K):
            # many rows: pairs of CTAs on the tensor cores, the activation applied as the tile leaves tensor memory
            return gemm_pair(x, w_gate_up, None, out_dtype, silu=True)
        if M > TCGEN05_MIN_ROWS and N % 16 == 0 and tcgen05_supports(M, N, K):
            return gemm_tcgen05(x, w_gate_up, None, out_dtype, silu=True)
    gu = linear(x, w_gate_up, None, x.dtype)
    return silu_mul(gu, interleave, out_dtype)


_QKV_ROPE = os.environ.get("SLLM_QKV_ROPE_FUSED", "1") != "0"     # 0: the product, then the rotary kernel


def qkv_rope_supports(x, w, table, rotary_dim, nq, nkv, hd, k_cache) -> bool:
    """Whether `linear_rope_kv_write` takes the product: bfloat16, few tokens, the whole head rotated
    (or no rotation at all), a head size that is a multiple of 16."""
    if not (_QKV_ROPE and x.is_cuda and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and k_cache.dtype == torch.bfloat16):
        return False
    rot = int(rotary_dim) if table is not None else 0
    M, K = x.shape
    return M <= WS_MAX_ROWS and _ws_tokens_ok(M, w.shape[0], K) and bool(lib().sllm_linear_ws_rope_supports(int(M), int(w.shape[0]), int(K), int(nq), int(nkv),
                                                                          int(hd), rot))


def linear_rope_kv_write(x, w, bias, positions, table, rotary_dim, nq, nkv, hd, slot_mapping, k_cache, v_cache,
                         scale: RowScale | None = None):
    """``x @ w.T`` for the fused q|k|v matrix with what follows it in an attention layer done in the
    product's epilogue: bias, rotary encoding of the query and key heads by the tokens' positions,
    the new keys and values written to ``slot_mapping`` of the paged caches (not written when it is
    None).  Returns the rotated queries ``[T, nq*hd]`` bfloat16.  Few tokens only (`qkv_rope_supports`).
    ``scale``: a norm still owed on ``x`` (`RowScale`)."""
    _chk(x, w, bias, positions, table, slot_mapping, k_cache, v_cache)
    M, K = x.shape
    N = w.shape[0]
    rot = int(rotary_dim) if table is not None else 0
    num_pages, nkv_c, page_size, hd_c = k_cache.shape
    if (nkv_c, hd_c) != (nkv, hd) or tuple(v_cache.shape) != tuple(k_cache.shape):
        raise KernelError("linear_rope_kv_write: the caches are [pages, kv heads, page size, head size]")
    if table is not None and (table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rot // 2)):
        raise KernelError("linear_rope_kv_write: rotary table must be float32 [positions, 2, rotary_dim/2]")
    q = torch.empty((M, nq * hd), dtype=torch.bfloat16, device=x.device)
    max_pos = table.shape[0] if table is not None else 0
    call("sllm_linear_ws_rope", _p(x), _p(w), _p(bias), M, N, K, _p(positions), _p(table), rot, max_pos, nq, nkv, hd,
         _p(slot_mapping), page_size, num_pages, _p(k_cache), _p(v_cache), _p(q),
         *(scale.args() if scale is not None else _NO_SCALE), _stream())
    return q


def rope_kv_write(qkv, bias, positions, table, rotary_dim, nq, nkv, hd, slot_mapping, k_cache, v_cache,
                  out_dtype: torch.dtype) -> torch.Tensor:
    """Bias, rotary encoding and the cache write for the fused q|k|v rows.
    Returns the rotated queries ``[T, nq*hd]`` in ``out_dtype``; keys and values go
    to ``slot_mapping`` in ``k_cache``/``v_cache`` ``[pages, nkv, page_size, hd]``
    (not written when ``slot_mapping`` is None)."""
    _chk(qkv, bias, positions, table, slot_mapping, k_cache, v_cache)
    parts, part_stride = 1, 0
    if qkv.dim() == 3:                       # a stack of partial sums from a k-split product
        parts, part_stride = qkv.shape[0], qkv.shape[1] * qkv.shape[2]
    T = qkv.shape[-2]
    if qkv.shape[-1] != (nq + 2 * nkv) * hd:
        raise KernelError(f"rope_kv_write: qkv width {qkv.shape[1]} is not (nq+2nkv)*hd")
    if k_cache.dtype != out_dtype or v_cache.dtype != out_dtype:
        raise KernelError("rope_kv_write: the cache and the queries share one dtype")
    num_pages, nkv_c, page_size, hd_c = k_cache.shape
    if (nkv_c, hd_c) != (nkv, hd) or tuple(v_cache.shape) != tuple(k_cache.shape):
        raise KernelError(f"rope_kv_write: cache shape {tuple(k_cache.shape)} does not fit nkv={nkv} hd={hd}")
    max_pos = 0
    if rotary_dim:
        if table is None or table.dtype != torch.float32 or tuple(table.shape[1:]) != (2, rotary_dim // 2):
            raise KernelError("rope_kv_write: rotary table must be float32 [positions, 2, rotary_dim/2]")
        max_pos = table.shape[0]
    q = torch.empty((T, nq * hd), dtype=out_dtype, device=qkv.device)
    call("sllm_rope_kv_write", _p(qkv), _dt(qkv), parts, part_stride, _p(bias), _p(positions), _p(table), int(rotary_dim), max_pos,
         nq, nkv, hd, _p(slot_mapping), page_size, num_pages, _p(k_cache), _p(v_cache), _p(q), _dtc(out_dtype),
         T, _stream())
    return q


def _gate_args(gate):
    """(pointer to the first token's logit of head 0, row length) of a per-head output gate given as (float32 product, column)."""
    if gate is None:
        return None, 0
    t, off = gate
    if t.dtype != torch.float32 or t.dim() != 2:
        raise KernelError("attention: the heads' gates are columns of a float32 product")
    return _p(t) + 4 * int(off), t.shape[1]


class DistanceBias:
    """A bias on attention scores by the distance from key to query and the query head: ``by_distance`` ``[n, heads]``, one row per distance
    0 .. n-1, larger distances as the last one.  Held as ``table`` float32 ``[kv heads, n, heads of the group]`` (the rows a tile of
    (token, head) pairs reads for one key lie side by side) beside each head's largest value.  ``narrow``: no head's values lie
    further apart than `NARROW`, so that the largest may stand for a row's own maximum in a float32 softmax."""

    NARROW = 40.0

    def __init__(self, by_distance, nkv: int, device):
        n, nq = by_distance.shape
        t = by_distance.to(torch.float32)
        self.n = int(n)
        self.table = t.reshape(n, nkv, nq // nkv).permute(1, 0, 2).contiguous().to(device)
        self.top = t.max(0).values.contiguous().to(device)
        self.narrow = bool(((t.max(0).values - t.min(0).values) <= self.NARROW).all())

    def nbytes(self) -> int:
        return 4 * self.table.numel()

    def args(self):
        return _p(self.table), self.n, _p(self.top)


_NO_REL = (None, 0, None)


def attention_simt(q, k_cache, v_cache, block_tables, positions, seq_of_token, nq, nkv, hd, scale, window, block=None, sink=None,
                   softcap: float = 0.0, gate=None, rel: "DistanceBias | None" = None):
    """The CUDA-core attention kernel: any head size up to 640 (one instance to 256, one beyond), float32 arithmetic.  ``sink`` (float32 ``[nq]``): the
    softmax's denominator also holds exp(sink_h), a term without key or value that the scale does not touch.  ``softcap``, ``gate``:
    see `paged_attention`."""
    _chk(q, k_cache, v_cache, block_tables, positions, seq_of_token)
    T = q.shape[0]
    if q.dtype != k_cache.dtype:
        raise KernelError("attention: queries and cache share one dtype")
    page_size = k_cache.shape[2]
    out = torch.empty_like(q)
    call("sllm_attention_simt", _p(q), _p(k_cache), _p(v_cache), _dt(q), _p(block_tables),
         block_tables.shape[1], _p(positions), _p(seq_of_token), T, nq, nkv, hd, page_size, float(scale),
         int(window or 0), int(block or 0), _p(sink), float(softcap or 0.0), *_gate_args(gate), *(rel.args() if rel else _NO_REL)[:2],
         _p(out), _stream())
    return out


_num_sms: dict = {}


def num_sms() -> int:
    """Streaming multiprocessors of the current device (the library asks the driver, once per device):
    what the dispatch sizes k-splits and context splits for."""
    dev = _current_device() if _current_device is not None else torch.cuda.current_device()
    n = _num_sms.get(dev)
    if n is None:
        n = _num_sms[dev] = max(1, int(lib().sllm_num_sms()))
    return n


def attention_tiles(q_lens, group_size: int, device, ctx_lens=None, large_rows: int = 128):
    """Tiles of (token, head-in-group) rows for the tensor-core attention kernels: requests
    whose rows fit one 16-row tile go to the decode form, the others are cut into tiles of
    `large_rows` rows (128, or 256 for the tcgen05 form with two row tiles a CTA) for the
    prefill form.  Returns ``(small, large)``, each ``None`` or
    ``(tile_seq, tile_row0, count)`` on the device."""
    small_s, large_s, large_r = [], [], []
    ctx_before = [(c - n) for c, n in zip(ctx_lens, q_lens)] if ctx_lens else [0] * len(q_lens)
    for s, n in enumerate(q_lens):
        rows = n * group_size
        if rows <= 16:
            small_s.append(s)
        else:
            for r0 in range(0, rows, large_rows):
                large_s.append(s)
                large_r.append(r0)

    # the tiles with the most keys to walk first: a long tile that starts last would run alone
    order = sorted(range(len(large_s)), key=lambda i: -(large_r[i] // max(group_size, 1) + ctx_before[large_s[i]]))
    large_s, large_r = [large_s[i] for i in order], [large_r[i] for i in order]

    def up(seqs, rows):
        if not seqs:
            return None
        t = torch.tensor([seqs, rows], dtype=torch.int32).to(device, non_blocking=True)
        return t[0], t[1], len(seqs)
    return up(small_s, [0] * len(small_s)), up(large_s, large_r)


SPLIT_OVERHEAD_TILES = 3      # what a CTA of the decode form costs before and after its keys, in 64-key tiles
MAX_SPLITS = 128              # the merge kernel keeps one weight a range in shared memory
SPLIT_MIN_KEYS = 128          # a range has at least two key tiles (one request at 1,024 keys: 11.0 us in 4 ranges, 8.6 in 8)
MMA_MAX_SPLITS = 32           # the mma.sync form's merge walks the ranges one after the other


@functools.lru_cache(maxsize=4096)
def choose_splits(num_small: int, nkv: int, max_ctx: int, ctas_per_sm: int = 2, max_splits: int = 0) -> int:
    """How many ways the decode form cuts the context: the cut whose CTAs finish first, counted in waves of
    ``ctas_per_sm`` CTAs an SM times the 64-key tiles a CTA walks (plus its fixed cost); never less than
    ``SPLIT_MIN_KEYS`` keys a range, at most ``MAX_SPLITS`` ranges (one request at 32,768 keys and 4 KV heads: 74 ranges of 7 tiles
    fill the GPU once, where 32 ranges of 16 tiles left more than half of it idle).  A cut one CTA larger than a wave costs a whole second wave, so the
    number of ranges is not simply "two CTAs an SM"."""
    ctas = max(num_small * nkv, 1)
    slots = max(1, ctas_per_sm * num_sms())
    best, best_cost = 1, None
    for s in range(1, max(1, min(max_ctx // SPLIT_MIN_KEYS, max_splits or MAX_SPLITS)) + 1):
        tiles = -(-(-(-max_ctx // s)) // 64)              # the kernel rounds a range up to whole tiles
        if -(-max_ctx // (tiles * 64)) != s:              # so some counts leave their last ranges empty
            continue
        # (the last term: every range of every tile leaves a partial result that the merge reads again)
        cost = -(-ctas * s // slots) * (tiles + SPLIT_OVERHEAD_TILES) + 0.5 * ctas * s / slots
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return best


def attention_mma(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles, decode: bool, num_splits: int,
                  nq, nkv, hd, scale, window, out=None, block=None, sink=None, softcap: float = 0.0, gate=None, rel=None):
    """The tensor-core attention kernel on one tile list (see `attention_tiles`); the merge of a split context
    touches the rows of that list's requests only."""
    _chk(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles[0], tiles[1])
    if q.dtype != torch.bfloat16 or k_cache.dtype != torch.bfloat16:
        raise KernelError("attention_mma: bfloat16 only")
    T = q.shape[0]
    if out is None:
        out = torch.empty_like(q)
    part_o = part_lse = None
    if num_splits > 1:
        part_o = torch.empty((num_splits, T, nq, hd), dtype=torch.float32, device=q.device)
        part_lse = torch.empty((num_splits, T, nq), dtype=torch.float32, device=q.device)
    call("sllm_attention_mma", _p(q), _p(k_cache), _p(v_cache), _p(out), _p(part_o), _p(part_lse), _p(block_tables),
         block_tables.shape[1], _p(q_start), _p(ctx_len), _p(tiles[0]), _p(tiles[1]), tiles[2], 1 if decode else 0,
         num_splits, T, nq, nkv, hd, k_cache.shape[2], float(scale), int(window or 0), int(block or 0), _p(sink),
         float(softcap or 0.0), *_gate_args(gate), *(rel.args() if rel else _NO_REL)[:2], _stream())
    if num_splits > 1:
        launches["own"] += 1          # the combine kernel
    return out


@functools.lru_cache(maxsize=4096)
def tma_attention_supports(hd: int, page_size: int) -> bool:
    return bool(lib().sllm_attention_tma_supports(int(hd), int(page_size)))


@functools.lru_cache(maxsize=16)
def _tma_ctas_per_sm(hd: int) -> int:
    return int(lib().sllm_attention_tma_ctas_per_sm(int(hd)))


def attention_tma_decode(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles, num_splits: int,
                         nq, nkv, hd, scale, window, out=None, block=None, sink=None, softcap: float = 0.0, gate=None, rel=None):
    """The decode form fed by TMA (16-row tiles only; see `attention_tiles`)."""
    _chk(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles[0], tiles[1])
    if q.dtype != torch.bfloat16 or k_cache.dtype != torch.bfloat16:
        raise KernelError("attention_tma: bfloat16 only")
    T = q.shape[0]
    if out is None:
        out = torch.empty_like(q)
    part_o = part_lse = None
    if num_splits > 1:
        part_o = torch.empty((num_splits, T, nq, hd), dtype=torch.float32, device=q.device)
        part_lse = torch.empty((num_splits, T, nq), dtype=torch.float32, device=q.device)
    call("sllm_attention_tma_decode", _p(q), _p(k_cache), _p(v_cache), k_cache.shape[0], _p(out), _p(part_o),
         _p(part_lse), _p(block_tables), block_tables.shape[1], _p(q_start), _p(ctx_len), _p(tiles[0]), _p(tiles[1]),
         tiles[2], num_splits, T, nq, nkv, hd, k_cache.shape[2], float(scale), int(window or 0), int(block or 0),
         _p(sink), float(softcap or 0.0), *_gate_args(gate), *(rel.args() if rel else _NO_REL)[:2], _p(_status_word(q.device)), _stream())
    _tc_used["since_check"] += 1
    if num_splits > 1:
        launches["own"] += 1
    return out


_TC_ATTENTION = os.environ.get("SLLM_ATTENTION_TCGEN05", "1") != "0"     # 0: prompt portions on the mma.sync form


def wait_probe(limit_ns: int, device="cuda"):
    """Run the kernel that waits on a barrier nothing arrives at (see csrc/wait_probe.cu); returns
    ``(status, waited_ns)``: 99 and about ``limit_ns`` when the bounded wait gave up as it must."""
    status = torch.zeros(1, dtype=torch.int32, device=device)
    waited = torch.zeros(1, dtype=torch.int64, device=device)
    call("sllm_wait_probe", _p(status), int(limit_ns), _p(waited), _stream())
    return int(status.item()), int(waited.item())


@functools.lru_cache(maxsize=4096)
def tc_attention_supports(hd: int, page_size: int) -> bool:
    return bool(lib().sllm_attention_tc_supports(int(hd), int(page_size)))


@functools.lru_cache(maxsize=4096)
def choose_tc_splits(num_tiles: int, nkv: int, max_ctx: int) -> tuple[int, int]:
    """(ranges, 64-key tiles a range) for the prefill form: few row tiles over a long context are cut
    so that about two CTAs an SM run, each range at least 16 key tiles long."""
    key_tiles = max(1, -(-max_ctx // 64))
    ctas = max(num_tiles * nkv, 1)
    want = max(1, min(2 * num_sms() // ctas, key_tiles // 16, 32))
    per = -(-key_tiles // want)
    return -(-key_tiles // per), per


def attention_tc(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles, nq, nkv, hd, scale, out=None,
                 row_tiles: int = 1, splits: tuple[int, int] = (1, 0), parts=None, window=None, sink=None, softcap: float = 0.0, gate=None, rel=None):
    """The prefill form on tcgen05 (tiles of 128 * row_tiles rows, row_tiles 1 or 2; see
    `attention_tiles`).  ``splits`` = (ranges, 64-key tiles a range) cuts the context into ranges
    that run as CTAs of their own and are merged afterwards; ranges x tiles must cover the longest
    context among the tiles' requests.  ``parts`` = (row of ``block_tables``, first page) per sequence of ``q_start`` /
    ``ctx_len`` when these describe parts of requests (see `block_parts`)."""
    _chk(q, k_cache, v_cache, block_tables, q_start, ctx_len, tiles[0], tiles[1])
    if q.dtype != torch.bfloat16 or k_cache.dtype != torch.bfloat16:
        raise KernelError("attention_tc: bfloat16 only")
    if out is None:
        out = torch.empty_like(q)
    n_splits, per = int(splits[0]), int(splits[1])
    part_o = part_lse = None
    T = q.shape[0]
    if n_splits > 1:
        part_o = torch.empty((n_splits, T, nq, hd), dtype=torch.float32, device=q.device)
        part_lse = torch.full((n_splits, T, nq), float("-inf"), dtype=torch.float32, device=q.device)
        launches["library"] += 1           # the fill
    call("sllm_attention_tc", _p(q), _p(k_cache), _p(v_cache), k_cache.shape[0], _p(out), _p(block_tables),
         block_tables.shape[1], _p(q_start), _p(ctx_len), _p(tiles[0]), _p(tiles[1]), tiles[2], int(row_tiles), nq, nkv,
         hd, k_cache.shape[2], float(scale), int(window or 0), n_splits, max(per, 1), T, _p(part_o), _p(part_lse),
         _p(parts[0]) if parts else None, _p(parts[1]) if parts else None, _p(sink), float(softcap or 0.0), *_gate_args(gate),
         *(rel.args() if rel else _NO_REL), _p(_status_word(q.device)), _stream())
    if n_splits > 1:
        launches["own"] += 1               # the merge kernel
    _tc_used["since_check"] += 1
    return out


def block_parts(q_lens, ctx_lens, group_size: int, block: int, page_size: int, device, rows: int = 128):
    """Attention inside blocks of positions as ordinary causal attention over parts of requests: a request's portion is
    cut where it crosses a block's border; a part's keys start at its block's first position, which is the first position
    of a page (``block`` is a multiple of ``page_size``), so the part reads the request's block table from that page on.
    Requests of at most 16 (token, head-in-group) rows stay one part each and get no tile (the decode form runs them).
    Returns ``(q_start, ctx_len, (table_row, first_page), tiles)`` on the device, ``tiles`` as `attention_tiles` gives
    them for the prefill form, longest first."""
    starts, ctxs, rows_of, shift = [0], [], [], []
    tile_s, tile_r, keys = [], [], []
    for s, (n, c) in enumerate(zip(q_lens, ctx_lens)):
        pos0 = c - n
        cuts = [(pos0, c)] if n * group_size <= 16 else \
            [(max(pos0, b * block), min(c, (b + 1) * block)) for b in range(pos0 // block, (c - 1) // block + 1)]
        for lo, hi in cuts:
            first = lo // block * block if n * group_size > 16 else 0
            if n * group_size > 16:
                for r0 in range(0, (hi - lo) * group_size, rows):
                    tile_s.append(len(ctxs))
                    tile_r.append(r0)
                    keys.append(lo - first + r0 // group_size)
            starts.append(starts[-1] + hi - lo)
            ctxs.append(hi - first)
            rows_of.append(s)
            shift.append(first // page_size)
    order = sorted(range(len(tile_s)), key=lambda i: -keys[i])
    S = len(ctxs)
    flat = starts + ctxs + rows_of + shift + [tile_s[i] for i in order] + [tile_r[i] for i in order]
    t = torch.tensor(flat, dtype=torch.int32).to(device, non_blocking=True)
    n = len(tile_s)
    o = S + 1
    return (t[:o], t[o:o + S], (t[o + S:o + 2 * S], t[o + 2 * S:o + 3 * S]),
            (t[o + 3 * S:o + 3 * S + n], t[o + 3 * S + n:o + 3 * S + 2 * n], n))


@functools.lru_cache(maxsize=4096)
def mma_supports(hd: int) -> bool:
    return bool(lib().sllm_attention_mma_supports(int(hd)))


def paged_attention(q, k_cache, v_cache, step, group: int, nq, nkv, hd, scale, window, block=None, sink=None, softcap: float = 0.0,
                    gate=None, rel: "DistanceBias | None" = None):
    """Causal attention of the step's tokens over their requests' pages.  ``sink`` (float32 ``[nq]``): exp(sink_h) joins
    each head's softmax denominator (every form takes it).  ``softcap`` > 0: a score becomes softcap tanh(score / softcap) before
    the softmax; ``gate`` = (float32 product, column): head h's output times sigmoid of column + h; ``rel``: a bias on the scores by distance, added after scale and
    cap (every form takes all three).  ``window``: only the last ``window`` keys;
    ``block``: only the keys of the query's own block of ``block`` positions, counted from the sequence's start.  bfloat16 with a head size
    the tensor-core kernels take: requests of at most 16 (token, head-in-group) rows go to the decode
    form (fed by TMA where the head and page sizes allow, split over the context), the others to the
    prefill form in 128-row tiles (on tcgen05 where the sizes allow, else on mma.sync).  Otherwise the CUDA-core kernel."""
    g = step.groups[group]
    if q.dtype != torch.bfloat16 or not mma_supports(hd):
        return attention_simt(q, k_cache, v_cache, g.block_tables, step.positions, step.seq_of_token,
                              nq, nkv, hd, scale, window, block, sink, softcap, gate, rel)
    G = nq // nkv
    # blocks that start on page borders: the prefill form runs each block's part of a portion as a causal sequence of its own
    blocked_tc = bool(block) and block % k_cache.shape[2] == 0 and bool(step.ctx_lens)
    use_tc = (not block or (blocked_tc and not window)) and _TC_ATTENTION and tc_attention_supports(hd, k_cache.shape[2]) and \
        (rel is None or (rel.narrow and not block))
    key = ("mma", G, nkv, use_tc, block or 0, bool(window))
    if key not in step.attn_tiles:
        # 128-row CTAs, two per SM.  (The kernel also has a form with two row tiles a CTA, one CTA per SM,
        # that fetches each key/value tile once for 256 rows; measured at 28/4 heads of 128 it is the
        # slower one at every length: 106 against 99 us for 2048 tokens, 787 against 733 us for 8192.)
        rows = 128
        small, large = attention_tiles(step.q_lens, G, q.device, step.ctx_lens, rows)
        tma = tma_attention_supports(hd, k_cache.shape[2])
        per_sm = _tma_ctas_per_sm(hd) if tma else 2
        # the decode form's cut of the context, by the longest context among ITS requests (a step may also hold prompt
        # portions: their rows are the prefill form's, and the decode form's merge touches its own requests' rows only)
        splits = 1
        if small:
            small_ctx = max((c for c, n in zip(step.ctx_lens, step.q_lens) if n * G <= 16), default=step.max_ctx_len) \
                if step.ctx_lens else step.max_ctx_len
            splits = choose_splits(small[2], nkv, small_ctx, per_sm, 0 if tma else MMA_MAX_SPLITS)
        tc_splits = choose_tc_splits(large[2], nkv, step.max_ctx_len) if (large and use_tc and not block and not window) else (1, 0)
        parts = block_parts(step.q_lens, step.ctx_lens, G, block, k_cache.shape[2], q.device, rows) if (large and use_tc and block) else None
        step.attn_tiles[key] = (small, large, splits, rows, tc_splits, parts)
    small, large, splits, rows, tc_splits, parts = step.attn_tiles[key]
    out = torch.empty_like(q)
    if small and tma_attention_supports(hd, k_cache.shape[2]):
        attention_tma_decode(q, k_cache, v_cache, g.block_tables, step.q_start, step.ctx_len, small, splits,
                             nq, nkv, hd, scale, window, out, block, sink, softcap, gate, rel)
    elif small:
        attention_mma(q, k_cache, v_cache, g.block_tables, step.q_start, step.ctx_len, small, True, splits,
                      nq, nkv, hd, scale, window, out, block, sink, softcap, gate, rel)
    if large and use_tc and parts is not None:
        attention_tc(q, k_cache, v_cache, g.block_tables, parts[0], parts[1], parts[3], nq, nkv, hd, scale, out,
                     row_tiles=rows // 128, parts=parts[2], sink=sink, softcap=softcap, gate=gate)
    elif large and use_tc:
        attention_tc(q, k_cache, v_cache, g.block_tables, step.q_start, step.ctx_len, large, nq, nkv, hd, scale, out,
                     row_tiles=rows // 128, splits=tc_splits, window=window, sink=sink, softcap=softcap, gate=gate, rel=rel)
    elif large:
        attention_mma(q, k_cache, v_cache, g.block_tables, step.q_start, step.ctx_len, large, False, 1,
                      nq, nkv, hd, scale, window, out, block, sink, softcap, gate, rel)
    return out


_POOLED_MMA = os.environ.get("SLLM_POOLED_ATTENTION_MMA", "1") != "0"     # 0: the pooled-window attention on the CUDA cores (comparisons)


@functools.lru_cache(maxsize=4096)
def pooled_splits(num_small: int, nkv: int, max_ctx: int, window: int, pool: int) -> int:
    """Into how many runs of 64-key tiles the 16-row form of the pooled-window attention cuts a request's keys (the blocks'
    entries and the window's tokens): enough CTAs for two an SM, at least two tiles a run, at most 16 runs."""
    keys = min(window, max_ctx) if window else max_ctx
    tiles = -(-keys // 64) + 1 + (-(-(max_ctx // pool) // 64) if pool else 0)
    want = (2 * num_sms()) // max(1, num_small * nkv)
    return max(1, min(want, tiles // 2, 16))


def pool_kv_write(k_cache, v_cache, step, group: int, pk_cache, pv_cache, pool_group: int, pool: int) -> None:
    """The tokens of the step that complete a block of ``pool`` positions write the means of the block's cached keys and of
    its values (float32 sums in an order that depends on the block's length alone) into the pooled pages, at the places the step's description gives."""
    _chk(k_cache, v_cache, pk_cache, pv_cache)
    g, pg = step.groups[group], step.groups[pool_group]
    num_pages, nkv, page_size, D = k_cache.shape
    if tuple(pk_cache.shape[1:]) != (nkv, page_size, D) or pk_cache.dtype != k_cache.dtype:
        raise KernelError("pool_kv_write: the pooled pages have the token pages' heads, page size and dtype")
    call("sllm_pool_kv_write", _p(k_cache), _p(v_cache), _dt(k_cache), _p(g.block_tables), g.block_tables.shape[1], _p(step.positions),
         _p(step.seq_of_token), _p(pg.slot_mapping), _p(pk_cache), _p(pv_cache), pk_cache.shape[0], step.num_tokens, nkv, D,
         page_size, int(pool), _stream())


def pooled_attention(q, k_cache, v_cache, pk_cache, pv_cache, step, group: int, pool_group, nq: int, nkv: int, vdim: int, scale: float,
                     window, pool: int, sink=None, out_scale: float = 1.0, out=None, out_off: int = 0) -> torch.Tensor:
    """Softmax attention of the step's queries ``q [T, nq*D]`` over the last ``window`` cached tokens and, beside them, over
    the pooled entry of every block of ``pool`` positions that lies wholly before the window (``window`` None: all earlier
    tokens, no entries).  ``sink`` (float32 ``[nq]``): exp(sink_h) joins the denominator.  The result, times ``out_scale``,
    goes to columns ``out_off ..`` of ``out`` (made ``[T, nq*vdim]`` if not given), ``vdim`` value channels a head.
    bfloat16 with a head size the tensor-core kernel takes (16, 32, 64, 128) and columns in multiples of 4: the mma.sync
    forms; otherwise the CUDA-core kernel."""
    _chk(q, k_cache, v_cache, pk_cache, pv_cache, sink, out)
    g = step.groups[group]
    T = q.shape[0]
    num_pages, nkv_c, page_size, D = k_cache.shape
    if nkv_c != nkv or q.shape[1] != nq * D or q.dtype != k_cache.dtype:
        raise KernelError("pooled_attention: queries [T, nq*D] in the cache's dtype, a cache [pages, nkv, page_size, D]")
    if out is None:
        out = torch.empty((T, nq * vdim), dtype=q.dtype, device=q.device)
    pg = step.groups[pool_group] if (pool_group is not None and window) else None
    if _POOLED_MMA and q.dtype == torch.bfloat16 and mma_supports(D) and vdim % 4 == 0 and out.shape[1] % 4 == 0 and out_off % 4 == 0 \
            and step.q_lens:
        # tensor cores: requests of at most 16 (token, head-in-group) rows on the 16-row form, the others in 128-row tiles;
        # the blocks' entries are key tiles of their own in front of the window's
        G = nq // nkv
        key = ("pooled", G, nkv)
        if key not in step.attn_tiles:
            step.attn_tiles[key] = attention_tiles(step.q_lens, G, q.device, step.ctx_lens, 128)
        for tiles, decode in zip(step.attn_tiles[key], (True, False)):
            if tiles:
                splits, part_o, part_lse = 1, None, None
                if decode:
                    splits = pooled_splits(tiles[2], nkv, step.max_ctx_len, int(window or 0), int(pool or 0) if pg else 0)
                if splits > 1:
                    part_o = torch.empty((splits, T, nq, D), dtype=torch.float32, device=q.device)
                    part_lse = torch.empty((splits, T, nq), dtype=torch.float32, device=q.device)
                    launches["own"] += 1          # the merge kernel
                call("sllm_attention_mma_pooled", _p(q), _p(k_cache), _p(v_cache), _p(pk_cache) if pg else None,
                     _p(pv_cache) if pg else None, _p(out), _p(g.block_tables), g.block_tables.shape[1],
                     _p(pg.block_tables) if pg else None, pg.block_tables.shape[1] if pg else 0, _p(step.q_start), _p(step.ctx_len),
                     _p(tiles[0]), _p(tiles[1]), tiles[2], 1 if decode else 0, splits, _p(part_o), _p(part_lse), T, nq, nkv, D,
                     int(vdim), page_size, float(scale),
                     int(window or 0), int(pool or 0) if pg else 0, _p(sink), float(out_scale), out.shape[1], int(out_off), _stream())
        return out
    call("sllm_attention_pooled_simt", _p(q), _p(k_cache), _p(v_cache), _p(pk_cache) if pg else None, _p(pv_cache) if pg else None,
         _dt(q), _p(g.block_tables), g.block_tables.shape[1], _p(pg.block_tables) if pg else None,
         pg.block_tables.shape[1] if pg else 0, _p(step.positions), _p(step.seq_of_token), T, nq, nkv, D, int(vdim), page_size,
         float(scale), int(window or 0), int(pool or 0), _p(sink), float(out_scale), _p(out), out.shape[1], int(out_off), _stream())
    return out


def gather_rows(x: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
    """``x[rows]``; a 3-d ``x`` is a stack of partial sums, added while gathering."""
    _chk(x, rows)
    parts, stride = 1, 0
    if x.dim() == 3:
        parts, stride = x.shape[0], x.shape[1] * x.shape[2]
    R, (n, H) = rows.numel(), x.shape[-2:]
    out = torch.empty((R, H), dtype=x.dtype, device=x.device)
    call("sllm_gather_rows", _p(x), _dt(x), parts, stride, _p(rows), _p(out), R, H, n, _stream())
    return out


def sample_rows(logits: torch.Tensor, temperature=None, uniform=None, top_k=None, top_p=None) -> torch.Tensor:
    """int32 token per row of float32 ``logits [R, V]``: the first maximum where the
    row's temperature is <= 0 (or none is given), else inverse-CDF sampling of
    softmax(logits / temperature) at the row's uniform (float64), over the tokens that
    the row's ``top_k`` (int32, <= 0: no filter) and then ``top_p`` (float32, < 0: no
    filter) keep."""
    _chk(logits, temperature, uniform, top_k, top_p)
    R, V = logits.shape
    if logits.dtype != torch.float32:
        raise KernelError("sample_rows: logits are float32")
    if temperature is not None and (temperature.dtype != torch.float32 or uniform is None
                                    or uniform.dtype != torch.float64):
        raise KernelError("sample_rows: temperature float32 and uniform float64, one per row")
    if (top_k is not None or top_p is not None) and temperature is None:
        raise KernelError("sample_rows: top_k/top_p filter sampled rows; give temperatures")
    if (top_k is not None and (top_k.dtype != torch.int32 or top_k.numel() != R)) or \
            (top_p is not None and (top_p.dtype != torch.float32 or top_p.numel() != R)):
        raise KernelError("sample_rows: top_k int32 and top_p float32, one per row")
    out = torch.empty((R,), dtype=torch.int32, device=logits.device)
    call("sllm_sample_rows", _p(logits), R, V, _p(temperature), _p(uniform), _p(top_k), _p(top_p), _p(out), _stream())
    return out


def repetition_penalty_(logits: torch.Tensor, pair_row, pair_id, pair_penalty) -> torch.Tensor:
    """In place on float32 ``logits [R, V]``: for each (row, id, penalty) triple a positive
    logit is divided by the penalty and a negative one multiplied.  A (row, id) pair must
    appear once; ids outside the vocabulary are ignored."""
    _chk(logits, pair_row, pair_id, pair_penalty)
    R, V = logits.shape
    n = pair_row.numel()
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise KernelError("repetition_penalty_: logits are contiguous float32")
    if pair_row.dtype != torch.int32 or pair_id.dtype != torch.int32 or pair_penalty.dtype != torch.float32 \
            or pair_id.numel() != n or pair_penalty.numel() != n:
        raise KernelError("repetition_penalty_: rows and ids int32, penalties float32, one per pair")
    call("sllm_repetition_penalty", _p(logits), R, V, _p(pair_row), _p(pair_id), _p(pair_penalty), n, _stream())
    return logits


def mark_seen(seen: torch.Tensor, step) -> None:
    """Record the step's tokens in ``seen [slots, V]`` (uint8): ``seen[slot of the token's request,
    token id] = 1``.  ``step`` is the `StepContext` (token ids, request of each token, state slots,
    all on the device)."""
    _chk(seen, step.token_ids, step.seq_of_token, step.state_slots)
    if seen.dtype != torch.uint8 or seen.dim() != 2:
        raise KernelError("mark_seen: the table is uint8 [slots, V]")
    call("sllm_mark_seen", _p(seen), seen.shape[0], seen.shape[1], _p(step.token_ids), _p(step.seq_of_token),
         _p(step.state_slots), int(step.num_tokens), _stream())


def penalty_from_seen_(logits: torch.Tensor, seen: torch.Tensor, step, penalty: torch.Tensor) -> torch.Tensor:
    """The repetition penalty in place on float32 ``logits [R, V]`` (row r belongs to the request of
    token ``step.logit_rows[r]``): every id that request has seen has a positive logit divided by
    ``penalty[r]`` and a negative one multiplied; rows with penalty 0 or 1 stay as they are."""
    _chk(logits, seen, penalty, step.logit_rows, step.seq_of_token, step.state_slots)
    R, V = logits.shape
    if logits.dtype != torch.float32 or seen.dtype != torch.uint8 or seen.shape[1] != V:
        raise KernelError("penalty_from_seen_: float32 logits [R, V] and a uint8 table [slots, V]")
    if penalty.dtype != torch.float32 or penalty.numel() != R or step.logit_rows.numel() < R:
        raise KernelError("penalty_from_seen_: one float32 penalty and one wanted row per logits row")
    call("sllm_penalty_seen", _p(logits), R, V, _p(seen), seen.shape[0], _p(step.logit_rows), _p(step.seq_of_token),
         _p(step.state_slots), _p(penalty), _stream())
    return logits
