"""Python entry points of ``csrc/parallel_mixers.cu``: layers that add a mixer and a feed-forward of the same fp32 stream (sums,
norms and the mixer's input filter in one or two kernels), attention rows with whole-row norms and rotation, and the delta
rule with separate removal and decay vectors.

Conventions of ``mixer_ops``: every wrapper has a PyTorch branch with identical semantics (CPU execution), CUDA tensors always
take the kernel; ``seq_info`` is int32 ``[n_seqs, 4]`` = (first row, rows, tokens seen, state slot).
"""
from __future__ import annotations

from typing import Optional, Tuple

import torch

from ....native import lib as _lib
from .mixer_ops import _rms, _rows, rotate_heads

_lib.register({
    "sxb_resid_sum_step": "pppppp" "ff" "pppppppppp" "iii" "i" "p",
    "sxb_norm_filter_rows": "pppppppppp" "iiii" "i" "p",
    "sxb_rope_append": "p" "l" "iii" "pppppppppp" "iiiiiiiii" "ff" "i" "p",
    "sxb_removal_prepare": "p" "l" "iiiii" "pppp" "iiii" "ff" "i" "p",
    "sxb_removal_recurrence": "pppp" "iiii" "p",
})


# ------------------------------------------------------------------------------------------------ stream + norms
class StreamSum:
    """What a finished layer has yet to add to the stream: ``y`` as it is, and ``mult * (rms_norm(a) * wa + rms_norm(b) * wb)``
    (without ``wa``: ``a`` as it is).  Any part may be None."""
    __slots__ = ("y", "a", "wa", "b", "wb", "mult")

    def __init__(self, y=None, a=None, wa=None, b=None, wb=None, mult: float = 1.0):
        self.y, self.a, self.wa, self.b, self.wb, self.mult = y, a, wa, b, wb, mult

    def value(self, rows: Optional[torch.Tensor], eps: float):
        def pick(t):
            return t.float() if rows is None else t.index_select(0, rows.long()).float()
        out = 0.0
        if self.y is not None:
            out = out + pick(self.y)
        if self.a is not None:
            if self.wa is None:
                out = out + pick(self.a)
            else:
                out = out + self.mult * _rms(pick(self.a), eps) * self.wa.float()
        if self.b is not None:
            out = out + self.mult * _rms(pick(self.b), eps) * self.wb.float()
        return out


_NOTHING = StreamSum()


def _resid_sum(resid, add: StreamSum, eps, dtype, n_rows, rstd=None, rows=None, w1=None, out=None, w2=None, out2=None,
               filt=None, state=None, seq_info=None, tok_seq=None):
    p = _lib.ptr
    _lib.call("sxb_resid_sum_step", resid.data_ptr(), p(add.y), p(add.a), p(add.wa), p(add.b), p(add.wb), float(add.mult),
              float(eps), p(rstd), p(rows), p(w1), p(out), p(w2), p(out2), p(filt), p(state), p(seq_info), p(tok_seq),
              filt.shape[0] if filt is not None else 1, int(n_rows), resid.shape[1], _lib.dtype_code(dtype),
              _lib.stream_ptr())


def stream_add(resid: torch.Tensor, add: StreamSum, eps: float, dtype: torch.dtype) -> None:
    """In place on the fp32 stream ``[T, W]``: add what is pending."""
    if resid.is_cuda:
        _resid_sum(resid, add, eps, dtype, resid.shape[0])
    else:
        resid += add.value(None, eps)


def stream_norm_rows(resid: torch.Tensor, add: Optional[StreamSum], rows: torch.Tensor, w: torch.Tensor, eps: float,
                     dtype: torch.dtype) -> torch.Tensor:
    """``rms_norm(resid[rows] + add[rows]) * w`` in ``dtype``; the stream itself is left as it is."""
    add = add or _NOTHING
    if resid.is_cuda:
        out = torch.empty(rows.numel(), resid.shape[1], dtype=dtype, device=resid.device)
        _resid_sum(resid, add, eps, dtype, rows.numel(), rows=rows, w1=w, out=out)
        return out
    return (_rms(resid.index_select(0, rows.long()) + add.value(rows, eps), eps) * w.float()).to(dtype)


def open_parallel_layer(resid: torch.Tensor, add: Optional[StreamSum], w_mix: torch.Tensor, filt: torch.Tensor,
                        state: Optional[torch.Tensor], w_ff: Optional[torch.Tensor], eps: float, dtype: torch.dtype,
                        seq_info: torch.Tensor, tok_seq: torch.Tensor, single_rows: bool
                        ) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """Close the layer before (``resid += add``, in place) and compute both inputs of a layer whose mixer and feed-forward
    read the same stream: ``(h + filter(h), rms_norm(resid) * w_ff)`` with ``h = rms_norm(resid) * w_mix``.  The causal filter
    ``filt`` ``[taps, W]`` (last row = current token) runs over each sequence's ``h``; ``state`` fp32 ``[slots, taps-1, W]``
    carries its last ``taps - 1`` rows (None for one tap).  ``single_rows``: every sequence has exactly one row here -- one
    kernel; otherwise the sums and row norms are one kernel, the two outputs another."""
    T, W = resid.shape
    add = add or _NOTHING
    taps = filt.shape[0]
    if resid.is_cuda:
        out = torch.empty(T, W, dtype=dtype, device=resid.device)
        out2 = torch.empty(T, W, dtype=dtype, device=resid.device) if w_ff is not None else None
        if single_rows:
            _resid_sum(resid, add, eps, dtype, T, w1=w_mix, out=out, w2=w_ff, out2=out2, filt=filt, state=state,
                       seq_info=seq_info, tok_seq=tok_seq)
            return out, out2
        rstd = torch.empty(T, dtype=torch.float32, device=resid.device)
        _resid_sum(resid, add, eps, dtype, T, rstd=rstd)
        _lib.call("sxb_norm_filter_rows", resid.data_ptr(), rstd.data_ptr(), w_mix.data_ptr(), filt.data_ptr(),
                  _lib.ptr(state), seq_info.data_ptr(), tok_seq.data_ptr(), out.data_ptr(), _lib.ptr(w_ff), _lib.ptr(out2), T,
                  seq_info.shape[0], W, taps, _lib.dtype_code(dtype), _lib.stream_ptr())
        return out, out2
    if add is not _NOTHING:
        resid += add.value(None, eps)
    normed = _rms(resid, eps)
    h = normed * w_mix.float()
    keep = taps - 1
    out = torch.empty_like(h)
    f = filt.float()
    for first, n, seen, slot in seq_info.tolist():
        hist = torch.zeros(keep, W) if (seen == 0 or keep == 0) else state[slot].clone()
        if 0 < seen < keep:
            hist[: keep - seen] = 0
        full = torch.cat([hist, h[first: first + n]])
        acc = h[first: first + n].clone()
        for j in range(taps):
            acc += f[j] * full[j: j + n]
        out[first: first + n] = acc
        if keep > 0:
            state[slot] = full[-keep:]
    return out.to(dtype), (normed * w_ff.float()).to(dtype) if w_ff is not None else None


# ------------------------------------------------------------------------------------------------ attention rows
def rope_append(proj: torch.Tensor, q0: int, k0: int, v0: int, q_w: Optional[torch.Tensor], k_w: Optional[torch.Tensor],
                inv_freq: torch.Tensor, interleaved: bool, q_scale: Optional[torch.Tensor], kcache: torch.Tensor,
                vcache: torch.Tensor, tok_seq: torch.Tensor, tok_pos: torch.Tensor, tables: torch.Tensor, Hq: int, G: int,
                d: int, dv: int, eps: float, amp: float = 1.0) -> torch.Tensor:
    """q (``Hq d`` columns at ``q0``), k (``G d`` at ``k0``) and v (``G dv`` at ``v0``; ``v0 = k0``: the values are the projected
    keys, untouched) of projection rows.  With ``q_w`` / ``k_w`` (``[Hq d]`` / ``[G d]``) the whole row of q / k is divided by its
    root mean square and multiplied by the weight.  The first ``2 len(inv_freq)`` channels of every head turn by ``pos *
    inv_freq[i]``: pairs ``(2i, 2i+1)`` if ``interleaved``, else ``(i, i + len(inv_freq))``, cos and sin times ``amp``.  Returns q fp32 ``[T, Hq, d]`` times
    ``q_scale`` (fp32 ``[Hq]``); k and v go to the paged caches ``[pages, block, G, d | dv]``."""
    T = proj.shape[0]
    bs = kcache.shape[1]
    n_rot = 2 * inv_freq.numel()
    if proj.is_cuda:
        if kcache.dtype != proj.dtype or vcache.dtype != proj.dtype:
            raise ValueError("the caches have the projection's dtype")
        q = torch.empty(T, Hq, d, dtype=torch.float32, device=proj.device)
        _lib.call("sxb_rope_append", _rows(proj).data_ptr(), proj.stride(0), int(q0), int(k0), int(v0), _lib.ptr(q_w),
                  _lib.ptr(k_w), inv_freq.data_ptr() if n_rot else None, _lib.ptr(q_scale), q.data_ptr(), kcache.data_ptr(),
                  vcache.data_ptr(), tok_seq.data_ptr(), tok_pos.data_ptr(), tables.data_ptr(), T, tables.shape[1], bs, Hq, G,
                  d, dv, n_rot, int(interleaved), float(eps), float(amp), _lib.dtype_code(proj.dtype), _lib.stream_ptr())
        return q
    x = proj.float()
    q, k = x[:, q0: q0 + Hq * d], x[:, k0: k0 + G * d]
    v = proj[:, v0: v0 + G * dv].reshape(T, G, dv)
    if q_w is not None:
        q = _rms(q, eps) * q_w.float()
    if k_w is not None:
        k = _rms(k, eps) * k_w.float()
    q = rotate_heads(q.reshape(T, Hq, d), tok_pos, inv_freq, interleaved, amp)
    k = rotate_heads(k.reshape(T, G, d), tok_pos, inv_freq, interleaved, amp)
    if q_scale is not None:
        q = q * q_scale.float()[:, None]
    page = tables[tok_seq.long(), (tok_pos // bs).long()].long()
    off = (tok_pos % bs).long()
    kcache[page, off] = k.to(kcache.dtype)
    vcache[page, off] = v.to(vcache.dtype)
    return q.contiguous()


# ------------------------------------------------------------------------------------------------ delta rule with removal
def removal_prepare(proj: torch.Tensor, r0: int, k0: int, v0: int, a0: int, low0: int, w2: torch.Tensor, w0: torch.Tensor,
                    a_bias: torch.Tensor, H: int, n: int, rate: float, eps: float) -> torch.Tensor:
    """fp32 ``[T, H, 5, n]`` = ``w | u | a | r | v'`` from projection rows (r, k, v, a: ``H n`` columns each; ``w2.shape[0]`` columns
    at ``low0``): ``w = exp(-rate * sigmoid(tanh(low) w2 + w0))``, ``u = k / sqrt(sum k^2 + eps)`` per head, ``a = sigmoid(a +
    a_bias)``, ``v' = v * sqrt(sum k^2 + eps)``.  ``w2`` ``[rank, H n]`` in the projection's dtype, ``w0`` / ``a_bias`` fp32."""
    T, rank, Hn = proj.shape[0], w2.shape[0], H * n
    if proj.is_cuda:
        if w2.dtype != proj.dtype or w0.dtype != torch.float32 or a_bias.dtype != torch.float32 or not w2.is_contiguous():
            raise ValueError("w2 is contiguous in the projection's dtype, w0 and a_bias are fp32")
        buf = torch.empty(T, H, 5, n, dtype=torch.float32, device=proj.device)
        _lib.call("sxb_removal_prepare", _rows(proj).data_ptr(), proj.stride(0), int(r0), int(k0), int(v0), int(a0), int(low0),
                  w2.data_ptr(), w0.data_ptr(), a_bias.data_ptr(), buf.data_ptr(), T, H, n, rank, float(rate), float(eps),
                  _lib.dtype_code(proj.dtype), _lib.stream_ptr())
        return buf
    x = proj.float()
    r, k, v, a = (x[:, c: c + Hn].reshape(T, H, n) for c in (r0, k0, v0, a0))
    w = torch.exp(-rate * torch.sigmoid(torch.tanh(x[:, low0: low0 + rank]) @ w2.float() + w0)).reshape(T, H, n)
    length = torch.sqrt(k.pow(2).sum(-1, keepdim=True) + eps)
    return torch.stack([w, k / length, torch.sigmoid(a + a_bias.reshape(H, n)), r, v * length], dim=2)


def removal_recurrence(buf: torch.Tensor, state: torch.Tensor, seq_info: torch.Tensor, single_rows: bool = False
                       ) -> torch.Tensor:
    """Per sequence and head, rows in order, with ``w | u | a | r | v'`` from :func:`removal_prepare`: ``S <- diag(w) S - (a u)
    (u^T S) + u v'^T`` (both products read the old ``S``), ``o = S^T r``.  ``state`` fp32 ``[slots, H, n (value), n (key)]`` is read
    (zero for a sequence that has seen no token) and written back.  Returns fp32 ``[T, H n]``."""
    T, H, _, n = buf.shape
    if buf.is_cuda:
        out = torch.empty(T, H * n, dtype=torch.float32, device=buf.device)
        _lib.call("sxb_removal_recurrence", buf.data_ptr(), state.data_ptr(), out.data_ptr(), seq_info.data_ptr(),
                  seq_info.shape[0], H, n, int(single_rows), _lib.stream_ptr())
        return out
    out = torch.empty(T, H, n)
    for first, rows, seen, slot in seq_info.tolist():
        S = state[slot].clone() if seen > 0 else torch.zeros_like(state[slot])           # [H, value, key]
        for t in range(first, first + rows):
            w, u, a, r, v = buf[t].unbind(1)                                              # [H, n] each
            z = torch.einsum("hvn,hn->hv", S, u)
            S = S * w[:, None, :] + u[:, None, :] * (v[:, :, None] - a[:, None, :] * z[:, :, None])
            out[t] = torch.einsum("hvn,hn->hv", S, r)
        state[slot] = S
    return out.reshape(T, H * n)
