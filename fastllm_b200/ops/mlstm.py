"""Matrix-memory LSTM: a ``[dim, vdim]`` fp32 state S and a normaliser row n per head and request, under a running maximum m.

    m' = max(f + m, i) ,  S <- e^(f + m - m') S + e^(i - m') k v^T ,  n <- e^(f + m - m') n + e^(i - m') k
    out = S^T q / (max(|n . q|, e^(-m')) + 1e-6)

with one log input gate i = cap tanh(z_i / cap) and one log forget gate f = log sigmoid(cap tanh(z_f / cap)) per head and token, followed by
an RMS norm of every head's output and ``* sigmoid(gate)``.  The states live in the engine's state slots, a row ``[S | n | m]`` per head.

* decoded tokens, short portions, float32 models, widths outside the tiling: ``csrc/mlstm.cu::mlstm_recurrent_kernel`` walks a request's
  tokens with the state in registers -- gates, update, read-out, norm and output gate in one launch;
* longer portions: the chunked form (``mlstm_chunk_*``, tensor cores): the state's increment of every 128 tokens, a scan over them, and
  the outputs from the chunk's first state and the weighted scores inside the chunk.
"""
from __future__ import annotations

import ctypes

import torch
import torch.nn.functional as F

from . import _lib
from . import latent as LA
from . import stream32 as S
from .basic import _ptr, _stream

P, I, FLT, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_mlstm_recurrent": [P, LL, P, LL, P, P, P, LL, P, P, P, LL, I, I, I, I, I, I, I, FLT, FLT, FLT, I, P],
    "fb_mlstm_chunked": [P, LL, I, P, LL, P, P, P, LL, P, I, P, I, P, P, P, P, P, P, P, LL, I, I, I, I, I, I, I, I, FLT, FLT, FLT, I, P],
}, ["mlstm"])

CHUNK = 128
ROW_TOKENS = 16                  # requests that bring at most this many tokens walk them one by one
SCRATCH_BYTES = 1 << 30          # chunk states held at once; more heads than fit run in groups


def state_len(dim: int, vdim: int) -> int:
    """fp32 values of one head's state row [S | n | m]."""
    return (dim * vdim + dim + 1 + 3) // 4 * 4


class MLSTMWeights:
    def __init__(self):
        self.heads = self.dim = self.vdim = 0
        self.cap = 1.0
        self.in_proj = None      # rows [queries | keys | values | output gate], every part a multiple of 8 rows
        self.gate_b = None       # fp32 [2 heads]: biases of the input gates, then of the forget gates
        self.norm = None         # [heads * vdim]
        self.cols = (0, 0, 0, 0)


def build(spec, q, k, v, g, i_b, f_b, norm):
    """(MLSTMWeights without ``in_proj``, merged input projection matrix) from the layer's matrices."""
    w = MLSTMWeights()
    w.heads, w.dim, w.vdim, w.cap = spec.heads, spec.dim, spec.vdim, float(spec.gate_cap)
    w.gate_b, w.norm = torch.cat([i_b, f_b]).float().contiguous(), norm
    parts = [LA.pad_rows(m, 8) for m in (q, k, v, g)]
    cols = [0]
    for m in parts[:-1]:
        cols.append(cols[-1] + m.shape[0])
    w.cols = tuple(cols)
    return w, LA.pad_rows(torch.cat(parts, dim=0), 32)


def chunk_ok(w, dtype) -> bool:
    if dtype not in (torch.float16, torch.bfloat16):
        return False
    ok = w.__dict__.get("_chunk_ok")
    if ok is None:
        ok = w._chunk_ok = bool(_lib.kernels()._lib.fb_mlstm_chunk_supported(w.dim, w.vdim))
    return ok


class _Plan:
    """Requests of a batch that are walked token by token, and the chunks of the others."""

    def __init__(self, fb, chunked: bool):
        dev, cu, slots = fb.page_table.device, fb.cu_q_host, fb.state_slots_host
        items, chunks, reqs = [], [], []
        for b, s in enumerate(slots):
            n = cu[b + 1] - cu[b]
            if n <= 0:
                continue
            if not chunked or n <= ROW_TOKENS:
                items.append((cu[b], n, s))
                continue
            reqs.append((len(chunks), (n + CHUNK - 1) // CHUNK, s))
            chunks += [(cu[b] + c, min(CHUNK, n - c), s if c + CHUNK >= n else -1) for c in range(0, n, CHUNK)]
        self.n_items, self.n_chunks, self.n_reqs = len(items), len(chunks), len(reqs)
        meta = torch.tensor([x for part in (items, chunks, reqs) for t in part for x in t], dtype=torch.int32).to(dev, non_blocking=True)
        self.items, self.chunks, self.reqs = meta.split([3 * self.n_items, 3 * self.n_chunks, 3 * self.n_reqs])


def _recurrent(w, proj, gates, state, slots, items, n, out, eps) -> None:
    _, kc, vc, gc = w.cols
    rc = _lib.kernels().fb_mlstm_recurrent(_ptr(proj), proj.stride(0), _ptr(gates), gates.stride(0), _ptr(w.gate_b), _ptr(w.norm), _ptr(state),
                                           state.stride(1), _ptr(slots), _ptr(items), _ptr(out), out.stride(0), n, w.heads, w.dim, w.vdim, kc, vc, gc,
                                           w.dim ** -0.5, w.cap, float(eps), S.act_code(proj.dtype), _stream())
    _lib.check(rc, "fb_mlstm_recurrent")


def _chunked(w, proj, gates, state, pl, out, eps) -> None:
    _, kc, vc, gc = w.cols
    D, V, Dp, dev = w.dim, w.vdim, (w.dim + 15) // 16 * 16, proj.device
    per_head = pl.n_chunks * (D * V + 2 * D + 3 * CHUNK + 4)                     # floats beside the 16-bit states
    step = max(1, min(w.heads, SCRATCH_BYTES // (4 * per_head + 4 * pl.n_chunks * Dp * V)))
    units = pl.n_chunks * step
    inc, ninc, n0, lg, m0 = torch.empty((units * (D * V + 2 * D + 3 * CHUNK + 1),), device=dev, dtype=torch.float32).split(
        [units * D * V, units * D, units * D, units * 3 * CHUNK, units])
    s0 = (torch.empty if Dp == D else torch.zeros)((units * 2 * Dp * V,), device=dev, dtype=proj.dtype)
    for h0 in range(0, w.heads, step):
        rc = _lib.kernels().fb_mlstm_chunked(_ptr(proj), proj.stride(0), proj.shape[0], _ptr(gates), gates.stride(0), _ptr(w.gate_b), _ptr(w.norm),
                                             _ptr(state), state.stride(1), _ptr(pl.chunks), pl.n_chunks, _ptr(pl.reqs), pl.n_reqs, _ptr(inc), _ptr(ninc),
                                             _ptr(lg), _ptr(m0), _ptr(n0), _ptr(s0), _ptr(out), out.stride(0), w.heads, h0, min(step, w.heads - h0), D, V,
                                             kc, vc, gc, D ** -0.5, w.cap, float(eps), S.act_code(proj.dtype), _stream())
        _lib.check(rc, "fb_mlstm_chunked")


def mix(w: MLSTMWeights, proj, gates, fb, state, eps: float, out=None):
    """``proj`` [T, >= all parts], ``gates`` fp32 logits [T, 2 heads] (without bias) -> normalised, gated heads [T, heads * vdim] (``out``, where
    given); advances ``state`` [slots, heads, state_len] (fp32) of every request of the batch."""
    T = proj.shape[0]
    if not proj.is_cuda:
        y = mix_ref(w, proj, gates, fb, state, eps)
        return y if out is None else out.copy_(y)
    if out is None:
        out = torch.empty((T, w.heads * w.vdim), device=proj.device, dtype=proj.dtype)
    if fb.is_decode:
        _recurrent(w, proj, gates, state, fb.state_slots, None, fb.state_slots.shape[0], out, eps)
        return out
    plans, ok = fb.__dict__.setdefault("_mlstm_plans", {}), chunk_ok(w, proj.dtype)
    pl = plans.get(ok) or plans.setdefault(ok, _Plan(fb, ok))
    if pl.n_items:
        _recurrent(w, proj, gates, state, None, pl.items, pl.n_items, out, eps)
    if pl.n_chunks:
        _chunked(w, proj, gates, state, pl, out, eps)
    return out


def mix_ref(w: MLSTMWeights, proj, gates, fb, state, eps: float):
    """PyTorch evaluation, token by token (CPU tensors)."""
    T, H, D, V = proj.shape[0], w.heads, w.dim, w.vdim
    qc, kc, vc, gc = w.cols
    pf = proj.float()
    q, k = pf[:, qc:qc + H * D].reshape(T, H, D) * D ** -0.5, pf[:, kc:kc + H * D].reshape(T, H, D)
    v, g = pf[:, vc:vc + H * V].reshape(T, H, V), pf[:, gc:gc + H * V]
    z = torch.tanh((gates.float() + w.gate_b) / w.cap) * w.cap
    ig, fg = z[:, :H], F.logsigmoid(z[:, H:])
    o = torch.empty((T, H, V), dtype=torch.float32)
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    for b, slot in enumerate(fb.state_slots.tolist()):
        St, n, m = state[slot, :, :D * V].unflatten(1, (D, V)), state[slot, :, D * V:D * V + D], state[slot, :, D * V + D]
        for t in range(cu[b], cu[b + 1]):
            mn = torch.maximum(fg[t] + m, ig[t])
            keep, add = torch.exp(fg[t] + m - mn), torch.exp(ig[t] - mn)
            St.mul_(keep[:, None, None]).add_((add[:, None] * k[t])[..., None] * v[t][:, None, :])
            n.mul_(keep[:, None]).add_(add[:, None] * k[t])
            m.copy_(mn)
            den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mn)) + 1e-6
            o[t] = torch.einsum("hdv,hd->hv", St, q[t]) / den[:, None]
    y = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
    return (y.reshape(T, -1) * w.norm.float() * torch.sigmoid(g)).to(proj.dtype)
