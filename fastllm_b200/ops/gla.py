"""Gated linear attention: a ``[dim, vdim]`` fp32 state S per head and request whose key channels d forget at their own data-dependent rate.

    S[d, :] <- f[d] S[d, :] + k[d] v ,   f[d] = sigmoid(z[d])^(1 / tau) ,   out = sum_d q[d] S[d, :]

with decay logits z from a low-rank projection of the layer's input, followed by an RMS norm of every head's output and ``* silu(gate)``.  The states live in the engine's state slots.

* decoded tokens, float32 models, widths outside the tiling: ``csrc/gla.cu::gla_recurrent_kernel`` walks a request's tokens with the
  state in registers -- decay, update, read-out, norm and gate in one launch;
* prompt portions: the chunked form (``gla_chunk_*``): per 64 tokens the state's increment, a scan over the chunks' increments, and the
  outputs from the chunk's first state and the decayed products inside the chunk.  Cumulative log-decays are only ever subtracted
  forwards in time, so no exponential exceeds one.
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
    "fb_gla_recurrent": [P, LL, P, P, P, P, P, P, P, LL, I, I, I, I, I, I, I, I, I, FLT, FLT, FLT, I, P],
    "fb_gla_chunked": [P, LL, P, P, P, P, P, I, P, I, P, P, P, P, LL, I, I, I, I, I, I, I, I, I, I, FLT, FLT, FLT, I, P],
}, ["gla"])

CHUNK = 64
SCRATCH_BYTES = 1 << 30          # chunk states held at once; more heads than fit run in groups


class GLAWeights:
    def __init__(self):
        self.heads = self.dim = self.vdim = self.rank = 0
        self.tau = 1.0
        self.in_proj = None      # rows [queries | keys | values | gate | decay rank], every part a multiple of 8 rows
        self.a2 = self.a2_b = self.norm = None
        self.cols = (0, 0, 0, 0, 0)


def build(spec, q, k, v, g, a1, a2, a2_b, norm):
    """(GLAWeights without ``in_proj``, merged input projection matrix) from the layer's matrices."""
    w = GLAWeights()
    w.heads, w.dim, w.vdim, w.rank, w.tau = spec.heads, spec.dim, spec.vdim, a1.shape[0], float(spec.tau)
    w.a2, w.a2_b, w.norm = a2, a2_b, norm
    parts = [LA.pad_rows(m, 8) for m in (q, k, v, g, a1)]
    cols = [0]
    for m in parts[:-1]:
        cols.append(cols[-1] + m.shape[0])
    w.cols = tuple(cols)
    return w, LA.pad_rows(torch.cat(parts, dim=0), 32)


def chunk_ok(w, dtype) -> bool:
    return dtype in (torch.float16, torch.bfloat16) and w.dim <= 256 and w.vdim <= 256 and w.dim % 8 == 0 and w.vdim % 8 == 0 and w.rank <= 64


class _ChunkPlan:
    def __init__(self, fb):
        dev, cu, slots = fb.page_table.device, fb.cu_q_host, fb.state_slots_host
        chunks, reqs = [], []
        for b, s in enumerate(slots):
            n = cu[b + 1] - cu[b]
            if n > 0:
                reqs.append((len(chunks), (n + CHUNK - 1) // CHUNK, s))
                chunks += [(cu[b] + c, min(CHUNK, n - c)) for c in range(0, n, CHUNK)]
        self.n_chunks, self.n_reqs = len(chunks), len(reqs)
        meta = torch.tensor([x for t in chunks for x in t] + [x for t in reqs for x in t], dtype=torch.int32).to(dev, non_blocking=True)
        self.chunks, self.reqs = meta[:2 * len(chunks)], meta[2 * len(chunks):]


def mix(w: GLAWeights, proj, fb, state, eps: float):
    """``proj`` [T, >= all parts] -> gated, normalised heads [T, heads * vdim]; advances ``state`` [slots, heads, dim, vdim] (fp32) of every
    request of the batch."""
    T = proj.shape[0]
    if not proj.is_cuda:
        return mix_ref(w, proj, fb, state, eps)
    out = torch.empty((T, w.heads * w.vdim), device=proj.device, dtype=proj.dtype)
    qc, kc, vc, gc, ac = w.cols
    if fb.is_decode or not chunk_ok(w, proj.dtype):
        cu = None if fb.is_decode else fb.cu_q
        rc = _lib.kernels().fb_gla_recurrent(_ptr(proj), proj.stride(0), _ptr(w.a2), _ptr(w.a2_b), _ptr(w.norm), _ptr(state), _ptr(fb.state_slots), _ptr(cu),
                                             _ptr(out), out.stride(0), fb.state_slots.shape[0], w.heads, w.dim, w.vdim, w.rank, kc, vc, gc, ac,
                                             w.dim ** -0.5, 1.0 / w.tau, float(eps), S.act_code(proj.dtype), _stream())
        _lib.check(rc, "fb_gla_recurrent")
        return out
    pl = fb.__dict__.get("_gla_plan")
    if pl is None:
        pl = fb._gla_plan = _ChunkPlan(fb)
    sizes = [pl.n_chunks * w.dim * CHUNK, pl.n_chunks * w.dim * w.vdim, pl.n_chunks * w.dim]      # log-decays, increments, chunk decays
    per_head = sum(sizes)
    step = max(1, min(w.heads, SCRATCH_BYTES // (4 * per_head)))
    lg, inc, dec = torch.empty((per_head * step,), device=proj.device, dtype=torch.float32).split([x * step for x in sizes])
    for h0 in range(0, w.heads, step):
        rc = _lib.kernels().fb_gla_chunked(_ptr(proj), proj.stride(0), _ptr(w.a2), _ptr(w.a2_b), _ptr(w.norm), _ptr(state), _ptr(pl.chunks), pl.n_chunks,
                                           _ptr(pl.reqs), pl.n_reqs, _ptr(inc), _ptr(dec), _ptr(lg), _ptr(out), out.stride(0), w.heads, h0,
                                           min(step, w.heads - h0), w.dim, w.vdim, w.rank, kc, vc, gc, ac, w.dim ** -0.5, 1.0 / w.tau, float(eps),
                                           S.act_code(proj.dtype), _stream())
        _lib.check(rc, "fb_gla_chunked")
    return out


def mix_ref(w: GLAWeights, proj, fb, state, eps: float):
    """PyTorch evaluation, token by token (CPU tensors)."""
    T, H, D, V = proj.shape[0], w.heads, w.dim, w.vdim
    qc, kc, vc, gc, ac = w.cols
    pf = proj.float()
    q, k = pf[:, qc:qc + H * D].reshape(T, H, D) * D ** -0.5, pf[:, kc:kc + H * D].reshape(T, H, D)
    v, g = pf[:, vc:vc + H * V].reshape(T, H, V), pf[:, gc:gc + H * V]
    z = pf[:, ac:ac + w.rank] @ w.a2.float().t() + w.a2_b.float()
    alpha = torch.exp(F.logsigmoid(z) / w.tau).reshape(T, H, D)
    o = torch.empty((T, H, V), dtype=torch.float32)
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    for b, slot in enumerate(fb.state_slots.tolist()):
        St = state[slot]
        for t in range(cu[b], cu[b + 1]):
            St.mul_(alpha[t][..., None]).add_(k[t][..., None] * v[t][:, None, :])
            o[t] = torch.einsum("hdv,hd->hv", St, q[t])
    return (S._rms(o, w.norm, eps).reshape(T, -1) * F.silu(g)).to(proj.dtype)
