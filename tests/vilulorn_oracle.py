"""Plain statement of the Vilulorn decoder: one function per mechanism, whole sequences, no cache, float64 by default.

Written from the equations alone and sharing no code with the package; the tests compare the framework with it.  ``weights`` is a
dict of tensors under the checkpoint's names, ``cfg`` the config.json dictionary.
"""
import math

import torch


def linear(w, x):
    """W x for a batch of rows: ``w`` [out, in], ``x`` [rows, in]."""
    return x @ w.to(x.dtype).T


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


def rotary_frequencies(rot):
    """One frequency per rotated pair: base^(-2i/dims), long wavelengths slowed down by ``factor``, a linear blend in between."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, positions, rot):
    """x [n, heads, dim]: dimensions 2i and 2i + 1 turn by position * frequency i; those beyond rot['dims'] stay."""
    out = x.clone()
    for i, f in enumerate(rotary_frequencies(rot)):
        a = positions.to(torch.float64) * f
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(n, size):
    """[n, n] bool: query i sees key j of its own chunk of ``size`` positions."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    return see & (i // size == j // size) if size else see


def keys_values(h, w, prefix, mx, eps):
    n = h.shape[0]
    k = linear(w[prefix + "k"], h).reshape(n, mx["kv_heads"], mx["dim"])
    k = rotate(rms_norm(k, w[prefix + "k.norm"], eps), torch.arange(n), mx["rot"])
    return k, linear(w[prefix + "v"], h).reshape(n, mx["kv_heads"], -1)


def chunked_core(q, k, v, gate, mx):
    """The rows ``q`` [n, heads, dim] are the last n of the len(k) tokens; ``gate`` [n, heads * vdim] before its sigmoid."""
    n, L, H = q.shape[0], k.shape[0], mx["heads"]
    see = visible(L, (mx.get("mask") or {}).get("size"))[L - n:]
    per = H // mx["kv_heads"]
    heads = []
    for h in range(H):
        s = q[:, h] @ k[:, h // per].T * mx["scale"]
        heads.append(torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, h // per])
    return torch.cat(heads, dim=-1) * torch.sigmoid(gate)


def attention(h, w, prefix, mx, eps, shared):
    """``shared``: keys and values of the layer named by kv_from, None where the layer has its own.  Returns (output, (k, v))."""
    n = h.shape[0]
    q = linear(w[prefix + "q"], h).reshape(n, mx["heads"], mx["dim"])
    q = rotate(rms_norm(q, w[prefix + "q.norm"], eps), torch.arange(n), mx["rot"])
    kv = shared if shared is not None else keys_values(h, w, prefix, mx, eps)
    o = chunked_core(q, kv[0], kv[1], linear(w[prefix + "g"], h), mx)
    return linear(w[prefix + "o"], o), kv


def gla_log_decay(z, tau):
    """log of sigmoid(z)^(1 / tau)"""
    return torch.nn.functional.logsigmoid(z) / tau


def gla_recurrence(q, k, v, log_decay, state):
    """q (scaled), k, log_decay [n, H, dim], v [n, H, vdim]; token by token.  Returns (o [n, H, vdim], the last state)."""
    out, S = torch.zeros_like(v), state
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t])[..., None] * S + k[t][..., None] * v[t][:, None, :]
        out[t] = (S * q[t][..., None]).sum(1)
    return out, S


def gla_finish(o, gate, norm_w, eps):
    """Norm of every head's output and the gate: o [n, H, vdim], gate [n, H * vdim]."""
    y = rms_norm(o, norm_w, eps).reshape(o.shape[0], -1)
    return y * gate * torch.sigmoid(gate)


def gla(h, w, prefix, mx, eps):
    n, H, D, V = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = linear(w[prefix + "q"], h).reshape(n, H, D) * D ** -0.5
    k = linear(w[prefix + "k"], h).reshape(n, H, D)
    v = linear(w[prefix + "v"], h).reshape(n, H, V)
    z = linear(w[prefix + "a2"], linear(w[prefix + "a1"], h)) + w[prefix + "a2.b"].to(h.dtype)
    o, _ = gla_recurrence(q, k, v, gla_log_decay(z.reshape(n, H, D), mx["tau"]), torch.zeros(H, D, V, dtype=h.dtype))
    return linear(w[prefix + "o"], gla_finish(o, linear(w[prefix + "g"], h), w[prefix + "norm"], eps))


def expert(x, w, prefix, limit):
    g = torch.clamp(linear(w[prefix + "gate"], x), max=limit)
    u = torch.clamp(linear(w[prefix + "up"], x), min=-limit, max=limit)
    return linear(w[prefix + "down"], g * torch.sigmoid(1.702 * g) * (u + 1.0))


def moe(h, w, prefix, mlp):
    """Sigmoid scores, the best ``top`` of them; the score scales the expert's input."""
    s = torch.sigmoid(linear(w[prefix + "router"], h))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in torch.argsort(s[t], descending=True)[:mlp["router"]["top"]].tolist():
            out[t] += expert(s[t, e] * h[t:t + 1], w, f"{prefix}e{e}.", mlp["expert"]["limit"])[0]
    return out


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out``: a list that collects the residual after every layer."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, cached = cfg["norm"]["eps"], {}
    x = w["embed"][tokens].to(dtype) + w["pos"][:len(tokens)].to(dtype)
    for i, spec in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", spec["mixer"]
        if spec["type"] == "gla":
            y = gla(x, w, p + "mix.", mx, eps)
        else:
            y, cached[i] = attention(x, w, p + "mix.", mx, eps, cached[mx["kv_from"]] if mx.get("kv_from") is not None else None)
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if spec.get("mlp") is not None:
            x = x + rms_norm(moe(x, w, p + "mlp.", spec["mlp"]), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(w["head"], rms_norm(x, w["final.norm"], eps))


def random_weights(cfg, seed=0, scale=1.0, rank=16):
    """bfloat16 weights of the right names and shapes (norm weights around one); ``rank``: inner width of the decay projections."""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, n, k, s=1.0):
        w[name] = (torch.randn(n, k, generator=g) * (s * scale / k ** 0.5)).to(torch.bfloat16)

    def norm(name, n, mean=1.0):
        w[name] = (mean + 0.2 * torch.randn(n, generator=g)).to(torch.bfloat16)

    w["embed"] = torch.randn(V, E, generator=g).to(torch.bfloat16)
    w["pos"] = (0.3 * torch.randn(cfg["max_positions"], E, generator=g)).to(torch.bfloat16)
    for i, spec in enumerate(cfg["layers"]):
        p, mx, ff = f"l{i}.", spec["mixer"], spec.get("mlp")
        H, D, Vd = mx["heads"], mx["dim"], mx["vdim"]
        norm(p + "norm1", E)
        mat(p + "mix.q", H * D, E)
        mat(p + "mix.g", H * Vd, E)
        mat(p + "mix.o", E, H * Vd)
        if spec["type"] == "gla":
            mat(p + "mix.k", H * D, E)
            mat(p + "mix.v", H * Vd, E)
            norm(p + "mix.norm", Vd)
            mat(p + "mix.a1", rank, E)
            mat(p + "mix.a2", H * D, rank, 2.0)
            norm(p + "mix.a2.b", H * D, 0.5)
        else:
            norm(p + "mix.q.norm", D, 1.5)
            if mx.get("kv_from") is None:
                mat(p + "mix.k", mx["kv_heads"] * D, E)
                mat(p + "mix.v", mx["kv_heads"] * Vd, E)
                norm(p + "mix.k.norm", D, 1.5)
        if ff is None:
            continue
        norm(p + "norm2", E)
        mat(p + "mlp.router", ff["router"]["experts"], E)
        for e in range(ff["router"]["experts"]):
            mat(f"{p}mlp.e{e}.gate", ff["expert"]["ff"], E, 1.5)
            mat(f"{p}mlp.e{e}.up", ff["expert"]["ff"], E, 1.5)
            mat(f"{p}mlp.e{e}.down", E, ff["expert"]["ff"])
    norm("final.norm", E)
    mat("head", V, E)
    return w
