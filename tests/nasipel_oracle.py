"""Plain statement of the Nasipel decoder: one function per mechanism, whole sequences, no cache, float64 by default.

Written from the equations alone and sharing no code with the package; the tests compare the framework with it.  ``weights`` is a
dict of tensors under the checkpoint's names, ``cfg`` the config.json dictionary.
"""
import math

import torch


def linear(w, x):
    """W x for a batch of rows: ``w`` [out, in], ``x`` [rows, in]."""
    return x @ w.to(x.dtype).T


def biased(w, name, h):
    return linear(w[name], h) + w[name + ".b"].to(h.dtype)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w.to(x.dtype)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ---- rotations ------------------------------------------------------------------------------------
def plain_freqs(dims, base):
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_freqs(dims, base, sc):
    """Frequencies between f / factor (slow pairs) and f (fast ones), and the factor of both cosine and sine."""
    dim = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_freqs(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def turn(x, positions, freqs, halves, sign=1.0, mag=1.0):
    """x [n, heads, >= 2 * len(freqs)]: pair i turns by sign * position * freqs[i]; pairs (i, i + len) or (2i, 2i + 1)."""
    n = len(freqs)
    ang = sign * positions.to(torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    c, s = (mag * torch.cos(ang)).to(x.dtype)[:, None], (mag * torch.sin(ang)).to(x.dtype)[:, None]
    first, second = (slice(0, n), slice(n, 2 * n)) if halves else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
    u, v, out = x[..., first], x[..., second], x.clone()
    out[..., first], out[..., second] = u * c - v * s, v * c + u * s
    return out


# ---- attention with sigmoid weights and rotated values --------------------------------------------
def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def sigmoid_attention(q, k, v, mx, bias):
    """Rows q [n, H, dim] are the last n of the len(k) tokens: weights sigmoid(score + bias[h]) over all keys up to the query."""
    n, L, per = q.shape[0], k.shape[0], mx["heads"] // mx["kv_heads"]
    see = torch.arange(L)[None, :] <= torch.arange(L - n, L)[:, None]
    out = []
    for h in range(mx["heads"]):
        s = capped(q[:, h] @ k[:, h // per].T * mx["scale"], mx.get("softcap"))
        p = torch.sigmoid(s + bias[h].to(s.dtype)) * see
        out.append(p @ v[:, h // per])
    return torch.stack(out, dim=1)


def attention(h, w, p, mx, eps):
    n, pos = h.shape[0], torch.arange(h.shape[0])
    q = linear(w[p + "q"], h).reshape(n, mx["heads"], mx["dim"])
    k = linear(w[p + "k"], h).reshape(n, mx["kv_heads"], mx["dim"])
    v = linear(w[p + "v"], h).reshape(n, mx["kv_heads"], mx["vdim"])
    fr, fv = plain_freqs(mx["rot"]["dims"], mx["rot"]["base"]), plain_freqs(mx["vdim"], mx["rot"]["base"])
    q, k = unit_rms(turn(q, pos, fr, True), eps), unit_rms(turn(k, pos, fr, True), eps)
    o = sigmoid_attention(q, k, turn(v, pos, fv, True), mx, w[p + "pb"])
    return linear(w[p + "o"], turn(o, pos, fv, True, sign=-1.0).reshape(n, -1))


# ---- latent attention ------------------------------------------------------------------------------
def latent_attention(h, w, p, mx, eps):
    n, H, D, R, V, pos = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], torch.arange(h.shape[0])
    q = linear(w[p + "uq"], rms_norm(linear(w[p + "dq"], h), w[p + "dq.norm"], eps)).reshape(n, H, D + R)
    kv = linear(w[p + "dkv"], h)
    c, kr = rms_norm(kv[:, :mx["kv_rank"]], w[p + "dkv.norm"], eps), kv[:, mx["kv_rank"]:].reshape(n, 1, R)
    rot = mx["rot"]
    fr, mag = yarn_freqs(R, rot["base"], rot["scaling"]) if rot.get("scaling") else (plain_freqs(R, rot["base"]), 1.0)
    qr, kr = turn(q[..., D:], pos, fr, False, mag=mag), turn(kr, pos, fr, False, mag=mag)[:, 0]
    k, v = linear(w[p + "uk"], c).reshape(n, H, D), linear(w[p + "uv"], c).reshape(n, H, V)
    see = torch.arange(n)[None, :] <= torch.arange(n)[:, None]
    out = []
    for i in range(H):
        s = (q[:, i, :D] @ k[:, i].T + qr[:, i] @ kr.T) * mx["scale"]
        out.append(torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1) @ v[:, i])
    o = torch.stack(out, dim=1) * torch.sigmoid(linear(w[p + "g"], h))[..., None]
    return linear(w[p + "o"], o.reshape(n, -1))


# ---- real-gated linear recurrent unit ---------------------------------------------------------------
def causal_conv(x, taps, bias, before=None):
    """x [n, C], taps [C, K] (the last column is the current token's), ``before`` [K - 1, C]: what precedes x (zeros)."""
    K = taps.shape[1]
    pad = before if before is not None else torch.zeros(K - 1, x.shape[1], dtype=x.dtype)
    xx = torch.cat([pad, x], dim=0)
    return sum(xx[i:i + x.shape[0]] * taps[:, i].to(x.dtype) for i in range(K)) + bias.to(x.dtype)


def block_gate(u, m, b):
    """sigmoid of every equal part of ``u`` times its own square matrix."""
    n, B = u.shape[0], m.shape[0]
    parts = u.reshape(n, B, -1)
    return torch.sigmoid(torch.cat([linear(m[i], parts[:, i]) + b[i].to(u.dtype) for i in range(B)], dim=1))


def rglru_recurrence(u, r, i, lam, state=None):
    """Token by token; returns (all states [n, width], the last one)."""
    S = torch.zeros(u.shape[1], dtype=u.dtype) if state is None else state
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * torch.nn.functional.softplus(lam.to(u.dtype))
        a = torch.exp(log_a)
        S = a * S + torch.sqrt(1.0 - a * a) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(h, w, p, mx, eps):
    y = gelu_tanh(biased(w, p + "y", h))
    u = causal_conv(biased(w, p + "x", h), w[p + "conv"], w[p + "conv.b"])
    S, _ = rglru_recurrence(u, block_gate(u, w[p + "ra"], w[p + "ra.b"]), block_gate(u, w[p + "ri"], w[p + "ri.b"]), w[p + "lam"])
    return linear(w[p + "o"], S * y)


MIXERS = {"attention": attention, "latent_attention": latent_attention, "rglru": rglru}


# ---- feed-forward ------------------------------------------------------------------------------------
def expert(h, w, p):
    return linear(w[p + "down"], silu(linear(w[p + "gate"], h)) * linear(w[p + "up"], h))


def choose(choice, router):
    """Experts of one token from its choice scores [experts]."""
    gr, E = router.get("groups"), choice.shape[0]
    ok = torch.ones(E, dtype=torch.bool)
    if gr:
        per = E // gr["count"]
        score = torch.stack([choice[g * per:(g + 1) * per].sort(descending=True).values[:2].sum() for g in range(gr["count"])])
        ok = torch.zeros(E, dtype=torch.bool)
        for g in torch.argsort(score, descending=True)[:gr["keep"]].tolist():
            ok[g * per:(g + 1) * per] = True
    return torch.argsort(choice.masked_fill(~ok, float("-inf")), descending=True)[:router["top"]].tolist()


def moe(h, w, p, mlp):
    r = mlp["router"]
    s = torch.sigmoid(linear(w[p + "router"], h))
    weight = torch.zeros_like(s)                                       # [tokens, experts], zero where an expert is not chosen
    for t in range(h.shape[0]):
        picked = choose(s[t] + w[p + "correction"].to(s.dtype), r)
        weight[t, picked] = s[t, picked] / (s[t, picked].sum() + 1e-20) * r.get("scale", 1.0)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows = weight[:, e].nonzero()[:, 0]
        out[rows] += weight[rows, e:e + 1] * expert(h[rows], w, f"{p}e{e}.")
    return out


# ---- the model ---------------------------------------------------------------------------------------
def layer(x, w, p, spec, eps):
    h = layer_norm(x, w[p + "norm1"], eps)
    y = MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], eps) * torch.sigmoid(biased(w, p + "rg1", h))
    if spec.get("mlp"):
        h2 = layer_norm(x, w[p + "norm2"], eps)
        y = y + moe(h2, w, p + "mlp.", spec["mlp"]) * torch.sigmoid(biased(w, p + "rg2", h2))
    return x + y


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out``: a list that collects the residual after every layer."""
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)].to(dtype)
    eps = cfg["norm"]["eps"]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, w, f"l{i}.", spec, eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(w["head"], layer_norm(x, w["final.norm"], eps))


def random_weights(cfg, seed=0, scale=1.0):
    """bfloat16 weights of the right names and shapes (norm weights around one)."""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, n, k, s=1.0):
        w[name] = (torch.randn(n, k, generator=g) * (s * scale / k ** 0.5)).to(torch.bfloat16)

    def vec(name, n, mean=1.0, s=0.2):
        w[name] = (mean + s * torch.randn(n, generator=g)).to(torch.bfloat16)

    w["embed"] = torch.randn(V, E, generator=g).to(torch.bfloat16)
    for i, spec in enumerate(cfg["layers"]):
        p, mx, ff = f"l{i}.", spec["mixer"], spec.get("mlp")
        vec(p + "norm1", E)
        mat(p + "rg1", E, E, 1.5)
        vec(p + "rg1.b", E, 0.5, 0.5)
        if spec["type"] == "rglru":
            W, n = mx["width"], mx["width"] // mx["blocks"]
            for z in "yx":
                mat(p + "mix." + z, W, E)
                vec(p + f"mix.{z}.b", W, 0.2, 0.3)
            mat(p + "mix.conv", W, mx["conv"], 1.2)
            vec(p + "mix.conv.b", W, 0.0, 0.3)
            for z in ("ra", "ri"):
                w[p + "mix." + z] = (torch.randn(mx["blocks"], n, n, generator=g) * 1.5 / n ** 0.5).to(torch.bfloat16)
                w[p + f"mix.{z}.b"] = (0.5 * torch.randn(mx["blocks"], n, generator=g)).to(torch.bfloat16)
            w[p + "mix.lam"] = torch.linspace(-7.0, 0.5, W)[torch.randperm(W, generator=g)].to(torch.bfloat16)      # memories of one to thousands of tokens
            mat(p + "mix.o", E, W, 1.5)
        elif spec["type"] == "latent_attention":
            H, D, R, Vd = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
            mat(p + "mix.dq", mx["q_rank"], E)
            vec(p + "mix.dq.norm", mx["q_rank"], 1.3)
            mat(p + "mix.uq", H * (D + R), mx["q_rank"])
            mat(p + "mix.dkv", mx["kv_rank"] + R, E, 1.3)
            vec(p + "mix.dkv.norm", mx["kv_rank"])
            mat(p + "mix.uk", H * D, mx["kv_rank"])
            mat(p + "mix.uv", H * Vd, mx["kv_rank"], 1.5)
            mat(p + "mix.g", H, E, 1.5)
            mat(p + "mix.o", E, H * Vd, 1.5)
        else:
            H, G = mx["heads"], mx["kv_heads"]
            mat(p + "mix.q", H * mx["dim"], E)
            mat(p + "mix.k", G * mx["dim"], E)
            mat(p + "mix.v", G * mx["vdim"], E)
            vec(p + "mix.pb", H, -3.0, 0.5)
            mat(p + "mix.o", E, H * mx["vdim"], 0.5)
        if ff:
            vec(p + "norm2", E)
            mat(p + "rg2", E, E, 1.5)
            vec(p + "rg2.b", E, 0.5, 0.5)
            n, f = ff["router"]["experts"], ff["expert"]["ff"]
            mat(p + "mlp.router", n, E, 1.5)
            vec(p + "mlp.correction", n, -0.4, 0.5)
            for e in range(n):
                mat(p + f"mlp.e{e}.gate", f, E, 1.5)
                mat(p + f"mlp.e{e}.up", f, E)
                mat(p + f"mlp.e{e}.down", E, f)
    vec("final.norm", E)
    mat("head", V, E)
    return w
