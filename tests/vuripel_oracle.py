"""Plain statement of the Vuripel decoder: one function per mechanism, whole sequences, no cache, float64 by default.

Written from the equations alone and sharing no code with the package; the tests compare the framework with it.  ``weights`` is a
dict of tensors under the checkpoint's names, ``cfg`` the config.json dictionary.
"""
import math

import torch


def linear(w, x):
    """W x for a batch of rows: ``w`` [out, in], ``x`` [rows, in]."""
    return x @ w.to(x.dtype).T


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w.to(x.dtype)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def rotate(x, positions, rot):
    """x [n, heads, dim]: dimensions i and i + dims/2 turn by position * base^(-2i/dims); those beyond rot['dims'] stay."""
    out, half = x.clone(), rot["dims"] // 2
    for i in range(half):
        a = positions.to(torch.float64) * rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def visible(n, mask=None):
    """[n, n] bool: query i sees key j <= i that is less than ``size`` away or among the first ``keep_first``."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    if mask and mask.get("size"):
        see = see & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return see


def capped(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def softmax_with_sink(s, sink=None):
    """Rows of scores; a sink adds exp(sink) to the denominator and nothing to the numerator."""
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink.to(s.dtype))
    e = torch.exp(s - m)
    z = e.sum(-1, keepdim=True)
    return e / (z if sink is None else z + torch.exp(sink.to(s.dtype) - m))


def attention_core(q, k, v, mx, sinks=None):
    """The rows ``q`` [n, heads, dim] are the last n of the len(k) tokens; returns [n, heads, vdim]."""
    n, L, H = q.shape[0], k.shape[0], mx["heads"]
    see = visible(L, mx.get("mask"))[L - n:]
    per = H // mx["kv_heads"]
    heads = []
    for h in range(H):
        s = capped(q[:, h] @ k[:, h // per].T * mx["scale"], mx.get("softcap"))
        heads.append(softmax_with_sink(s.masked_fill(~see, float("-inf")), sinks[h] if sinks is not None else None) @ v[:, h // per])
    return torch.stack(heads, dim=1)


def biased(w, name, h):
    return linear(w[name], h) + w[name + ".b"].to(h.dtype)


def attention(h, w, p, mx, eps):
    """Causal, no positions, a sink in every head's softmax, one output gate per head."""
    n = h.shape[0]
    q = biased(w, p + "q", h).reshape(n, mx["heads"], mx["dim"])
    k = biased(w, p + "k", h).reshape(n, mx["kv_heads"], mx["dim"])
    v = biased(w, p + "v", h).reshape(n, mx["kv_heads"], mx["vdim"])
    o = attention_core(q, k, v, mx, w[p + "sink"]) * torch.sigmoid(linear(w[p + "g"], h))[..., None]
    return linear(w[p + "o"], o.reshape(n, -1))


def attention_2(h, w, p, mx, eps):
    """Normalised and rotated queries and keys, a sliding window beside the first tokens, no sink, no gate."""
    n, pos = h.shape[0], torch.arange(h.shape[0])
    q = biased(w, p + "q", h).reshape(n, mx["heads"], mx["dim"])
    k = biased(w, p + "k", h).reshape(n, mx["kv_heads"], mx["dim"])
    v = biased(w, p + "v", h).reshape(n, mx["kv_heads"], mx["vdim"])
    q = rotate(rms_norm(q, w[p + "q.norm"], eps), pos, mx["rot"])
    k = rotate(rms_norm(k, w[p + "k.norm"], eps), pos, mx["rot"])
    return linear(w[p + "o"], attention_core(q, k, v, mx).reshape(n, -1))


def mlstm_recurrence(q, k, v, i_gate, log_f, state=None):
    """q (scaled), k [n, H, dim], v [n, H, vdim], log gates [n, H]; token by token.  Returns (o [n, H, vdim], (S, nrm, m))."""
    n, H, D = q.shape
    if state is None:
        state = (torch.zeros(H, D, v.shape[2], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    S, nr, m = state
    out = torch.zeros_like(v)
    for t in range(n):
        m_new = torch.maximum(log_f[t] + m, i_gate[t])
        keep, add = torch.exp(log_f[t] + m - m_new), torch.exp(i_gate[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        nr = keep[:, None] * nr + add[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((nr * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    return out, (S, nr, m)


def mlstm_gates(h, w, p, cap):
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(biased(w, p + "i", h)), torch.nn.functional.logsigmoid(soft(biased(w, p + "f", h)))


def mlstm(h, w, p, mx, eps):
    n, H, D, V = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = linear(w[p + "q"], h).reshape(n, H, D) * D ** -0.5
    k = linear(w[p + "k"], h).reshape(n, H, D)
    v = linear(w[p + "v"], h).reshape(n, H, V)
    o, _ = mlstm_recurrence(q, k, v, *mlstm_gates(h, w, p, mx["gate_cap"]))
    y = unit_rms(o, eps).reshape(n, H * V) * w[p + "norm"].to(h.dtype) * torch.sigmoid(linear(w[p + "g"], h))
    return linear(w[p + "o"], y)


MIXERS = {"attention": attention, "attention_2": attention_2, "mlstm": mlstm}


def dense(h, w, p):
    return linear(w[p + "down"], gelu_tanh(linear(w[p + "gate"], h)) * linear(w[p + "up"], h))


def expert(h, w, p):
    return linear(w[p + "down"], gelu_erf(linear(w[p + "up"], h)))


def choose(s, router):
    """Experts of one token from its scores ``s`` [experts]."""
    gr = router.get("groups")
    E = s.shape[0]
    ok = torch.ones(E, dtype=torch.bool)
    if gr:
        per = E // gr["count"]
        best = torch.argsort(torch.stack([s[g * per:(g + 1) * per].max() for g in range(gr["count"])]), descending=True)[:gr["keep"]]
        ok = torch.zeros(E, dtype=torch.bool)
        for g in best.tolist():
            ok[g * per:(g + 1) * per] = True
    return torch.argsort(torch.where(ok, s, torch.full_like(s, -1.0)), descending=True)[:router["top"]].tolist()


def moe(h, w, p, mlp):
    s = torch.softmax(linear(w[p + "router"], h), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose(s[t], mlp["router"]):
            out[t] += s[t, e] * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(linear(w[p + "shared.sg"], h)) * expert(h, w, p + "shared.")
    return out


def token_input(x, w, p, e, eps):
    y = linear(w[p + "proj"], gelu_tanh(linear(w[p + "gate"], x)) * e)
    return x + rms_norm(y, w[p + "norm"], eps)


def order(cfg):
    """(layer, pass or None where no loop pass starts) of every layer run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    return ([(i, None) for i in range(a)] + [(i, t if i == a else None) for t in range(lp["times"]) for i in range(a, b)]
            + [(i, None) for i in range(b, n)])


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out``: a list that collects the residual after every layer run."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    first = x = w["embed"][tokens].to(dtype)
    ts = cfg.get("token_side")
    for i, start in order(cfg):
        if start is not None:
            x = (x + first if start > 0 else x) + w["loop.step"][start].to(dtype)
        spec, p = cfg["layers"][i], f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        y = MIXERS[spec["type"]](h, w, p + "mix.", spec["mixer"], eps)
        ff = spec.get("mlp")
        if ff is not None:
            y = y + (dense(h, w, p + "mlp.") if ff["kind"] == "dense" else moe(h, w, p + "mlp.", ff))
        x = x + y
        if ts:
            e = w["side.embed"][tokens, i * ts["dim"]:(i + 1) * ts["dim"]].to(dtype)
            x = token_input(x, w, p + "side.", e, eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(w["head"], rms_norm(x, w["final.norm"], eps))


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
    ts, lp = cfg.get("token_side"), cfg.get("loop")
    if lp:
        w["loop.step"] = (0.3 * torch.randn(lp["times"], E, generator=g)).to(torch.bfloat16)
    if ts:
        w["side.embed"] = torch.randn(V, len(cfg["layers"]) * ts["dim"], generator=g).to(torch.bfloat16)
    for i, spec in enumerate(cfg["layers"]):
        p, mx, ff = f"l{i}.", spec["mixer"], spec.get("mlp")
        H, D, Vd = mx["heads"], mx["dim"], mx["vdim"]
        vec(p + "norm1", E)
        mat(p + "mix.q", H * D, E)
        mat(p + "mix.o", E, H * Vd)
        if spec["type"] == "mlstm":
            mat(p + "mix.k", H * D, E)
            mat(p + "mix.v", H * Vd, E)
            mat(p + "mix.g", H * Vd, E)
            vec(p + "mix.norm", H * Vd)
            for z, mean in (("i", -0.5), ("f", 3.0)):
                mat(p + "mix." + z, H, E, 2.0)
                vec(p + f"mix.{z}.b", H, mean, 1.0)
        else:
            mat(p + "mix.k", mx["kv_heads"] * D, E)
            mat(p + "mix.v", mx["kv_heads"] * Vd, E)
            for z, n in (("q", H * D), ("k", mx["kv_heads"] * D), ("v", mx["kv_heads"] * Vd)):
                vec(p + f"mix.{z}.b", n, 0.0, 0.4)
            if spec["type"] == "attention":
                vec(p + "mix.sink", H, 0.5, 1.0)
                mat(p + "mix.g", H, E, 1.5)
            else:
                vec(p + "mix.q.norm", D, 1.5)
                vec(p + "mix.k.norm", D, 1.5)
        if ff is not None and ff["kind"] == "dense":
            mat(p + "mlp.gate", ff["ff"], E, 1.5)
            mat(p + "mlp.up", ff["ff"], E)
            mat(p + "mlp.down", E, ff["ff"])
        elif ff is not None:
            mat(p + "mlp.router", ff["router"]["experts"], E, 2.0)
            units = [(f"e{e}.", ff["expert"]["ff"]) for e in range(ff["router"]["experts"])]
            if ff.get("shared"):
                units.append(("shared.", ff["shared"]["ff"]))
                mat(p + "mlp.shared.sg", 1, E)
            for nm, f in units:
                mat(p + f"mlp.{nm}up", f, E, 1.5)
                mat(p + f"mlp.{nm}down", E, f, 1.5)
        if ts:
            mat(p + "side.gate", ts["dim"], E, 0.7)
            mat(p + "side.proj", E, ts["dim"])
            vec(p + "side.norm", E, 0.5)
    vec("final.norm", E)
    mat("head", V, E)
    return w
