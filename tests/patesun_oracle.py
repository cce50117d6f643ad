"""Plain statement of the Patesun decoder: one function per mechanism, whole sequences, no cache, float64 by default.

Written from the equations alone and sharing no code with the package; the tests compare the framework with it.  ``weights`` is a
dict of tensors under the checkpoint's names, ``cfg`` the config.json dictionary.
"""
import torch


def linear(w, x):
    """W x for a batch of rows: ``w`` [out, in], ``x`` [rows, in]."""
    return x @ w.to(x.dtype).T


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(x.dtype)


def sinusoid(positions, width, dtype=torch.float64):
    """Row p: sin(p / 10000^(2i / width)) in entry 2i, the cosine of the same angle in entry 2i + 1."""
    out = torch.zeros(len(positions), width, dtype=torch.float64)
    for c in range(width):
        i = c // 2
        angle = positions.to(torch.float64) * 10000.0 ** (-2.0 * i / width)
        out[:, c] = torch.sin(angle) if c % 2 == 0 else torch.cos(angle)
    return out.to(dtype)


def visible(n, window):
    """[n, n] bool: query i sees key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = j <= i
    if window:
        see = see & (i - j < window)
    return see


def latent(h, w, prefix, eps):
    return rms_norm(linear(w[prefix + "dkv"], h), w[prefix + "dkv.norm"], eps)


def latent_core(q, c, uk, uv, gate, mixer):
    """Attention of the rows ``q`` [n, heads * dim], which are the last n of the len(c) tokens, over the latents ``c`` [L, rank];
    ``gate`` [n, heads * vdim] is the projection before its sigmoid."""
    n, L, H, D, V = q.shape[0], c.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    k = linear(uk, c).reshape(L, H, D)
    v = linear(uv, c).reshape(L, H, V)
    s = torch.einsum("ihd,jhd->hij", q.reshape(n, H, D), k) * mixer["scale"]
    s = s.masked_fill(~visible(L, (mixer.get("mask") or {}).get("size"))[L - n:], float("-inf"))
    o = torch.einsum("hij,jhv->ihv", torch.softmax(s, dim=-1), v).reshape(n, H * V)
    return o * torch.sigmoid(gate)


def latent_attention(h, w, prefix, mixer, eps):
    """``h`` [n, width] is one whole sequence."""
    c = latent(h, w, prefix, eps)
    o = latent_core(linear(w[prefix + "q"], h), c, w[prefix + "uk"], w[prefix + "uv"], linear(w[prefix + "g"], h), mixer)
    return linear(w[prefix + "o"], o)


def relu2_ff(h, w, prefix):
    u = torch.relu(linear(w[prefix + "up"], h))
    return linear(w[prefix + "down"], u * u)


def glu_ff(h, w, prefix):
    g = linear(w[prefix + "gate"], h)
    return linear(w[prefix + "down"], g * torch.sigmoid(g) * linear(w[prefix + "up"], h))


def table_moe(h, tokens, w, prefix, mlp):
    """Experts picked by the token id's row of the table, equal weights; the shared expert runs for every row."""
    out = torch.zeros_like(h)
    table, top = w[prefix + "table"], mlp["router"]["top"]
    for t in range(h.shape[0]):
        for e in table[int(tokens[t])].tolist():
            out[t] += glu_ff(h[t:t + 1], w, f"{prefix}e{e}.")[0] / top
    if mlp.get("shared"):
        out = out + glu_ff(h, w, prefix + "shared.")
    return out


def layer_order(cfg):
    loop = cfg.get("loop")
    idx = list(range(len(cfg["layers"])))
    if not loop:
        return idx
    return idx[:loop["start"]] + idx[loop["start"]:loop["stop"]] * loop["times"] + idx[loop["stop"]:]


def embed(tokens, w, width, dtype=torch.float64):
    return w["embed"][tokens].to(dtype) + sinusoid(torch.arange(len(tokens)), width, dtype)


def forward(cfg, w, tokens, dtype=torch.float64, layers_out=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out``: a list that collects the residual after every layer run."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(tokens, w, cfg["width"], dtype)
    for i in layer_order(cfg):
        spec, p = cfg["layers"][i], f"l{i}."
        x = x + m * latent_attention(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
        mlp = spec.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            y = relu2_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else table_moe(h, tokens, w, p + "mlp.", mlp)
            x = x + m * y
        if layers_out is not None:
            layers_out.append(x)
    return linear(w["head"], rms_norm(x, w["final.norm"], eps))


def random_weights(cfg, seed=0, scale=1.0):
    """bfloat16 weights of the right names and shapes (norm weights around one, a table with distinct entries per row)."""
    g = torch.Generator().manual_seed(seed)
    E, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, n, k, s=1.0):
        w[name] = (torch.randn(n, k, generator=g) * (s * scale / k ** 0.5)).to(torch.bfloat16)

    def norm(name, n):
        w[name] = (1.0 + 0.2 * torch.randn(n, generator=g)).to(torch.bfloat16)

    w["embed"] = torch.randn(V, E, generator=g).to(torch.bfloat16)
    for i, spec in enumerate(cfg["layers"]):
        p, mx, ff = f"l{i}.", spec["mixer"], spec.get("mlp")
        H, D, Vd, R = mx["heads"], mx["dim"], mx["vdim"], mx["kv_rank"]
        norm(p + "norm1", E)
        mat(p + "mix.q", H * D, E, 1.5)
        mat(p + "mix.dkv", R, E)
        norm(p + "mix.dkv.norm", R)
        mat(p + "mix.uk", H * D, R, 1.5)
        mat(p + "mix.uv", H * Vd, R)
        mat(p + "mix.g", H * Vd, E)
        mat(p + "mix.o", E, H * Vd, 2.0)
        if ff is None:
            continue
        norm(p + "norm2", E)
        if ff["kind"] == "dense":
            mat(p + "mlp.up", ff["ff"], E)
            mat(p + "mlp.down", E, ff["ff"])
            continue
        n, top = ff["router"]["experts"], ff["router"]["top"]
        parts = [(f"e{e}", ff["expert"]["ff"]) for e in range(n)] + ([("shared", ff["shared"]["ff"])] if ff.get("shared") else [])
        for nm, inter in parts:
            mat(f"{p}mlp.{nm}.gate", inter, E, 1.5)
            mat(f"{p}mlp.{nm}.up", inter, E)
            mat(f"{p}mlp.{nm}.down", E, inter, 2.0)
        w[p + "mlp.table"] = torch.stack([torch.randperm(n, generator=g)[:top] for _ in range(V)]).to(torch.int32)
    norm("final.norm", E)
    mat("head", V, E)
    return w
