"""Throughput and kernel times of models whose layers are listed one by one, beside the closest other family at equal sizes; random
weights.

``python bench.py --layers patesun`` (beside multi-head latent attention with routed experts, DeepSeek-V3 layout), ``--layers vilulorn``
(beside Gated DeltaNet + gated attention with routed experts, Qwen3-Next layout), ``--layers vuripel`` (beside Vilulorn) and ``--layers
nasipel`` (beside Vuripel) print one JSON line per measurement:
  * ``step``   -- prefill and decode tokens/s of a stack of four layers through the engine's runner;
  * ``kernel`` -- one operator alone: microseconds, its bytes / FLOPs and the fraction of the measured copy bandwidth or GEMM peak.
Operators are timed with CUDA events behind an L2 flush that also hides the host's launch time; the median of the repeats is kept.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

SIZES = {
    # width, heads, latent rank, window, dense ff, experts, top, expert ff, shared ff
    "2k": dict(width=2048, heads=16, rank=512, window=2048, ff=8192, experts=64, top=6, eff=1024, shared=2048),
    "4k": dict(width=4096, heads=32, rank=512, window=2048, ff=14336, experts=64, top=6, eff=1024, shared=2048),
    "7k": dict(width=7168, heads=128, rank=512, window=4096, ff=18432, experts=64, top=8, eff=2048, shared=2048),
}
HEAD, VOCAB, LAYERS = 128, 32768, 4
HYBRID_SIZES = {
    # width, query heads, key / value heads, linear heads, chunk, experts, top, expert ff
    "2k": dict(width=2048, heads=16, kv=4, lin=16, chunk=4096, experts=64, top=6, eff=1024),
    "4k": dict(width=4096, heads=32, kv=8, lin=32, chunk=4096, experts=64, top=6, eff=1024),
    "7k": dict(width=7168, heads=64, kv=8, lin=56, chunk=8192, experts=64, top=8, eff=2048),
}


def patesun_config(z):
    from ..models.config import from_hf_dict

    mx = {"heads": z["heads"], "dim": HEAD, "vdim": HEAD, "kv_rank": z["rank"], "scale": HEAD ** -0.5, "mask": {"size": z["window"]}}
    moe = {"kind": "moe", "expert": {"ff": z["eff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared"]}}
    return from_hf_dict(dict(architecture="Patesun", vocab=VOCAB, width=z["width"], norm={"eps": 1e-6}, residual_mult=0.4, loop=None,
                             layers=[{"type": "latent_attention", "mixer": mx, "mlp": {"kind": "dense", "ff": z["ff"]} if i == 0 else moe}
                                     for i in range(LAYERS)]))


def mla_config(z):
    from ..models.config import from_hf_dict

    return from_hf_dict(dict(model_type="deepseek_v3", vocab_size=VOCAB, hidden_size=z["width"], num_hidden_layers=LAYERS,
                             num_attention_heads=z["heads"], num_key_value_heads=z["heads"], intermediate_size=z["ff"],
                             moe_intermediate_size=z["eff"], n_routed_experts=z["experts"], num_experts_per_tok=z["top"],
                             n_shared_experts=z["shared"] // z["eff"], first_k_dense_replace=1, n_group=1, topk_group=1,
                             scoring_func="sigmoid", topk_method="noaux_tc", norm_topk_prob=True, kv_lora_rank=z["rank"],
                             qk_nope_head_dim=HEAD, qk_rope_head_dim=64, v_head_dim=HEAD, rms_norm_eps=1e-6, max_position_embeddings=65536))


def vilulorn_config(z):
    from ..models.config import from_hf_dict

    at = {"heads": z["heads"], "kv_heads": z["kv"], "dim": HEAD, "vdim": HEAD, "scale": HEAD ** -0.5, "mask": {"size": z["chunk"]},
          "rot": {"base": 5e5, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    gl = {"heads": z["lin"], "dim": HEAD, "vdim": HEAD, "tau": 16.0}
    moe = {"kind": "moe", "expert": {"ff": z["eff"], "limit": 7.0}, "router": {"experts": z["experts"], "top": z["top"]}}
    return from_hf_dict(dict(architecture="Vilulorn", vocab=VOCAB, width=z["width"], norm={"eps": 1e-6}, max_positions=1 << 16,
                             layers=[{"type": t, "mixer": m, "mlp": moe} for t, m in (("gla", gl), ("attention", at), ("gla", gl), ("attention", dict(at, kv_from=1)))]))


def vuripel_config(z):
    from ..models.config import from_hf_dict

    full = {"heads": z["heads"], "kv_heads": z["kv"], "dim": HEAD, "vdim": HEAD, "scale": HEAD ** -0.5, "softcap": 50.0}
    local = dict(full, mask={"size": z["chunk"], "keep_first": 16}, rot={"base": 5e5, "dims": 64})
    lstm = {"heads": z["lin"], "dim": HEAD, "vdim": HEAD, "gate_cap": 15.0}
    moe = {"kind": "moe", "expert": {"ff": z["eff"]}, "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": 8, "keep": 4}}, "shared": {"ff": z["eff"]}}
    return from_hf_dict(dict(architecture="Vuripel", vocab=VOCAB, width=z["width"], norm={"eps": 1e-6}, token_side={"dim": 256},
                             layers=[{"type": t, "mixer": m, "mlp": moe} for t, m in (("mlstm", lstm), ("attention_2", local), ("mlstm", lstm), ("attention", full))]))


def nasipel_config(z):
    from ..models.config import from_hf_dict

    at = {"heads": z["heads"], "kv_heads": z["kv"], "dim": HEAD, "vdim": HEAD, "scale": HEAD ** -0.5, "softcap": 50.0, "rot": {"base": 5e5, "dims": HEAD}}
    la = {"heads": z["heads"], "dim": HEAD, "vdim": HEAD, "q_rank": z["width"] // 2, "kv_rank": 512, "rot_dim": 64, "scale": (HEAD + 64) ** -0.5,
          "rot": {"base": 5e5, "dims": 64, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    rg = {"width": z["lin"] * HEAD, "blocks": z["lin"] // 2, "conv": 4}
    moe = {"kind": "moe", "expert": {"ff": z["eff"]}, "router": {"experts": z["experts"], "top": z["top"], "groups": {"count": 8, "keep": 4}, "scale": 2.0}}
    return from_hf_dict(dict(architecture="Nasipel", vocab=VOCAB, width=z["width"], norm={"eps": 1e-6},
                             layers=[{"type": t, "mixer": m, "mlp": moe} for t, m in (("rglru", rg), ("latent_attention", la), ("rglru", rg), ("attention", at))]))


def deltanet_config(z):
    from ..models.config import from_hf_dict

    return from_hf_dict(dict(model_type="qwen3_next", vocab_size=VOCAB, hidden_size=z["width"], num_hidden_layers=LAYERS, num_attention_heads=z["heads"],
                             num_key_value_heads=z["kv"], head_dim=HEAD, intermediate_size=z["eff"], num_experts=z["experts"],
                             num_experts_per_tok=z["top"], moe_intermediate_size=z["eff"], linear_num_key_heads=z["lin"], linear_num_value_heads=z["lin"],
                             linear_key_head_dim=HEAD, linear_value_head_dim=HEAD, full_attention_interval=2, partial_rotary_factor=0.5, rms_norm_eps=1e-6,
                             max_position_embeddings=65536))


class Timer:
    def __init__(self, repeats: int = 15):
        self.flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
        self.repeats = repeats

    def us(self, fn) -> float:
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        out = []
        for _ in range(self.repeats):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            self.flush.fill_(1)
            self.flush.fill_(0)
            a.record()
            fn()
            b.record()
            b.synchronize()
            out.append(a.elapsed_time(b) * 1e3)
        return statistics.median(out)


def peaks() -> tuple[float, float, str]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return float(d["hbm_gbs"]), float(d["bf16_tflops"]), "measured"
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0, "fallback"


# ---------------------------------------------------------------------------------------------------
# whole steps
# ---------------------------------------------------------------------------------------------------
def bench_steps(family: str, cfg, size: str, cases, emit) -> None:
    from ..engine.runner import EngineConfig, ModelRunner
    from ..models import random_init
    from ..ops import _lib

    model = random_init(cfg, "cuda", torch.bfloat16, seed=0, expert_pool=4)
    gen = torch.Generator().manual_seed(0)
    for batch, ctx in cases:
        pages = (ctx + 64) // 128 + 1
        runner = ModelRunner(model, EngineConfig(max_batch=batch, max_context=pages * 128, prefix_cache=False, graph_batch_sizes=[batch]), num_pages=batch * pages + 1)
        owned = [list(range(b * pages, (b + 1) * pages)) for b in range(batch)]
        states = list(range(batch)) if runner.state_slots else None
        toks = torch.randint(0, VOCAB, (ctx,), generator=gen).tolist()
        per = max(1, 8192 // ctx)                       # requests of a prefill step of about 8192 tokens
        n_pre = min(per, batch)

        def prefill(first, count):
            for s in range(0, ctx, 8192):
                runner.prefill([(toks[s:s + 8192], s, owned[b], s + 8192 >= ctx, b if states else None) for b in range(first, first + count)])

        for _ in range(2):
            prefill(0, n_pre)
        torch.cuda.synchronize()
        ms = []
        for _ in range(5):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            prefill(0, n_pre)
            b.record()
            b.synchronize()
            ms.append(a.elapsed_time(b))
        emit(dict(kind="step", family=family, size=size, what="prefill", requests=n_pre, tokens=ctx * n_pre, ms=statistics.median(ms),
                  tokens_per_s=ctx * n_pre / statistics.median(ms) * 1e3))
        for b in range(0, batch, n_pre):
            prefill(b, min(n_pre, batch - b))
        ids = torch.randint(0, VOCAB, (batch,), generator=gen).tolist()
        pos = [ctx] * batch
        for _ in range(4):
            runner.decode(ids, pos, owned, state_slots=states)
        slot = runner.slots[batch]
        torch.cuda.synchronize()
        ms = []
        for _ in range(20):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            if slot.graph is not None:
                slot.graph.replay()
            else:
                runner._decode_forward(slot)
            b.record()
            b.synchronize()
            ms.append(a.elapsed_time(b))
        emit(dict(kind="step", family=family, size=size, what="decode", batch=batch, context=ctx, ms=statistics.median(ms),
                  tokens_per_s=batch / statistics.median(ms) * 1e3, launches=runner.launches_per_decode_step, graph=slot.graph is not None))
        _lib.check_device_errors()
        runner.slots.clear()
        del runner, slot
        torch.cuda.empty_cache()
    del model
    torch.cuda.empty_cache()


# ---------------------------------------------------------------------------------------------------
# operators alone: the new one, then the like one of the other family
# ---------------------------------------------------------------------------------------------------
def bench_kernels(z, size: str, emit) -> None:
    from ..models.config import LatentSpec
    from ..models.decoder import ForwardBatch
    from ..ops import attention as A
    from ..ops import basic as B
    from ..ops import latent as LA
    from ..ops import moe as MOE
    from ..ops import stream32 as S

    tm = Timer()
    hbm, tf, src = peaks()
    dev, dt = "cuda", torch.bfloat16
    W, H, R, win = z["width"], z["heads"], z["rank"], z["window"]
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=dt) * 0.05
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)

    def put(name, role, fn, nbytes, flops, **info):
        us = tm.us(fn)
        t_mem, t_mm = nbytes / hbm / 1e3, flops / tf / 1e6           # microseconds at the measured peaks
        emit(dict(kind="kernel", size=size, name=name, role=role, us=round(us, 2), gbytes=nbytes / 1e9, gflop=flops / 1e9,
                  bound="memory" if t_mem > t_mm else "tensor", roofline_frac=round(max(t_mem, t_mm) / us, 4), peak=src, **info))

    # latent decode: windowed latent rows against latent + rotary rows over as many keys
    for batch, ctx in ((64, win), (64, 4 * win)):
        pages = ctx // 128
        lens = i32([ctx] * batch)
        pt = torch.randperm(batch * pages, device=dev).to(torch.int32).view(batch, pages)
        for name, role, dq, w in (("latent_decode", "new", R, win), ("mla_decode", "like", R + 64, 0)):
            pool = rnd(batch * pages + 1, 128, 1, dq)
            q = rnd(batch, H, dq)
            keys = min(ctx, w) if w else ctx
            put(name, role, lambda: A.mla_decode(q, pool, pt, lens, 0.1, lora=R, window=w), batch * (keys * dq * 2 + H * (dq + R) * 2),
                2.0 * batch * H * keys * (dq + R), batch=batch, context=ctx, keys=keys)
            del pool
    # row operators at a prefill-sized batch
    T, top = 8192, z["top"]
    nw, h, y16 = torch.ones(W, device=dev, dtype=dt), torch.randn(T, W, device=dev), rnd(T, W)
    put("rmsnorm32", "new", lambda: S.rmsnorm32(h, nw, 1e-6), T * W * 6, 0)
    put("rmsnorm", "like", lambda: B.rmsnorm(y16, nw, 1e-6), T * W * 4, 0)
    ids, pos = torch.randint(0, VOCAB, (T,), device=dev, dtype=torch.int32), torch.arange(T, device=dev, dtype=torch.int32)
    table, freq = rnd(VOCAB, W), S.sinusoid_inv_freq(W, 10000.0, dev)
    put("embed_pos_norm", "new", lambda: S.embed_pos_norm(ids, pos, table, freq, nw, 1e-6), T * W * 8, 0)
    put("embedding+rmsnorm", "like", lambda: B.rmsnorm(B.embedding(ids, table), nw, 1e-6), T * W * 8, 0)
    rows = T * top
    ys, where, wts = rnd(rows, W), torch.randperm(rows, device=dev).to(torch.int32).view(T, top), torch.full((T, top), 1.0 / top, device=dev)
    put("moe_combine_norm32", "new", lambda: S.moe_combine_norm(ys, where, None, 1.0 / top, y16, h, nw, 0.4, 1e-6), rows * W * 2 + T * W * 12, 0)

    def like_combine():
        out = torch.empty((T, W), device=dev, dtype=dt)
        from ..ops import _lib

        _lib.kernels().fb_moe_combine(B._ptr(ys), B._ptr(where), B._ptr(wts), B._ptr(None), B._ptr(out), T, top, W, 1, B._stream())
        r = out + y16
        return B.rmsnorm(r + y16, nw, 1e-6)
    put("combine+add+add+rmsnorm", "like", like_combine, rows * W * 2 + T * W * 8, 0)
    del ys, where
    # routing plan of the layers of a stack
    class _L:
        pass
    fake = []
    for _ in range(LAYERS - 1):
        l = _L()
        l.route_table = torch.rand((VOCAB, z["experts"]), device=dev).topk(top, dim=1).indices.to(torch.int32).contiguous()
        l.experts = _L()
        l.experts.stacked, l.experts.count = True, z["experts"]
        fake.append(l)
    router = MOE.TableRouter(fake, dev)
    logits, bias = torch.randn(T, z["experts"], device=dev), torch.zeros(z["experts"], device=dev)
    put(f"table plans of {LAYERS - 1} layers", "new", lambda: router.plan(ids), (LAYERS - 1) * T * top * 8, 0)

    def like_plan():
        idx, w_ = MOE.route_topk(logits, bias, top, 1, True)
        c = torch.empty(z["experts"], device=dev, dtype=torch.int32)
        o, t1, p_ = torch.empty_like(c), torch.empty(1, device=dev, dtype=torch.int32), torch.empty((T, top), device=dev, dtype=torch.int32)
        from ..ops import _lib, moe_grouped

        _lib.kernels().fb_moe_plan(B._ptr(idx), T, top, 0, z["experts"], B._ptr(c), B._ptr(o), B._ptr(p_), B._ptr(t1), moe_grouped.PAD, B._stream())
    put("top-k and plan of 1 layer", "like", like_plan, T * top * 8, 0)
    # projections onto the residual
    for M in (64, T):
        x, w, hm, rm = rnd(M, H * HEAD), rnd(W, H * HEAD), torch.randn(M, W, device=dev), rnd(M, W)
        fl = 2.0 * M * W * H * HEAD
        put("gemm_res32", "new", lambda: B.linear_res32(x, w, hm, 0.4), W * H * HEAD * 2 + M * (H * HEAD * 2 + W * 8), fl, rows=M)
        put("gemm_residual", "like", lambda: B.linear(x, w, residual=rm), W * H * HEAD * 2 + M * (H * HEAD * 2 + W * 4), fl, rows=M)
    # prompt chunk: latents -> keys and values -> windowed attention, against the latent-space products of the other family
    spec = LatentSpec(H, HEAD, HEAD, R, HEAD ** -0.5, win)
    lw, _, _ = LA.build(spec, rnd(H * HEAD, W), rnd(H * HEAD, W), rnd(R, W), torch.ones(R, device=dev, dtype=dt), rnd(H * HEAD, R), rnd(H * HEAD, R))
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages = n // 128
        cu = [n * b for b in range(n_req + 1)]
        fb = ForwardBatch(ids=ids, positions=pos % n, slots=pos, page_table=torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages),
                          kv_lens=i32([n] * n_req), cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
        keys = sum(min(i + 1, win) for i in range(n)) * n_req         # (query, key) pairs
        pool, proj = rnd(n_req * pages + 1, 128, 1, R), rnd(T, lw.latent_col + 64)
        LA.attention(lw, proj, pool, fb)
        grp = fb._latent_plans[next(iter(fb._latent_plans))].groups[0]
        kv = B.linear(S.gather_rows(pool.view(-1, R), grp.key_idx), lw.w_ukv)
        put("latent expand", "new", lambda: B.linear(S.gather_rows(pool.view(-1, R), grp.key_idx), lw.w_ukv), T * (R * 2 + 2 * H * HEAD * 2), 2.0 * T * R * 2 * H * HEAD,
            requests=n_req, tokens=n)
        out = torch.empty((T, H * HEAD), device=dev, dtype=dt)
        put("windowed prefill attention", "new", lambda: LA.window_attention(lw, grp, proj[:, :H * HEAD], proj[:, lw.gate_col:lw.latent_col], kv, out),
            T * H * HEAD * 10, 4.0 * keys * H * HEAD, requests=n_req, tokens=n)
        causal = n * (n + 1) // 2 * n_req
        del kv, out
        if causal * H * 6 / n_req < 40e9:                             # the other family keeps all scores of a request in memory
            q_full, pool2 = rnd(T, H, R + 64), rnd(n_req * pages + 1, 128, 1, R + 64)
            put("mla prefill products", "like", lambda: MOE.mla_paged_attention(q_full, pool2, fb, 0.1, R), T * H * (2 * R + 64) * 2,
                2.0 * causal * H * (2 * R + 64), requests=n_req, tokens=n)
            del q_full, pool2
        torch.cuda.empty_cache()


def bench_hybrid_kernels(z, size: str, emit) -> None:
    """Operators of the chunked-attention / gated-linear-attention stack, each before the like one of the Gated-DeltaNet stack."""
    from ..models.config import AttnSpec, GLASpec
    from ..models.decoder import ForwardBatch
    from ..ops import attention as A
    from ..ops import basic as B
    from ..ops import gla as GLA
    from ..ops import grouped as GR
    from ..ops import linear_attn as L
    from ..ops import moe as MOE
    from ..ops import moe_grouped as MG
    from ..ops import stream32 as S
    from ..ops._lib import kernels

    tm = Timer()
    hbm, tf, src = peaks()
    dev, dt = "cuda", torch.bfloat16
    W, H, G, N, C, E, top, eff = (z[k] for k in ("width", "heads", "kv", "lin", "chunk", "experts", "top", "eff"))
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=dt) * 0.05
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    rope = {"theta": 5e5, "rot_dim": 64, "scaling": None}
    cos, sin = A.build_rope_tables(64, 65536, 5e5, None, dev)

    def put(name, role, fn, nbytes, flops, **info):
        us = tm.us(fn)
        t_mem, t_mm = nbytes / hbm / 1e3, flops / tf / 1e6
        emit(dict(kind="kernel", size=size, name=name, role=role, us=round(us, 2), gbytes=nbytes / 1e9, gflop=flops / 1e9,
                  bound="memory" if t_mem > t_mm else "tensor", roofline_frac=round(max(t_mem, t_mm) / us, 4), peak=src, **info))

    # recurrent step of 64 requests: state read and written once
    Bn, D = 64, HEAD
    gw, _ = GLA.build(GLASpec(N, D, D, 16.0), *(rnd(N * D, 16) for _ in range(4)), rnd(16, 16), rnd(N * D, 16), rnd(N * D), rnd(D))
    st, slots = torch.zeros((Bn + 1, N, D, D), device=dev), i32(list(range(Bn)))
    proj = rnd(Bn, gw.cols[-1] + 32)
    fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=None, kv_lens=None, cu_q=None, is_decode=True, state_slots=slots)
    nb = Bn * N * (2 * D * D * 4 + 5 * D * 2)
    put("gla step", "new", lambda: GLA.mix(gw, proj, fb, st, 1e-6), nb, 0, batch=Bn)
    mixed, ab, zz, par = rnd(Bn, 3 * N * D), rnd(Bn, N), rnd(Bn, N * D), torch.zeros(N, device=dev)
    put("delta-rule step", "like", lambda: L.gated_delta_decode(mixed, ab, ab, zz, par, par, gw.norm, 1e-6, st, slots, N, N, D, D), nb, 0, batch=Bn)
    # prompts: chunked forms
    T = 8192
    for n_req, n in ((1, T), (T // 2048, 2048)):
        cu = [n * b for b in range(n_req + 1)]
        proj, sl = rnd(T, gw.cols[-1] + 32), list(range(n_req))
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, state_slots=i32(sl), state_slots_host=sl)
        nb, fl = T * N * D * 2 * 5, T * N * (4.0 * D * D + 2.0 * 64 * D)
        put("gla prompt", "new", lambda: GLA.mix(gw, proj, fb, st, 1e-6), nb, fl, requests=n_req, tokens=n)
        q, k, v, a = rnd(T, N, D), rnd(T, N, D), rnd(T, N, D), rnd(T, N)

        def like():
            o = L.gated_delta_rule(q, k, v, a, a, par, par, st, cu, sl, 1)
            return L.rmsnorm_gated(o, v, gw.norm, 1e-6)
        put("delta-rule prompt", "like", like, nb, fl, requests=n_req, tokens=n)
        del q, k, v, a, proj
    del st
    # attention: decoded rows, prompts, post-processing
    spec = AttnSpec(H, G, HEAD, HEAD, HEAD ** -0.5, C, rope)
    at, _ = GR.build(spec, rnd(H * HEAD, 16), rnd(G * HEAD, 16), rnd(G * HEAD, 16), rnd(H * HEAD, 16), rnd(HEAD), rnd(HEAD))
    ctxs = (C, 2 * C)
    for ctx in ctxs:
        pages = ctx // 128
        pool = (rnd(Bn * pages, 128, G, HEAD), rnd(Bn * pages, 128, G, HEAD))
        pt, lens = torch.randperm(Bn * pages, device=dev).to(torch.int32).view(Bn, pages), i32([ctx] * Bn)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=pt, kv_lens=lens, cu_q=None, is_decode=True)
        proj = rnd(Bn, (at.v_col + G * HEAD + 31) // 32 * 32)
        GR.attention(at, proj, pool, fb)
        put("grouped decode", "new", lambda: GR.attention(at, proj, pool, fb), Bn * (C * G * HEAD * 4 + H * HEAD * 6), 4.0 * Bn * H * C * HEAD, batch=Bn, context=ctx, keys=C)
        ws = A.DecodeWorkspace(Bn, G, H // G, pages, torch.device(dev), HEAD)
        ws.plan(lens)
        q = rnd(Bn, H * HEAD)
        put("decode attention", "like", lambda: A.attn_decode(q, *pool, pt, lens, 0.1, H, G, HEAD, ws=ws, planned=True), Bn * (ctx * G * HEAD * 4 + H * HEAD * 4),
            4.0 * Bn * H * ctx * HEAD, batch=Bn, context=ctx, keys=ctx)
        del pool, ws
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages, cu = n // 128, [n * b for b in range(n_req + 1)]
        pool = (rnd(n_req * pages, 128, G, HEAD), rnd(n_req * pages, 128, G, HEAD))
        pt, lens = torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages), i32([n] * n_req)
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        fb = ForwardBatch(ids=pos, positions=pos % n, slots=pos, page_table=pt, kv_lens=lens, cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
        proj = rnd(T, (at.v_col + G * HEAD + 31) // 32 * 32)
        causal = lambda m: m * (m + 1) // 2
        seen = (n // C * causal(C) + causal(n % C)) * n_req
        GR.attention(at, proj, pool, fb)
        put("grouped prompt attention", "new", lambda: GR.attention(at, proj, pool, fb), T * (H * HEAD * 6 + G * HEAD * 4), 4.0 * seen * H * HEAD, requests=n_req, tokens=n)
        q = rnd(T, H * HEAD)
        put("prompt attention", "like", lambda: A.attn_prefill(q, *pool, pt, lens, fb.cu_q, 0.1, H, G, HEAD, cu_q_host=cu), T * (H * HEAD * 4 + G * HEAD * 4),
            4.0 * causal(n) * n_req * H * HEAD, requests=n_req, tokens=n)
    nb = T * (2 * H + 4 * G) * HEAD * 2
    put("head norm + rotary + append", "new", lambda: GR.post(at, proj, fb, pool, cos, sin, 1e-6), nb, 0, rows=T)
    qkv, nw = rnd(T, (H + 2 * G) * HEAD), rnd(HEAD)
    put("qkv post", "like", lambda: A.qkv_post(qkv, fb.positions, fb.slots, *pool, H, G, HEAD, cos, sin, A.ROPE_INTERLEAVED, 64, nw, nw), nb, 0, rows=T)
    del pool, proj, qkv
    # row operators
    h, y, nw = torch.randn(T, W, device=dev), rnd(T, W), torch.ones(W, device=dev, dtype=dt)
    res = rnd(T, W)
    put("output norm + residual", "new", lambda: S.add_norm(h, y, nw, None, 1e-6), T * W * 12, 0)
    put("residual + norm", "like", lambda: B.rmsnorm(y, nw, 1e-6, residual=res), T * W * 8, 0)
    ids, pos, table, ptab = torch.randint(0, VOCAB, (T,), device=dev, dtype=torch.int32), torch.arange(T, device=dev, dtype=torch.int32), rnd(VOCAB, W), rnd(T, W)
    put("embedding + learned positions", "new", lambda: S.embed_pos_norm(ids, pos, table, None, None, 1e-6, pos_table=ptab), T * W * 10, 0)
    put("embedding + norm", "like", lambda: B.rmsnorm(B.embedding(ids, table), nw, 1e-6), T * W * 8, 0)
    # experts: routing, plan, gather, the two grouped products, combine
    ex = MOE.ExpertWeights(E, 0, [], [])
    ex.count, ex.act, ex.limit, ex.scale_input = E, "gptoss", 7.0, True
    ex.stacked = MG.StackedExperts("dense", rnd(E * 2 * eff, W), rnd(E * W, eff), E, eff, W)
    ey = MOE.ExpertWeights(E, 0, [], [])
    ey.count, ey.stacked = E, ex.stacked

    class _M:
        router_bias = None
    MOE.set_router(_M, rnd(E, W), top, True)
    for M in (64, T):
        x, h, res = rnd(M, W), torch.randn(M, W, device=dev), rnd(M, W)
        logits, bias = torch.randn(M, E, device=dev), torch.zeros(E, device=dev)
        put("router + top-k", "new", lambda: MOE.route_scored(_M, x), M * W * 2 + E * W * 2, 2.0 * M * E * W, rows=M)
        put("router + top-k", "like", lambda: MOE.route_topk(B.linear(x, _M.router_16, out_f32=True), None, top, 0, True), M * W * 2 + E * W * 2, 2.0 * M * E * W, rows=M)
        idx, wts = MOE.route_topk(logits, bias, top, 1, False)
        fl, nb = 6.0 * M * top * W * eff, 3 * E * W * eff * 2 + M * top * (4 * W + 2 * eff) * 2

        def new():
            ys, p_, _ = MG.forward(x, idx, wts, ex, combine=False, rows32=h)
            return S.moe_combine_norm(ys, p_, None, 1.0, None, h, None, 1.0, 1e-6, post_w=nw, dtype=dt)
        put("experts, scaled inputs, output norm", "new", new, nb, fl, rows=M)
        put("experts, residual, norm", "like", lambda: B.rmsnorm(MG.forward(x, idx, wts, ey), nw, 1e-6, residual=res), nb, fl, rows=M)
        plan = MG._make_plan(idx, ex)
        xs, rows = torch.empty((M * top + E * 16 + 128, W), device=dev, dtype=dt), M * top
        put("scaled gather", "new", lambda: S.moe_gather_scaled(h, plan[2], wts, xs), M * W * 4 + rows * W * 2, 0, rows=M)
        put("gather", "like", lambda: kernels().fb_moe_gather(B._ptr(x), B._ptr(plan[2]), B._ptr(xs), M, top, W, B._stream()), M * W * 2 + rows * W * 2, 0, rows=M)
        put("combine, output norm, residual", "new", lambda: S.moe_combine_norm(xs, plan[2], None, 1.0, None, h, None, 1.0, 1e-6, post_w=nw, dtype=dt),
            rows * W * 2 + M * W * 10, 0, rows=M)

        def comb():
            out = torch.empty((M, W), device=dev, dtype=dt)
            kernels().fb_moe_combine(B._ptr(xs), B._ptr(plan[2]), B._ptr(wts), B._ptr(None), B._ptr(out), M, top, W, 1, B._stream())
            return B.rmsnorm(out, nw, 1e-6, residual=res)
        put("combine, residual, norm", "like", comb, rows * W * 2 + M * W * 8, 0, rows=M)
    torch.cuda.empty_cache()


def bench_parallel_kernels(z, size: str, emit) -> None:
    """Operators of the parallel-block stack (matrix-memory LSTM, capped attention with sinks and kept tokens), each before the like one
    of the chunked-attention / gated-linear-attention stack."""
    from ..models.config import AttnSpec, GLASpec, MLSTMSpec
    from ..models.decoder import ForwardBatch
    from ..ops import attention as A
    from ..ops import basic as B
    from ..ops import gla as GLA
    from ..ops import grouped as GR
    from ..ops import mlstm as ML
    from ..ops import moe as MOE
    from ..ops import moe_grouped as MG
    from ..ops import stream32 as S

    tm = Timer()
    hbm, tf, src = peaks()
    dev, dt = "cuda", torch.bfloat16
    W, H, G, N, C, E, top, eff = (z[k] for k in ("width", "heads", "kv", "lin", "chunk", "experts", "top", "eff"))
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=dt) * 0.05
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    D, T, Bn = HEAD, 8192, 64

    def put(name, role, fn, nbytes, flops, **info):
        us = tm.us(fn)
        t_mem, t_mm = nbytes / hbm / 1e3, flops / tf / 1e6
        emit(dict(kind="kernel", size=size, name=name, role=role, us=round(us, 2), gbytes=nbytes / 1e9, gflop=flops / 1e9,
                  bound="memory" if t_mem > t_mm else "tensor", roofline_frac=round(max(t_mem, t_mm) / us, 4), peak=src, **info))

    # recurrent layers: a step of 64 requests, prompts
    mw, _ = ML.build(MLSTMSpec(N, D, D, 15.0), *(rnd(N * D, 16) for _ in range(4)), rnd(N), rnd(N) + 4.0, rnd(N * D))
    gw, _ = GLA.build(GLASpec(N, D, D, 16.0), *(rnd(N * D, 16) for _ in range(4)), rnd(16, 16), rnd(N * D, 16), rnd(N * D), rnd(D))
    sm, sg = torch.zeros((Bn + 1, N, ML.state_len(D, D)), device=dev), torch.zeros((Bn + 1, N, D, D), device=dev)
    step = ForwardBatch(ids=None, positions=None, slots=None, page_table=None, kv_lens=None, cu_q=None, is_decode=True, state_slots=i32(list(range(Bn))))
    proj, gates = rnd(Bn, gw.cols[-1] + 32), torch.randn(Bn, 2 * N, device=dev)
    nb = Bn * N * (2 * D * D * 4 + 5 * D * 2)
    put("matrix-memory step", "new", lambda: ML.mix(mw, proj, gates, step, sm, 1e-6), nb, 0, batch=Bn)
    put("gated linear step", "like", lambda: GLA.mix(gw, proj, step, sg, 1e-6), nb, 0, batch=Bn)
    for n_req, n in ((1, T), (T // 2048, 2048)):
        cu, sl = [n * b for b in range(n_req + 1)], list(range(n_req))
        proj, gates = rnd(T, gw.cols[-1] + 32), torch.randn(T, 2 * N, device=dev)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, state_slots=i32(sl), state_slots_host=sl)
        nb, fl = T * N * D * 2 * 5, T * N * (4.0 * D * D + 2.0 * 64 * D)
        put("matrix-memory prompt", "new", lambda: ML.mix(mw, proj, gates, fb, sm, 1e-6), nb, fl, requests=n_req, tokens=n)
        put("gated linear prompt", "like", lambda: GLA.mix(gw, proj, fb, sg, 1e-6), nb, fl, requests=n_req, tokens=n)
        del proj
    del sm, sg
    # attention
    rope = {"theta": 5e5, "rot_dim": 64, "scaling": None, "mode": "neox"}
    cos, sin = A.build_rope_tables(64, 65536, 5e5, None, dev)

    def layer(**kw):
        spec = AttnSpec(H, G, D, D, D ** -0.5, **kw)
        norms = (rnd(D), rnd(D)) if spec.qk_norm else (None, None)
        w, _ = GR.build(spec, rnd(H * D, 16), rnd(G * D, 16), rnd(G * D, 16), rnd(H * D, 16) if spec.gate == "elem" else None, *norms, None,
                        rnd(H) if spec.sinks else None)
        return w
    capped = dict(softcap=50.0, bias=True)
    pairs = (("attention, cap + sinks + head gate", layer(sinks=True, qk_norm=False, gate="head", **capped), "attention", layer(), 0),
             ("attention, window + kept + cap", layer(window=C, keep=16, gate="", rope=rope, **capped), "attention, chunk", layer(chunk=C, rope=dict(rope, mode="interleaved")), C))
    for ctx in (C, 2 * C):
        pages = ctx // 128
        pool = (rnd(Bn * pages, 128, G, D), rnd(Bn * pages, 128, G, D))
        pt, lens = torch.randperm(Bn * pages, device=dev).to(torch.int32).view(Bn, pages), i32([ctx] * Bn)
        for new, wn, like, wl, span in pairs:
            keys = min(ctx, span) if span else ctx
            for name, role, w in ((new, "new", wn), (like, "like", wl)):
                fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=pt, kv_lens=lens, cu_q=None, is_decode=True)
                proj, hg = rnd(Bn, (w.v_col + G * D + 31) // 32 * 32), torch.randn(Bn, H, device=dev) if w.gate == "head" else None
                GR.attention(w, proj, pool, fb, head_gate=hg)
                put("decode " + name, role, lambda: GR.attention(w, proj, pool, fb, head_gate=hg), Bn * (keys * G * D * 4 + H * D * (6 if w.gate == "elem" else 4)),
                    4.0 * Bn * H * keys * D, batch=Bn, context=ctx, keys=keys)
        del pool
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages, cu = n // 128, [n * b for b in range(n_req + 1)]
        pool = (rnd(n_req * pages, 128, G, D), rnd(n_req * pages, 128, G, D))
        pt, lens = torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages), i32([n] * n_req)
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        fb = ForwardBatch(ids=pos, positions=pos % n, slots=pos, page_table=pt, kv_lens=lens, cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
        causal = lambda m: m * (m + 1) // 2
        for new, wn, like, wl, span in pairs:
            inside = causal(n) - (causal(n - span) if span and n > span else 0)
            chunked = n // span * causal(span) + causal(n % span) if span else causal(n)
            for name, role, w, seen in ((new, "new", wn, inside), (like, "like", wl, chunked)):
                proj, hg = rnd(T, (w.v_col + G * D + 31) // 32 * 32), torch.randn(T, H, device=dev) if w.gate == "head" else None
                GR.attention(w, proj, pool, fb, head_gate=hg)
                put("prompt " + name, role, lambda: GR.attention(w, proj, pool, fb, head_gate=hg), T * (H * D * (6 if w.gate == "elem" else 4) + G * D * 4),
                    4.0 * seen * n_req * H * D, requests=n_req, tokens=n)
    proj = rnd(T, (H * 2 + 2 * G) * D)
    for name, role, w, heads in (("append", "new", pairs[0][1], 2 * G), ("head norm + rotary (halves) + append", "new", pairs[1][1], H + 2 * G),
                                 ("head norm + rotary (pairs) + append", "like", pairs[1][3], H + 2 * G)):
        put(name, role, lambda: GR.post(w, proj, fb, pool, cos, sin, 1e-6), T * heads * D * 4, 0, rows=T)
    del pool, proj
    # row operators
    h, y, nw, table = torch.randn(T, W, device=dev), rnd(T, W), torch.ones(W, device=dev, dtype=dt), rnd(VOCAB, W)
    ids = torch.randint(0, VOCAB, (T,), device=dev, dtype=torch.int32)
    put("output norm + residual + pass start + norm", "new", lambda: S.add_norm(h, y, nw, nw, 1e-6, start=(table, ids, nw)), T * W * 14, 0)
    put("output norm + residual + norm", "new", lambda: S.add_norm(h, y, nw, nw, 1e-6), T * W * 12, 0)
    put("output norm + residual", "like", lambda: S.add_norm(h, y, nw, None, 1e-6), T * W * 12, 0)
    # products of a layer: the joint one, gated units, the token input's two, logits
    for M in (64, T):
        x, K, side = rnd(M, W), H * D + eff, 256
        a, wj, wg, hm, cp = rnd(M, K), rnd(W, K), rnd(2 * eff * 4, W), torch.randn(M, W, device=dev), torch.empty((M, W), device=dev, dtype=dt)
        nb, fl = W * K * 2 + M * (K * 2 + W * 8), 2.0 * M * W * K
        put("joint product onto the residual + copy", "new", lambda: B.linear_res32(a, wj, hm, 1.0, cp), nb + M * W * 2, fl, rows=M)
        put("product onto the residual", "like", lambda: B.linear_res32(a, wj, hm, 1.0), nb, fl, rows=M)
        nb, fl = wg.numel() * 2 + M * (W + 4 * eff) * 2, 2.0 * M * wg.numel()
        put("gated gelu units", "new", lambda: B.linear(x, wg, swiglu=True, geglu=True), nb, fl, rows=M)
        put("gated silu units", "like", lambda: B.linear(x, wg, swiglu=True), nb, fl, rows=M)
        tab, ws, wp, mid, wl = rnd(VOCAB, 4 * side), rnd(side, W), rnd(W, side), rnd(M, side), rnd(96, W)
        nb, fl = side * W * 2 + M * (W + 2 * side) * 2, 2.0 * M * W * side
        put("token input, gate", "new", lambda: B.linear_act(x, ws, "gelu_tanh", mul=tab[:, side:2 * side], mul_rows=ids[:M]), nb, fl, rows=M)
        put("relu^2 product of that size", "like", lambda: B.linear(x, ws, relu2=True), nb - M * side * 2, fl, rows=M)
        put("token input, projection", "new", lambda: B.linear(mid, wp), nb - M * side * 2, fl, rows=M)
        wu, rg = rnd(eff, W), torch.randn(M, 96, device=dev)
        nb, fl = eff * W * 2 + M * (W + eff) * 2, 2.0 * M * W * eff
        put("shared expert, gelu + row gate", "new", lambda: B.linear_act(x, wu, "gelu", row_gate=rg[:, 70]), nb, fl, rows=M)
        put("relu^2 product of that size", "like", lambda: B.linear(x, wu, relu2=True), nb, fl, rows=M)
        put("logits + grouped top-k", "new", lambda: MOE.route_topk(B.linear(x, wl, out_f32=True)[:, :E], None, top, 0, False, 8, 4, group_max=True), M * W * 2 + E * W * 2,
            2.0 * M * E * W, rows=M)
        put("router + top-k", "like", lambda: MOE.route_topk(B.linear(x, wl[:E].contiguous(), out_f32=True), None, top, 1, False), M * W * 2 + E * W * 2, 2.0 * M * E * W, rows=M)
    # experts with and without a gate branch, to the residual
    ex, ey = (MOE.ExpertWeights(E, 0, [], []) for _ in range(2))
    ex.count = ey.count = E
    ex.act, ey.act, ey.limit, ey.scale_input = "gelu", "gptoss", 7.0, True
    up, down = rnd(E * 2 * eff, W), rnd(E * W, eff)
    ex.stacked, ey.stacked = MG.StackedExperts("dense", up[:E * eff], down, E, eff, W), MG.StackedExperts("dense", up, down, E, eff, W)
    for M in (64, T):
        x, h, sh = rnd(M, W), torch.randn(M, W, device=dev), rnd(M, W)
        idx, wts = MOE.route_topk(torch.randn(M, E, device=dev), None, top, 0, False)
        for name, role, e, mats in (("experts without gate branch, shared rows, residual", "new", ex, 2), ("experts, scaled inputs, output norm", "like", ey, 3)):
            fl, nb = 2.0 * mats * M * top * W * eff, mats * E * W * eff * 2 + M * top * (4 * W + 2 * eff) * 2

            def fn():
                ys, p_, _ = MG.forward(x, idx, wts, e, combine=False, rows32=h if e.scale_input else None)
                return S.moe_combine_norm(ys, p_, None if e.scale_input else wts, 1.0, None if e.scale_input else sh, h, None, 1.0, 1e-6,
                                          post_w=nw if e.scale_input else None, dtype=dt)
            put(name, role, fn, nb, fl, rows=M)
    torch.cuda.empty_cache()


def bench_gated_kernels(z, size: str, emit) -> None:
    """Operators of the gated-sub-layer stack (recurrent units, sigmoid-weighted attention over rotated values, latent attention with rotated
    parts), each before the like one of the parallel-block stack or, for latent attention, of the latent families."""
    from ..models.config import AttnSpec, LatentSpec, MLSTMSpec, RGLRUSpec
    from ..models.decoder import ForwardBatch
    from ..ops import attention as A
    from ..ops import basic as B
    from ..ops import grouped as GR
    from ..ops import latent as LA
    from ..ops import mlstm as ML
    from ..ops import moe as MOE
    from ..ops import moe_grouped as MG
    from ..ops import rglru as RG
    from ..ops import stream32 as S

    tm = Timer()
    hbm, tf, src = peaks()
    dev, dt = "cuda", torch.bfloat16
    W, H, G, N, C, E, top, eff = (z[k] for k in ("width", "heads", "kv", "lin", "chunk", "experts", "top", "eff"))
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=dt) * 0.05
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    D, T, Bn = HEAD, 8192, 64
    causal = lambda m: m * (m + 1) // 2

    def put(name, role, fn, nbytes, flops, **info):
        us = tm.us(fn)
        t_mem, t_mm = nbytes / hbm / 1e3, flops / tf / 1e6
        emit(dict(kind="kernel", size=size, name=name, role=role, us=round(us, 2), gbytes=nbytes / 1e9, gflop=flops / 1e9,
                  bound="memory" if t_mem > t_mm else "tensor", roofline_frac=round(max(t_mem, t_mm) / us, 4), peak=src, **info))

    # recurrent layers: a step of 64 requests, prompts
    R, part = N * D, 2 * D
    rw, _ = RG.build(RGLRUSpec(R, N // 2, 4), rnd(R, 16), rnd(R, 16), rnd(R, 4), rnd(R), rnd(N // 2, part, part), rnd(N // 2, part), rnd(N // 2, part, part), rnd(N // 2, part),
                     torch.linspace(-6, -2, R, device=dev).to(dt))
    mw, _ = ML.build(MLSTMSpec(N, D, D, 15.0), *(rnd(N * D, 16) for _ in range(4)), rnd(N), rnd(N) + 4.0, rnd(N * D))
    sr, sm = (torch.zeros((Bn + 1, R, 3), device=dev, dtype=dt), torch.zeros((Bn + 1, R), device=dev)), torch.zeros((Bn + 1, N, ML.state_len(D, D)), device=dev)
    step = ForwardBatch(ids=None, positions=None, slots=None, page_table=None, kv_lens=None, cu_q=None, is_decode=True, state_slots=i32(list(range(Bn))))
    proj, proj_m, gates = rnd(Bn, 2 * R + W), rnd(Bn, mw.cols[-1] + R + 32), torch.randn(Bn, 2 * N, device=dev)
    weights = 2 * R * part * 2
    put("recurrent unit step", "new", lambda: RG.mix(rw, proj, step, sr), Bn * R * (2 * 3 + 2 * 4 + 2 * 3 * 2) + weights, 4.0 * Bn * R * part, batch=Bn)
    put("matrix-memory step", "like", lambda: ML.mix(mw, proj_m, gates, step, sm, 1e-6), Bn * N * (2 * D * D * 4 + 5 * D * 2), 0, batch=Bn)
    for n_req, n in ((1, T), (T // 2048, 2048)):
        cu, sl = [n * b for b in range(n_req + 1)], list(range(n_req))
        proj, proj_m, gates = rnd(T, 2 * R + W), rnd(T, mw.cols[-1] + R + 32), torch.randn(T, 2 * N, device=dev)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, state_slots=i32(sl), state_slots_host=sl)
        put("recurrent unit prompt", "new", lambda: RG.mix(rw, proj, fb, sr), T * R * 2 * 3 + weights, 4.0 * T * R * part, requests=n_req, tokens=n)
        put("matrix-memory prompt", "like", lambda: ML.mix(mw, proj_m, gates, fb, sm, 1e-6), T * N * D * 2 * 5, T * N * (4.0 * D * D + 2.0 * 64 * D), requests=n_req, tokens=n)
    u = rnd(T, R)
    put("gate logits, block products", "new", lambda: B.linear_blocks(u, rw.gates), T * R * (2 + 8) + weights, 4.0 * T * R * part, rows=T)
    wide = rnd(2 * R, part)
    put("product of that inner width", "like", lambda: B.linear(u[:, :part], wide, out_f32=True), T * (2 * part + 8 * R) + weights, 4.0 * T * R * part, rows=T)
    del sr, sm, proj, proj_m, u, wide
    # grouped-query attention
    rope = {"theta": 5e5, "rot_dim": D, "scaling": None, "mode": "neox"}
    tables = A.build_rope_tables(D, 65536, 5e5, None, dev)

    def layer(**kw):
        spec = AttnSpec(H, G, D, D, D ** -0.5, softcap=50.0, rope=rope, **kw)
        norms = (rnd(D), rnd(D)) if spec.qk_norm and spec.norm_weight else (None, None)
        w, _ = GR.build(spec, rnd(H * D, 16), rnd(G * D, 16), rnd(G * D, 16), None, *norms, None, rnd(H) if spec.sinks else None, rnd(H) - 4.0)
        w.turn = tables
        return w
    pairs = (("sigmoid weights + cap + turned values", "new", layer(gate="", norm_weight=False, weights="sigmoid", rope_values=rope)),
             ("cap + sinks + head gate", "like", layer(gate="head", sinks=True)))
    for ctx in (C // 2, C):
        pages = ctx // 128
        pool = (rnd(Bn * pages, 128, G, D), rnd(Bn * pages, 128, G, D))
        pt, lens = torch.randperm(Bn * pages, device=dev).to(torch.int32).view(Bn, pages), i32([ctx] * Bn)
        for name, role, w in pairs:
            fb = ForwardBatch(ids=None, positions=lens - 1, slots=None, page_table=pt, kv_lens=lens, cu_q=None, is_decode=True)
            proj, hg = rnd(Bn, (w.v_col + G * D + 31) // 32 * 32), torch.randn(Bn, H, device=dev) if w.gate == "head" else None
            GR.attention(w, proj, pool, fb, head_gate=hg)
            put("decode attention, " + name, role, lambda: GR.attention(w, proj, pool, fb, head_gate=hg), Bn * (ctx * G * D * 4 + H * D * 4), 4.0 * Bn * H * ctx * D, batch=Bn, context=ctx)
        del pool
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages, cu = n // 128, [n * b for b in range(n_req + 1)]
        pool = (rnd(n_req * pages, 128, G, D), rnd(n_req * pages, 128, G, D))
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        fb = ForwardBatch(ids=pos, positions=pos % n, slots=pos, page_table=torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages), kv_lens=i32([n] * n_req),
                          cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
        for name, role, w in pairs:
            proj, hg = rnd(T, (w.v_col + G * D + 31) // 32 * 32), torch.randn(T, H, device=dev) if w.gate == "head" else None
            GR.attention(w, proj, pool, fb, head_gate=hg)
            put("prompt attention, " + name, role, lambda: GR.attention(w, proj, pool, fb, head_gate=hg), T * (H * D * 4 + G * D * 4), 4.0 * causal(n) * n_req * H * D, requests=n_req, tokens=n)
    proj = rnd(T, (H + 2 * G) * D)
    for name, role, w in (("unit norm + rotary + append of turned values", "new", pairs[0][2]), ("norm + rotary + append", "like", pairs[1][2])):
        put(name, role, lambda: GR.post(w, proj, fb, pool, *tables, 1e-6), T * (H + 2 * G) * D * 4, 0, rows=T)
    del pool, proj
    # latent attention
    K, Rd, Q, ln = 512, 64, W // 2, {"theta": 5e5, "rot_dim": 64, "scaling": None, "mode": "interleaved"}
    cs = A.build_rope_tables(Rd, 65536, 5e5, None, dev)
    lw, _, up = LA.build(LatentSpec(H, D, D, K, (D + Rd) ** -0.5, q_rank=Q, rot_dim=Rd, rope=ln, gate="head"), rnd(Q, 16), rnd(H, 16), rnd(K + Rd, 16), rnd(K), rnd(H * D, K), rnd(H * D, K),
                         rnd(H * (D + Rd), Q), rnd(Q))
    from ..ops.quant import LinearWeight

    lw.q_up = LinearWeight.from_dense(up, act_dtype=dt)
    lp, _, _ = LA.build(LatentSpec(H, D, D, K, D ** -0.5), rnd(H * D, 16), rnd(H * D, 16), rnd(K, 16), rnd(K), rnd(H * D, K), rnd(H * D, K))
    for ctx in (C // 2, C):
        pages = ctx // 128
        lens = i32([ctx] * Bn)
        pt = torch.randperm(Bn * pages, device=dev).to(torch.int32).view(Bn, pages)
        pool, q, hg = rnd(Bn * pages + 1, 128, 1, K + Rd), rnd(Bn, H, K + Rd), torch.randn(Bn, H, device=dev)
        for name, role, gate in (("latent decode, head gate", "new", hg), ("mla decode", "like", None)):
            put(name, role, lambda: A.mla_decode(q, pool, pt, lens, 0.1, lora=K, head_gate=gate), Bn * (ctx * (K + Rd) * 2 + H * (2 * K + Rd) * 2), 2.0 * Bn * H * ctx * (2 * K + Rd), batch=Bn, context=ctx)
        del pool
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages, cu = n // 128, [n * b for b in range(n_req + 1)]
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        for name, role, w, rot in (("latent prompt attention, rotated part + head gate", "new", lw, Rd), ("latent prompt attention", "like", lp, 0)):
            fb = ForwardBatch(ids=pos, positions=pos % n, slots=pos, page_table=torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages), kv_lens=i32([n] * n_req),
                              cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
            pool, proj, out = rnd(n_req * pages + 1, 128, 1, w.ld), rnd(T, w.more_col + 32), torch.empty((T, H * D), device=dev, dtype=dt)
            q, hg = LA.post(w, proj, fb, pool, cs if rot else None, 1e-6)
            LA.attention(w, proj, pool, fb, q, hg, cs)
            grp = fb._latent_plans[next(iter(fb._latent_plans))].groups[0]
            rows = S.gather_rows(pool.view(-1, w.ld), grp.key_idx)
            expand = lambda: B.linear(S.gather_rows(pool.view(-1, w.ld), grp.key_idx)[:, :w.lv], w.w_ukv)
            kv = expand()
            gate = proj[:, w.gate_col:w.latent_col] if not rot else None
            put(name, role, lambda: LA.window_attention(w, grp, q, gate, kv, out, hg, rows[:, w.lv:] if rot else None), T * H * (4 * D + 2 * rot) * 2, 2.0 * causal(n) * n_req * H * (2 * D + rot),
                requests=n_req, tokens=n)
            put("latent expand", role, expand, T * (w.ld * 2 + 2 * H * D * 2), 4.0 * T * K * H * D, requests=n_req, tokens=n)
            if n_req == 1:
                args = (proj, w.latent_col, w.kv_norm, w.rank, fb.slots, pool, 1e-6, w.lv, w.rot_col, w.rot, False, fb.positions, *(cs if rot else (None, None)), w.q_norm, w.q_pad, w.gate_col, w.n_gates)
                put("latent norms + rotary key + append", role, lambda: S.latent_post(*args), T * (2 * w.q_pad + 2 * w.ld) * 2, 0, rows=T)
                if rot:
                    qr = q[:, w.dim:]
                    put("rotary query parts", "new", lambda: S.rope_heads(qr, w.hd, qr, w.hd, H, Rd, Rd, fb.positions, *cs), T * H * Rd * 4, 0, rows=T)
            del pool, proj, kv, rows, q
        torch.cuda.empty_cache()
    # the join of a layer, the products beside it, routing
    nw = torch.ones(W, device=dev, dtype=dt)
    for M in (64, T):
        h, x, y, gcol = torch.randn(M, W, device=dev), rnd(M, W), rnd(M, W), rnd(M, 2 * W)
        ys, where, wts, zz = rnd(M * top, W), torch.randperm(M * top, device=dev).to(torch.int32).view(M, top), torch.rand(M, top, device=dev), torch.randn(M, W + E, device=dev)
        put("gated join of mixer and experts + two norms", "new", lambda: S.gated_join(h, (y, gcol[:, W:]), (ys, where, wts, zz[:, :W]), nw, nw, 1e-6, dt), M * W * (2 * top + 2 + 2 + 4 + 8 + 4), 0, rows=M)
        put("combine + shared rows + residual + norm", "like", lambda: S.moe_combine_norm(ys, where, wts, 1.0, y, h, nw, 1.0, 1e-6, dtype=dt), M * W * (2 * top + 2 + 8 + 2), 0, rows=M)
        wz, bz, wp = rnd(W + E, W), rnd(W + E), rnd(W + E, W)
        nb, fl = (W + E) * W * 2 + M * (W * 2 + (W + E) * 4), 2.0 * M * W * (W + E)
        put("gate + router logits", "new", lambda: B.linear(x, wz, bz, out_f32=True), nb, fl, rows=M)
        put("product of that size", "like", lambda: B.linear(x, wp), nb - M * (W + E) * 2, fl, rows=M)
        cor = torch.zeros(E, device=dev)
        put("corrected grouped top-k", "new", lambda: MOE.route_topk(zz[:, W:], cor, top, 1, True, 8, 4, 2.0), M * (E * 4 + top * 8), 0, rows=M)
        put("grouped top-k", "like", lambda: MOE.route_topk(zz[:, W:], None, top, 0, False, 8, 4, group_max=True), M * (E * 4 + top * 8), 0, rows=M)
        del ys
    table, ids = rnd(VOCAB, W), torch.randint(0, VOCAB, (T,), device=dev, dtype=torch.int32)
    put("embedding + two norms", "new", lambda: S.gated_join(h, None, None, nw, nw, 1e-6, dt, embed=(table, ids)), T * W * 10, 0, rows=T)
    put("embedding + norm", "like", lambda: S.embed_pos_norm(ids, ids, table, None, nw, 1e-6), T * W * 8, 0, rows=T)
    ex = MOE.ExpertWeights(E, 0, [], [])
    ex.count, ex.stacked = E, MG.StackedExperts("dense", rnd(E * 2 * eff, W), rnd(E * W, eff), E, eff, W)
    ey = MOE.ExpertWeights(E, 0, [], [])
    ey.count, ey.act, ey.stacked = E, "gelu", MG.StackedExperts("dense", ex.stacked.gate_up[:E * eff], ex.stacked.down, E, eff, W)
    for M in (64, T):
        x = rnd(M, W)
        idx, wts = MOE.route_topk(torch.randn(M, E, device=dev), None, top, 0, False)
        for name, role, e, mats in (("gated experts", "new", ex, 3), ("experts without gate branch", "like", ey, 2)):
            put(name, role, lambda: MG.forward(x, idx, wts, e, combine=False), mats * E * W * eff * 2 + M * top * (4 * W + 2 * eff) * 2, 2.0 * mats * M * top * W * eff, rows=M)
    torch.cuda.empty_cache()


def run(family: str, sizes, steps: bool = True, kernels: bool = True, emit=None) -> None:
    emit = emit or (lambda d: print(json.dumps(d), flush=True))
    hybrid = family != "patesun"
    operators = {"patesun": bench_kernels, "vilulorn": bench_hybrid_kernels, "vuripel": bench_parallel_kernels, "nasipel": bench_gated_kernels}[family]
    stacks = {"patesun": (("patesun", patesun_config), ("mla", mla_config)), "vilulorn": (("vilulorn", vilulorn_config), ("deltanet", deltanet_config)),
              "vuripel": (("vuripel", vuripel_config), ("vilulorn", vilulorn_config)), "nasipel": (("nasipel", nasipel_config), ("vuripel", vuripel_config))}[family]
    for size in sizes:
        z = (HYBRID_SIZES if hybrid else SIZES)[size]
        if kernels:
            operators(z, size, emit)
        torch.cuda.empty_cache()
        if steps:
            span = z["chunk" if hybrid else "window"]
            for fam, make in stacks:
                # (a chunk's first token sees only itself: the longest context of a decoded token ends just before the next chunk)
                full = span - 128 if hybrid else span
                bench_steps(fam, make(z), size, ((1, full), (64, span // 2), (64, full)), emit)
