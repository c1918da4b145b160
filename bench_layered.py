"""`bench.py --model sulepel-...` or `sefalorn-...`: decode and prefill throughput of a layer-list decoder with random weights, its kernels one by
one against their rooflines, and beside them the like kernels and the throughput of the framework's closest other model
(Qwen3-MoE) at the same width, head counts, number of layers, batch and context lengths.

Called by bench.py; prints one JSON line.  Every kernel is launched once per layer on that layer's own weights and pages
(together far more than the 126 MB L2), between CUDA events, several times over; a kernel's roofline is the longer of its
bytes at the measured copy bandwidth and its flops at the measured bf16 rate.
"""
from __future__ import annotations

import importlib
import json
import os
import time

import numpy as np
import torch

ROOT = os.path.dirname(os.path.abspath(__file__))
PAGE = 16


def pkg(sub):
    return importlib.import_module("inference-server_b200." + sub)


def peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return float(p["hbm_gbs"]), float(p["bf16_tflops"]), "measured (MEASURED_PEAKS.json)"
    except Exception:
        return 6650.0, 1590.0, "fallback (6.65 TB/s, 1.59 PFLOP/s)"


def timed(fns, reps: int = 4) -> float:
    """Median over `reps` rounds of the mean device time (us) of the launches in `fns`, run one after the other."""
    for f in fns[:3] if len(fns) >= 3 else fns * 3:
        f()
    torch.cuda.synchronize()
    out = []
    for _ in range(reps):
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda._sleep(200_000)  # the launches queue up behind it, so host time does not show
        e0.record()
        for f in fns:
            f()
        e1.record()
        torch.cuda.synchronize()
        out.append(e0.elapsed_time(e1) * 1e3 / len(fns))
    return float(np.median(out))


class Table:
    """Kernel -> time and roofline fraction."""

    def __init__(self):
        self.hbm, self.tf, self.source = peaks()
        self.rows = {}

    def add(self, name: str, fns, nbytes: float, flops: float) -> None:
        us = timed(fns)
        t_mem, t_math = nbytes / self.hbm / 1e3, flops / self.tf / 1e6
        self.rows[name] = {"us": round(us, 2), "bound": "hbm" if t_mem >= t_math else "tensor",
                           "roofline_us": round(max(t_mem, t_math), 2), "frac": round(max(t_mem, t_math) / us, 3)}


def pairs_seen(first: int, n: int, chunk: int) -> int:
    p = np.arange(first, first + n)
    return int((p - (p // chunk * chunk if chunk else 0) + 1).sum())


def decode_kernels(eng, B: int, lens) -> dict:
    """The decode step's kernels, each alone."""
    lay, ops, cfg = pkg("layered"), pkg("ops"), eng.cfg
    t = Table()
    dev, W = eng.device, eng.W
    table, pos = eng.block_table[:B], eng.ctx_lens[:B]
    new_len = pos + 1
    bf = dict(device=dev, dtype=torch.bfloat16)
    x, d, h = torch.randn(B, W, device=dev), torch.randn(B, W, **bf), torch.randn(B, W, **bf)
    att = [i for i, s in enumerate(cfg.layer_list) if isinstance(s.mixer, lay.AttentionSpec)]
    lat = [i for i in range(cfg.layers) if i not in att]
    glu = [i for i, s in enumerate(cfg.layer_list) if s.mlp is not None]
    norm = dict(eps=cfg.norm_eps, width=cfg.width, groups=cfg.norm_groups, status=eng.status)
    row = B * W
    t.add("norm + convolution (decode form)", [lambda w=w, hs=hs: ops.group_rmsnorm(x, d, w.norm1, conv_w=w.conv, hist=hs, positions=pos,
                                                                      block_table=table, page=PAGE, out=h, **norm)
                                 for w, hs in zip(eng.layers, eng.hist)], row * (8 + 2 + 2 + 2 * cfg.taps), 0)
    t.add("norm", [lambda w=w: ops.group_rmsnorm(x, d, w.norm1, out=h, **norm) for w in eng.layers], row * (8 + 2 + 2), 0)
    splits, ws = eng._attn_for(B)
    for ids, kind in ((att, "attention"), (lat, "latent")):
        if not ids:
            continue
        m, w0 = cfg.layer_list[ids[0]].mixer, eng.layers[ids[0]]
        H, D, N = m.heads, w0.D, w0.wproj.shape[0]
        q, gate, out = torch.randn(B, H, D, **bf), torch.randn(B, H, device=dev), torch.empty(B, H, D, **bf)
        if kind == "attention":
            t.add("attention projection + page write", [lambda i=i: ops.proj_split(
                h, eng.layers[i].wproj, [(ops.SEG_ROWS, q), (ops.SEG_PAGES, eng.k_pools[i]), (ops.SEG_PAGES, eng.v_pools[i]),
                                         (ops.SEG_F32, gate)], eng.layers[i].col_scale, pos, table, eng.status) for i in ids],
                N * W * 2 + B * (W + N) * 2, 2 * B * N * W)
            seen = sum(n - (n - 1) // m.chunk * m.chunk if m.chunk else n for n in (lens + 1))
            t.add("chunked attention + split reduce", [lambda i=i: ops.paged_attn_decode_chunked(
                q, eng.k_pools[i], eng.v_pools[i], table, new_len, w0.scale, splits[i], ws, m.chunk, gate, out) for i in ids],
                seen * m.kv_heads * D * 4 + B * H * D * 4, 4 * seen * H * D)
        else:
            raw = torch.empty(B, w0.R, device=dev)
            qc, oc = torch.randn(B, H, w0.R, **bf), torch.empty(B, H, w0.R, **bf)
            t.add("latent projection", [lambda i=i: ops.proj_split(h, eng.layers[i].wproj, [(ops.SEG_ROWS, q), (ops.SEG_F32, raw),
                                                                                         (ops.SEG_F32, gate)], status=eng.status)
                                        for i in ids], N * W * 2 + B * W * 2 + B * (H * D * 2 + w0.R * 4), 2 * B * N * W)
            t.add("latent norm + page write", [lambda i=i: ops.latent_norm_append(raw, eng.layers[i].c_norm, cfg.norm_eps, m.rank,
                                                                                 eng.c_pools[i], pos, table, eng.status) for i in ids],
                  B * w0.R * 6, 0)
            hb = H * D * w0.R * 2 + B * H * (D + w0.R) * 2
            t.add("queries to latents", [lambda i=i: ops.grouped_gemm(q, eng.layers[i].wuk_t, H, out=qc) for i in ids], hb,
                  2 * B * H * D * w0.R)
            total = int((lens + 1).sum())
            t.add("latent attention + split reduce", [lambda i=i: ops.latent_attn_decode(
                qc, eng.c_pools[i], table, new_len, w0.scale, splits[i], ws, gate, oc) for i in ids],
                total * w0.R * 2 + B * H * w0.R * 4, 4 * total * H * w0.R)
            t.add("values of latents", [lambda i=i: ops.grouped_gemm(oc, eng.layers[i].wuv, H, out=out) for i in ids], hb,
                  2 * B * H * D * w0.R)
        y = torch.empty(B, W, **bf)
        t.add(f"{kind} output projection", [lambda i=i: ops.dense_gemm(out.view(B, H * D), eng.layers[i].wo, out=y, status=eng.status,
                                                                      workspace=eng.gemm_ws) for i in ids],
              W * H * D * 2 + B * (W + H * D) * 2, 2 * B * W * H * D)
    F = eng.layers[glu[0]].wdown.shape[1]
    a = torch.randn(B, F, **bf)
    t.add("gate/up + gated unit", [lambda i=i: ops.glu_proj(h, eng.layers[i].wgu, cfg.layer_list[i].mlp.limit, lay.GLU_ALPHA, out=a)
                                   for i in glu], 2 * F * W * 2 + B * (W + F) * 2, 4 * B * F * W)
    t.add("down", [lambda i=i: ops.dense_gemm(a, eng.layers[i].wdown, out=y, status=eng.status, workspace=eng.gemm_ws) for i in glu],
          F * W * 2 + B * (W + F) * 2, 2 * B * F * W)
    t.add("lm_head + arg-max", [lambda: eng._pick(h)] * 4, eng.lm_head.numel() * 2 + B * W * 2, 2 * B * eng.lm_head.numel())
    eng.check_status("decode kernels")
    return t.rows


def prompt_kernels(eng, first: int, n: int) -> dict:
    """A prompt chunk's kernels at positions first.. of one sequence."""
    lay, ops, cfg = pkg("layered"), pkg("ops"), eng.cfg
    t = Table()
    dev, W = eng.device, eng.W
    bf = dict(device=dev, dtype=torch.bfloat16)
    ctx = first + n
    row = torch.zeros(eng.max_pages, dtype=torch.int32, device=dev)
    row[: -(-ctx // PAGE)] = torch.randperm(eng.num_blocks, device=dev)[: -(-ctx // PAGE)].int()
    table = row[None].expand(n, -1).contiguous()
    pos = torch.arange(first, ctx, dtype=torch.int32, device=dev)
    x, d, h = torch.randn(n, W, device=dev), torch.randn(n, W, **bf), torch.randn(n, W, **bf)
    y = torch.empty(n, W, **bf)
    att = [i for i, s in enumerate(cfg.layer_list) if isinstance(s.mixer, lay.AttentionSpec)]
    lat = [i for i in range(cfg.layers) if i not in att]
    glu = [i for i, s in enumerate(cfg.layer_list) if s.mlp is not None]
    t.add("norm", [lambda w=w: ops.group_rmsnorm(x, d, w.norm1, cfg.norm_eps, cfg.width, cfg.norm_groups, out=h) for w in eng.layers],
          n * W * 12, 0)
    t.add("convolution", [lambda w=w, hs=hs: ops.short_conv(h, w.conv, hs, row, first, out=y) for w, hs in zip(eng.layers, eng.hist)],
          n * W * 4, 0)
    for ids, kind in ((att, "attention"), (lat, "latent")):
        if not ids:
            continue
        m, w0 = cfg.layer_list[ids[0]].mixer, eng.layers[ids[0]]
        H, D, N = m.heads, w0.D, w0.wproj.shape[0]
        q, gate, out = torch.randn(n, H, D, **bf), torch.randn(n, H, device=dev), torch.empty(n, H, D, **bf)
        if kind == "attention":
            t.add("attention projection + page write", [lambda i=i: ops.proj_split(
                h, eng.layers[i].wproj, [(ops.SEG_ROWS, q), (ops.SEG_PAGES, eng.k_pools[i]), (ops.SEG_PAGES, eng.v_pools[i]),
                                         (ops.SEG_F32, gate)], eng.layers[i].col_scale, pos, table, eng.status) for i in ids],
                N * W * 2 + n * (W + N) * 2, 2 * n * N * W)
            t.add("chunked attention", [lambda i=i: ops.paged_attn_prefill_chunked(
                q, eng.k_pools[i], eng.v_pools[i], row, first, w0.scale, eng.status, m.chunk, gate, out) for i in ids],
                n * H * D * 4, 4 * H * D * pairs_seen(first, n, m.chunk))
        else:
            raw = torch.empty(n, w0.R, device=dev)
            ks, vs, order = eng._expanded_kv(H, D, -(-ctx // PAGE))
            c = ops.gather_pages(eng.c_pools[ids[0]], row, ctx)
            t.add("latent projection", [lambda i=i: ops.proj_split(h, eng.layers[i].wproj, [(ops.SEG_ROWS, q), (ops.SEG_F32, raw),
                                                                                         (ops.SEG_F32, gate)], status=eng.status)
                                        for i in ids], N * W * 2 + n * W * 2 + n * (H * D * 2 + w0.R * 4), 2 * n * N * W)
            t.add("latent norm + page write", [lambda i=i: ops.latent_norm_append(raw, eng.layers[i].c_norm, cfg.norm_eps, m.rank,
                                                                                 eng.c_pools[i], pos, table, eng.status) for i in ids],
                  n * w0.R * 6, 0)
            t.add("latents of the context, gathered", [lambda i=i: ops.gather_pages(eng.c_pools[i], row, ctx) for i in ids],
                  ctx * w0.R * 4, 0)
            t.add("keys and values of the context", [lambda i=i: ops.proj_split(c, eng.layers[i].wukv, [(ops.SEG_PAGES, ks),
                                                                                                        (ops.SEG_PAGES, vs)])
                                                     for i in ids], ctx * (w0.R + 2 * H * D) * 2, 4 * ctx * H * D * w0.R)
            t.add("latent layer's attention", [lambda i=i: ops.paged_attn_prefill_chunked(q, ks, vs, order, first, w0.scale, eng.status,
                                                                                          0, gate, out) for i in ids],
                  n * H * D * 4 + ctx * H * D * 4, 4 * H * D * pairs_seen(first, n, 0))
        t.add(f"{kind} output projection", [lambda i=i: ops.dense_gemm(out.view(n, H * D), eng.layers[i].wo, out=y, status=eng.status,
                                                                      workspace=eng.gemm_ws) for i in ids],
              W * H * D * 2 + n * (W + H * D) * 2, 2 * n * W * H * D)
    F = eng.layers[glu[0]].wdown.shape[1]
    a = torch.randn(n, F, **bf)
    t.add("gate/up + gated unit", [lambda i=i: ops.glu_proj(h, eng.layers[i].wgu, cfg.layer_list[i].mlp.limit, lay.GLU_ALPHA, out=a)
                                   for i in glu], 2 * F * W * 2 + n * (W + F) * 2, 4 * n * F * W)
    t.add("down", [lambda i=i: ops.dense_gemm(a, eng.layers[i].wdown, out=y, status=eng.status, workspace=eng.gemm_ws) for i in glu],
          F * W * 2 + n * (W + F) * 2, 2 * n * F * W)
    eng.check_status("prompt kernels")
    return t.rows


def qwen_kernels(eng, B: int, lens, first: int, n: int) -> tuple[dict, dict]:
    """The like kernels of the Qwen3-MoE engine: (decode, prompt chunk)."""
    ops, cfg = pkg("ops"), eng.cfg
    dev, W, D, Hq, Hkv = eng.device, cfg.hidden, cfg.head_dim, cfg.q_heads, cfg.kv_heads
    bf = dict(device=dev, dtype=torch.bfloat16)
    out = []
    for rows, decode in ((B, True), (n, False)):
        t = Table()
        x, d = torch.randn(rows, W, **bf), torch.randn(rows, W, **bf)
        h = torch.randn(rows, W, **bf)
        if decode:
            table, pos = eng.block_table[:B], eng.ctx_lens[:B]
        else:
            ctx = first + n
            row = torch.zeros(eng.max_pages, dtype=torch.int32, device=dev)
            row[: -(-ctx // PAGE)] = torch.randperm(eng.num_blocks, device=dev)[: -(-ctx // PAGE)].int()
            table, pos = row[None].expand(n, -1).contiguous(), torch.arange(first, ctx, dtype=torch.int32, device=dev)
        t.add("norm", [lambda w=w: ops.add_rmsnorm(x, d, w.ln1, cfg.rms_eps, out=h) for w in eng.layers], rows * W * 8, 0)
        q, o, y = torch.randn(rows, Hq, D, **bf), torch.empty(rows, Hq, D, **bf), torch.empty(rows, W, **bf)
        N = (Hq + 2 * Hkv) * D
        t.add("attention projection + page write", [lambda li=li, w=w: ops.qkv_rope_append_gemm(
            h, w.wqkv, w.q_norm, w.k_norm, eng.cos, eng.sin, pos, table, eng.k_pools[li], eng.v_pools[li], Hq, cfg.rms_eps,
            eng.gemm_status, q) for li, w in enumerate(eng.layers)], N * W * 2 + rows * (W + N) * 2, 2 * rows * N * W)
        q.normal_()
        if decode:
            seen = int((lens + 1).sum())
            t.add("attention + split reduce", [lambda li=li: ops.paged_attn_decode(
                q, eng.k_pools[li], eng.v_pools[li], table, pos + 1, eng.scale, eng.split_tokens, eng.attn_ws, o)
                for li in range(cfg.layers)], seen * Hkv * D * 4 + rows * Hq * D * 4, 4 * seen * Hq * D)
        else:
            st = torch.zeros(64, dtype=torch.int32, device=dev)
            t.add("attention", [lambda li=li: ops.paged_attn_prefill(q, eng.k_pools[li], eng.v_pools[li], row, first, eng.scale, st, o)
                                for li in range(cfg.layers)], rows * Hq * D * 4, 4 * Hq * D * pairs_seen(first, n, 0))
        t.add("output projection", [lambda w=w: ops.dense_gemm(o.view(rows, Hq * D), w.wo, out=y, status=eng.gemm_status,
                                                               workspace=eng.gemm_ws) for w in eng.layers],
              W * Hq * D * 2 + rows * (W + Hq * D) * 2, 2 * rows * W * Hq * D)
        ids, _ = ops.moe_route(torch.randn(rows, cfg.experts, device=dev), cfg.top_k, True)
        perm, xq, xs = ops.moe_permute_quant(ids, h, cfg.experts)
        hit = int(torch.unique(ids).numel())
        w0 = eng.layers[0]
        hq, hs = ops.moe_fp8_gemm_gate_up(xq, xs, w0.w13, w0.w13_scale, perm)
        I = cfg.moe_inter
        # e4m3 operands: the dense rate is twice bf16's
        t.add("experts gate/up + gated unit (e4m3)", [lambda w=w: ops.moe_fp8_gemm_gate_up(xq, xs, w.w13, w.w13_scale, perm)
                                                      for w in eng.layers], hit * 2 * W * I + rows * cfg.top_k * (W + I),
              2 * rows * cfg.top_k * W * I)
        t.add("experts down (e4m3)", [lambda w=w: ops.moe_fp8_gemm_down(hq, hs, w.w2, w.w2_scale, perm) for w in eng.layers],
              hit * W * I + rows * cfg.top_k * (I + 2 * W), rows * cfg.top_k * W * I)
        if decode:
            t.add("lm_head + arg-max", [lambda: eng._pick(h)] * 4, eng.lm_head.numel() * 2 + B * W * 2, 2 * B * eng.lm_head.numel())
        out.append(t.rows)
    eng.check_status("qwen kernels")
    return out[0], out[1]


def fill(eng, gen):
    for pools in (getattr(eng, n, None) for n in ("k_pools", "v_pools", "c_pools", "hist")):
        first = {}
        for p in pools or []:
            if p is not None:
                same = first.get(p.shape)
                if same is None:
                    first[p.shape] = p.normal_(generator=gen)
                else:
                    p.copy_(same)


def throughput(eng, args, table, lens, prompt_tokens: int, prompt_blocks: int, clocks):
    """Decode steps of the whole batch (graph replays) and end to end through the backend, prompt passes of one sequence."""
    backend_mod = pkg("backend")
    B = args.batch
    V = eng.vocab_size
    eng.block_table[:, : table.shape[1]].copy_(torch.from_numpy(table))

    def restart():
        """Contexts and states as they were: with random weights the states of all rows drift the same way, step by step, and the
        rows then choose fewer and fewer experts."""
        eng.ctx_lens.copy_(torch.tensor(lens, dtype=torch.int32))
        gen = torch.Generator(device=eng.device).manual_seed(7)
        for pool in [*(getattr(eng, "states", None) or []), *(getattr(eng, "rings", None) or [])]:
            if pool is not None:
                pool.normal_(generator=gen)

    restart()
    # Random weights' own next tokens fall together over the steps, and with them the experts that a step reads: every step is
    # given new random tokens instead.
    feeds = torch.randint(0, V, (8, B), generator=torch.Generator().manual_seed(0))
    on_device, on_host = feeds.to(eng.device), [f.view(B, 1).pin_memory() for f in feeds]

    def events(fn, steps):
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for i in range(steps):
            fn(i)
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / steps

    def step(i):
        eng.tokens[:B].copy_(on_device[i % 8])
        eng.step(B)

    for i in range(1 + max(3, args.warmup)):
        step(i)
    restart()
    if clocks is not None:
        clocks.mark()
    out = {"decode_ms": events(step, args.steps)}
    out["decode_tok_s"] = B / out["decode_ms"] * 1e3
    be = backend_mod.B200Backend(eng)
    be._alloc.free, be._slots.free = [], []
    rows = [backend_mod.SeqKV(block_ids=table[b][: -(-(lens[b] + args.gen_tokens) // PAGE)].tolist(), ctx_len=lens[b],
                              slot=b if getattr(eng, "num_slots", 0) else None) for b in range(B)]
    batch = backend_mod.PagedBatch(rows=rows)
    for i in range(3):
        be.decode_step_batched(on_host[i], batch)
    restart()
    for row in batch.rows:
        row.ctx_len -= 3
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    for i in range(args.steps):
        _, batch = be.decode_step_batched(on_host[i % 8], batch)
    torch.cuda.synchronize()
    out["decode_e2e_tok_s"] = B * args.steps / (time.perf_counter() - t0)
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, V, (prompt_tokens,), generator=g).tolist() for _ in range(4)]
    blocks = list(range(prompt_blocks, prompt_blocks + -(-prompt_tokens // PAGE)))

    spare_slot = max(0, getattr(eng, "num_slots", 0) - 1)

    def prefill(i):
        eng.prefill(prompts[i % 4], blocks, slot=spare_slot)

    for i in range(3):
        prefill(i)
    steps = max(4, args.steps // 4)
    out["prefill_ms"] = events(prefill, steps)
    out["prefill_tok_s"] = prompt_tokens / out["prefill_ms"] * 1e3
    eng.check_status("throughput")
    eng.ctx_lens.copy_(torch.tensor(lens, dtype=torch.int32))
    return out


def run(args, build_workload, ClockSampler) -> None:
    eng_mod, lay = pkg("engine"), pkg("layered")
    cfg = lay.CONFIGS[args.model]
    pkg("_lib").load()
    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    lens, table, blocks, max_pages = build_workload(cfg, args.batch, args.gen_tokens, seed=0, ctx_min=args.ctx_min, ctx_max=args.ctx_max)
    prompt_pages = -(-args.prompt_tokens // PAGE)
    max_pages = max(max_pages, prompt_pages)
    spare = blocks
    blocks += prompt_pages
    lens_np = np.array(lens)
    gen = torch.Generator(device=dev).manual_seed(5)
    sizes = dict(num_blocks=blocks, max_batch=args.batch, max_pages_per_seq=max_pages, device=dev)
    chunk_first, chunk_n = max(0, args.prompt_tokens - 2048), min(2048, args.prompt_tokens)
    att = next(s.mixer.left for s in cfg.layer_list if hasattr(s.mixer, "left")) if cfg.gated else \
        next(s.mixer for s in cfg.layer_list if isinstance(s.mixer, lay.AttentionSpec))

    eng = lay.LayeredEngine(cfg, **sizes)
    fill(eng, gen)
    with ClockSampler(0) as clocks:
        mine = throughput(eng, args, table, lens, args.prompt_tokens, spare, clocks)
    clock_info = clocks.summary()
    if cfg.gated:
        import bench_gated
        mine["decode_kernels"] = bench_gated.decode_kernels(eng, args.batch, lens_np)
        mine["prompt_kernels"] = bench_gated.prompt_kernels(eng, chunk_first, chunk_n)
        mine["state_bytes_per_sequence"] = eng.state_bytes_per_sequence()
    else:
        mine["decode_kernels"] = decode_kernels(eng, args.batch, lens_np)
        mine["prompt_kernels"] = prompt_kernels(eng, chunk_first, chunk_n)
    launches, kv = eng.kernel_launches_per_step, eng.kv_bytes_per_token()
    del eng
    torch.cuda.empty_cache()

    base = eng_mod.CONFIGS["qwen3-30b-a3b" if cfg.width <= 2048 else "qwen3-235b-a22b"]
    like = eng_mod.ModelConfig("qwen3-moe-like", cfg.vocab_size, cfg.width, cfg.layers, att.heads, att.kv_heads, att.dim, base.experts,
                               base.top_k, base.moe_inter)
    eng = eng_mod.DecodeEngine(like, **sizes)
    fill(eng, gen)
    other = throughput(eng, args, table, lens, args.prompt_tokens, spare, None)
    other["decode_kernels"], other["prompt_kernels"] = qwen_kernels(eng, args.batch, lens_np, chunk_first, chunk_n)
    B = args.batch
    t = Table()
    line = {"metric": "decode tok/s", "value": mine["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
            "warmup": max(3, args.warmup), "ms_per_step": mine["decode_ms"], "higher_is_better": True, "scaling": "weak",
            "vs_baseline": None, "dtype": "bf16 (fp32 residual, norms, scores)", "data": "synthetic",
            "config": {"workload": f"{args.model} ({cfg.layers} layers, random weights) decode, {B} sequences, contexts "
                                   f"U{{{args.ctx_min}..{args.ctx_max}}}, page {PAGE}; prompts of {args.prompt_tokens} tokens; beside "
                                   f"qwen3-moe of the same width, heads, layers and vocabulary",
                       "mean_ctx": float(lens_np.mean()), "kv_bytes_per_token": kv, "peaks": [t.hbm, t.tf, t.source],
                       "l2": "every step and every round of kernel launches reads far more than the 126 MB L2"},
            "e2e": {"value": mine["decode_e2e_tok_s"], "unit": "tok/s", "h2d_bytes_per_step": B * 8, "d2h_bytes_per_step": B * 8,
                    "api": "B200Backend.decode_step_batched"},
            "gpu_launches": launches * args.steps, "clocks": clock_info, "layered": mine, "closest_model": other}
    print(json.dumps(line))
