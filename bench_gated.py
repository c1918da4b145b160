"""Kernel tables of gated layer-list decoders (Sefalorn) for `bench.py --model sefalorn-...`; bench_layered.py runs them and
prints the line.  As there: every kernel is launched once per layer on that layer's own weights, pages and states, between
CUDA events, and its roofline is the longer of its bytes at the measured copy bandwidth and its flops at the measured bf16
rate.  A recurrence counts the products of the plain recurrence (state against key and query, and the rank-one update)."""
from __future__ import annotations

import numpy as np
import torch

from bench_layered import PAGE, Table, pkg


def window_pairs(positions, window: int) -> int:
    return int(np.minimum(np.asarray(positions) + 1, window).sum())


def kernels(eng, rows, positions, ids: dict, decode: bool) -> dict:
    """Each kernel of one pass over `rows` (gated.Rows) whose positions are `positions` (host)."""
    g, ops, cfg = pkg("gated"), pkg("ops"), eng.cfg
    t = Table()
    dev, W, n = eng.device, eng.W, rows.pos.shape[0]
    bf = dict(device=dev, dtype=torch.bfloat16)
    f32 = dict(device=dev, dtype=torch.float32)
    x, d, h, gate, y = torch.randn(n, W, **f32), torch.randn(n, W, **bf), torch.randn(n, W, **bf), torch.rand(n, W, **bf), torch.empty(n, W, **bf)
    pend = g.Pending(gate, dense=d)
    t.add("residual gate + layer norm", [lambda w=w: ops.residual_norm(x, pend, w.norm1, cfg.norm_eps, cfg.width, out=h)
                                         for w in eng.layers], n * W * (8 + 2 + 2 + 2), 0)
    h.normal_()
    for kind in ("parallel", "lightning"):
        li = ids[kind]
        if not li:
            continue
        m, w0 = cfg.layer_list[li[0]].mixer, eng.layers[li[0]]
        N = w0.wproj.shape[0]
        H, S = w0.heads, w0.d * w0.dv
        out = torch.randn(n, w0.out_ld, **bf)
        act = torch.randn(n, w0.channels, **bf)
        gt = torch.rand(n, H * w0.dv, **bf)
        o = torch.empty(n, H, w0.dv, **f32)
        if kind == "parallel":
            a, r = m.left, m.right
            q, pre, ba = torch.empty(n, a.heads, w0.Dk, **bf), torch.randn(n, w0.channels, **bf), torch.randn(n, 2 * H, **f32)

            def proj(i):
                w = eng.layers[i]
                ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, q), (ops.SEG_PAGES, eng.k_pools[i]), (ops.SEG_PAGES, eng.v_pools[i]),
                                            (ops.SEG_ROWS, pre), (ops.SEG_ROWS, gt, ops.ACT_SILU), (ops.SEG_ROWS, gate, ops.ACT_SIGMOID),
                                            (ops.SEG_F32, ba)], positions=rows.pos, block_table=rows.table, status=eng.status,
                               col_bias=w.proj_bias)

            t.add("parallel projection + page write", [lambda i=i: proj(i) for i in li], N * W * 2 + n * (W + N) * 2, 2 * n * N * W)
            q.normal_().mul_(a.dim ** -0.5)
            seen = window_pairs(positions, a.window)
            kv = a.kv_heads * (w0.Dk + w0.Dv) * 2
            read = seen * kv if decode else n * kv
            t.add("windowed attention with mixed heads (all its kernels)",
                  [lambda i=i: eng._window_attention(q, eng.k_pools[i], eng.v_pools[i], a, eng.layers[i], rows, 1.0, out) for i in li],
                  read + n * a.heads * (w0.Dk + w0.Dv) * 2, 2 * seen * a.heads * (w0.Dk + w0.Dv))
            pre.normal_()
            if not decode:
                t.add("convolution + SiLU", [lambda i=i: ops.conv_silu(pre, eng.layers[i].conv, eng.rings[i], rows.slots, rows.pos, True,
                                                                       eng.status, act) for i in li], n * w0.channels * 4, 0)
                act.normal_()
            ba.normal_()
        else:
            ba = None

            def proj(i):
                w = eng.layers[i]
                ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, act, ops.ACT_SILU), (ops.SEG_ROWS, gt, ops.ACT_SIGMOID),
                                            (ops.SEG_ROWS, gate, ops.ACT_SIGMOID)], status=eng.status, col_bias=w.proj_bias)

            t.add("lightning projection", [lambda i=i: proj(i) for i in li], N * W * 2 + n * (W + N) * 2, 2 * n * N * W)
            act.normal_()
        moved = n * H * S * 8 if decode else H * S * 8
        flops = (6 if kind == "parallel" else 4) * n * H * S
        if kind == "parallel" and decode:
            t.add("gated delta rule with convolution, head norm and gate", [
                lambda i=i: eng._delta(pre, ba, gt, i, m.right, eng.layers[i], rows, 1.0, out[:, m.left.heads * w0.Dv:]) for i in li],
                moved + n * (w0.channels * (2 + 2 * m.right.taps) + H * w0.dv * 4), flops)
        else:
            t.add("gated delta rule" if kind == "parallel" else "lightning recurrence",
                  [lambda i=i: eng._recurrence(act, i, eng.layers[i], rows, 0, n, not decode, o, ba, 0.1) for i in li],
                  moved + n * (w0.channels * 2 + H * w0.dv * 4), flops)
        if kind == "parallel":
            args = (m.right.vdim, True, 1.0, out[:, m.left.heads * w0.Dv:])
            og = o.normal_()
        else:
            args = (H * m.vdim, False, 1.0, out)
            og = o.normal_().view(n, 1, -1)
        if not (kind == "parallel" and decode):
            t.add(f"{kind}: head norm and gate", [lambda i=i: ops.group_norm_gate(og, eng.layers[i].head_norm, gt, cfg.norm_eps, *args) for i in li],
                  n * H * w0.dv * 8, 0)
        t.add(f"{kind} output projection", [lambda i=i: ops.dense_gemm(out, eng.layers[i].wo, out=y, status=eng.status, workspace=eng.gemm_ws)
                                            for i in li], W * w0.out_ld * 2 + n * (W + w0.out_ld) * 2, 2 * n * W * w0.out_ld)
    moe = [i for i, s in enumerate(cfg.layer_list) if s.mlp is not None]
    e, w0 = cfg.layer_list[moe[0]].mlp, eng.layers[moe[0]]
    logits = torch.empty(n, e.experts, **f32)
    t.add("router + second gate", [lambda i=i: ops.proj_split(h, eng.layers[i].w_route, [(ops.SEG_ROWS, gate, ops.ACT_SIGMOID), (ops.SEG_F32, logits)],
                                                              status=eng.status, col_bias=eng.layers[i].route_bias) for i in moe],
          (W + e.experts) * W * 2 + n * W * 4 + n * e.experts * 4, 2 * n * (W + e.experts) * W)
    lg = torch.randn(n, e.experts, **f32)
    ids_, pw = ops.moe_route_sigmoid(lg, e.top, e.scale)
    t.add("routing", [lambda: ops.moe_route_sigmoid(lg, e.top, e.scale)] * 4, n * e.experts * 4, 0)
    ws = eng._moe_workspace(n, e)
    t.add("ranks, scatter and row copy", [lambda: ops.moe_permute_copy(ids_, h, e.experts, ws)] * 4, n * W * 2 * (1 + e.top), 0)
    perm = ops.moe_permute_copy(ids_, h, e.experts, ws)
    hit, F = int(torch.unique(ids_).numel()), w0.w_down.shape[2]
    a13 = ops.moe_gate_up(perm, w0.w_gate_up, eng.status)
    pairs = n * e.top
    t.add("experts gate/up + gated unit (bf16)", [lambda i=i: ops.moe_gate_up(perm, eng.layers[i].w_gate_up, eng.status) for i in moe],
          hit * 2 * F * W * 2 + pairs * (W + F) * 2, 4 * pairs * F * W)
    yr = ops.moe_down(perm, a13, w0.w_down, eng.status)
    t.add("experts down (bf16)", [lambda i=i: ops.moe_down(perm, a13, eng.layers[i].w_down, eng.status) for i in moe],
          hit * F * W * 2 + pairs * (W + F) * 2, 2 * pairs * F * W)
    pe = g.Pending(gate, expert_rows=yr, row_of_pair=perm.row_of_pair, pair_weight=pw)
    t.add("experts' sum + gate + layer norm", [lambda w=w: ops.residual_norm(x, pe, w.norm1, cfg.norm_eps, cfg.width, out=h) for w in eng.layers],
          n * W * (8 + 2 * e.top + 2 + 2), 0)
    if decode:
        h.normal_()
        t.add("lm_head + arg-max", [lambda: eng._pick(h)] * 4, eng.lm_head.numel() * 2 + n * W * 2, 2 * n * eng.lm_head.numel())
    eng.check_status("kernels")
    return t.rows


def layer_ids(cfg) -> dict:
    g = pkg("gated")
    par = [i for i, s in enumerate(cfg.layer_list) if isinstance(s.mixer, g.ParallelSpec)]
    return {"parallel": par, "lightning": [i for i in range(cfg.layers) if i not in par]}


def decode_kernels(eng, B: int, lens) -> dict:
    rows = pkg("gated").Rows(eng.ctx_lens[:B], eng.block_table[:B], eng.state_slots[:B])
    return kernels(eng, rows, lens, layer_ids(eng.cfg), True)


def prompt_kernels(eng, first: int, n: int) -> dict:
    dev, ctx = eng.device, first + n
    row = torch.zeros(eng.max_pages, dtype=torch.int32, device=dev)
    row[: -(-ctx // PAGE)] = torch.randperm(eng.num_blocks, device=dev)[: -(-ctx // PAGE)].int()
    rows = pkg("gated").Rows(torch.arange(first, ctx, dtype=torch.int32, device=dev), row[None].expand(n, -1).contiguous(),
                             torch.zeros(n, dtype=torch.int32, device=dev), first, n)
    return kernels(eng, rows, np.arange(first, ctx), layer_ids(eng.cfg), False)
