"""Mechanisms of gated layer-list decoders (design: Sefalorn) for the engine in ``layered.py``: sliding-window attention with
mixed heads, the gated delta rule, lightning attention, routed experts in bf16 or fp32, and the gated residual.

    per layer   x += sigmoid(R1 h + b1) * mixer(h), h = norm1 x;   x += sigmoid(R2 h + b2) * experts(h), h = norm2 x
    logits      = logit_scale * head norm(x)                      (norm: layer norm without a bias)

Weights in run-time form (`GatedWeights`): everything that reads the same h is one product - a mixer's maps with the residual
gate's, the router with the second gate's -, split in the epilogue, where biases and the gates' activations are applied too.
Sizes are padded with zero rows and columns that change no result: per-head key and value sizes of attention to multiples of
64, those of a recurrence to 16, an output map's input to 64, an expert's inner size to 128.

Scores mixed over the heads are linear in the queries, so the mixing matrix moves to the queries (``ops.mix_heads``: a head's
query becomes one vector over the keys of all kv heads, made inside the attention kernels where they can) and the distance
penalty becomes one table per head over the window (csrc/mixed_attn.cu).

State.  Attention keeps K/V in pages like every other layer.  A recurrence keeps a matrix per head, and its convolution the
last inputs, in a slot per sequence (csrc/state_scan.cu, csrc/gated_glue.cu); both can be stepped twice from the same position,
and neither needs clearing when a slot changes hands.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import ops

PAGE = 16
# Prompt chunks of fewer tokens than this run a recurrence token by token; longer ones in blocks of 64 on the tensor cores.
BLOCKED_ROWS = 32
SILU_GLU = dict(limit=float("inf"), alpha=1.0, shift=0.0)  # the clamped gated unit as silu(g) * u


# -------------------------------------------------------------- configuration


@dataclass(frozen=True)
class WindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int


@dataclass(frozen=True)
class DeltaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class ParallelSpec:
    left: WindowAttentionSpec
    right: DeltaSpec
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    inner: int
    scale: float


def mixer_from_json(kind: str, m: dict):
    if kind == "parallel":
        a, r = m["left"], m["right"]
        for side in (a, r):
            if side["heads"] % side["kv_heads"]:
                raise ValueError(f"{side['heads']} heads over {side['kv_heads']} kv heads")
        if a["mask"]["size"] < 1 or r["conv"] < 1:
            raise ValueError("a window or a convolution of no tokens")
        return ParallelSpec(WindowAttentionSpec(a["heads"], a["kv_heads"], a["dim"], a["vdim"], float(a["scale"]), a["mask"]["size"]),
                            DeltaSpec(r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]),
                            float(m["left_scale"]), float(m["right_scale"]))
    if kind == "lightning":
        if len(m["decay"]) != m["heads"]:
            raise ValueError(f"{len(m['decay'])} decays for {m['heads']} heads")
        return LightningSpec(m["heads"], m["dim"], m["vdim"], tuple(float(d) for d in m["decay"]))
    raise ValueError(f"unknown mixer {kind!r}")


def mlp_from_json(m: dict | None):
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward {m['kind']!r}")
    r = m["router"]
    if not 1 <= r["top"] <= r["experts"]:
        raise ValueError(f"top {r['top']} of {r['experts']} experts")
    return MoeSpec(r["experts"], r["top"], m["expert"]["ff"], float(r["scale"]))


def layer_shapes(spec, W: int) -> dict[str, tuple[int, ...]]:
    """Names (after the layer's prefix) and shapes of one layer's tensors."""
    out = {"norm1": (W,), "rg1": (W, W), "rg1.b": (W,)}
    m = spec.mixer
    if isinstance(m, ParallelSpec):
        a, r = m.left, m.right
        for name, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
            out["mix.left." + name], out[f"mix.left.{name}.b"] = (rows, W), (rows,)
        out.update({"mix.left.r1": (a.heads,), "mix.left.r2": (a.heads,), "mix.left.talk": (a.heads, a.heads),
                    "mix.left.o": (W, a.heads * a.vdim), "mix.left.o.b": (W,)})
        for name, rows in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", r.heads * r.vdim)):
            out["mix.right." + name], out[f"mix.right.{name}.conv"] = (rows, W), (rows, r.taps)
        out.update({"mix.right.b": (r.heads, W), "mix.right.a": (r.heads, W), "mix.right.A_log": (r.heads,),
                    "mix.right.dt_bias": (r.heads,), "mix.right.norm": (r.vdim,), "mix.right.g": (r.heads * r.vdim, W),
                    "mix.right.o": (W, r.heads * r.vdim)})
    else:
        for name, rows in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("g", m.heads * m.vdim)):
            out["mix." + name] = (rows, W)
        out.update({"mix.o": (W, m.heads * m.vdim), "mix.norm": (m.heads * m.vdim,)})
    if spec.mlp is not None:
        out.update({"norm2": (W,), "rg2": (W, W), "rg2.b": (W,), "mlp.router": (spec.mlp.experts, W)})
        for e in range(spec.mlp.experts):
            out[f"mlp.e{e}.gate"] = out[f"mlp.e{e}.up"] = (spec.mlp.inner, W)
            out[f"mlp.e{e}.down"] = (W, spec.mlp.inner)
    return out


# -------------------------------------------------------------------- weights


def _up(n: int, k: int) -> int:
    return -(-n // k) * k


def _heads(t: torch.Tensor, heads: int, size: int, to: int) -> torch.Tensor:
    """[heads * size, ...] -> [heads * to, ...], zero rows after each head's own."""
    if size == to:
        return t
    out = t.new_zeros(heads, to, *t.shape[1:])
    out[:, :size] = t.view(heads, size, *t.shape[1:])
    return out.view(heads * to, *t.shape[1:])


def _pad(t: torch.Tensor, dim: int, to: int) -> torch.Tensor:
    if t.shape[dim] == to:
        return t
    shape = list(t.shape)
    shape[dim] = to
    out = t.new_zeros(shape)
    out.narrow(dim, 0, t.shape[dim]).copy_(t)
    return out


def distance_table(talk: torch.Tensor, r1: torch.Tensor, r2: torch.Tensor, distances: int) -> torch.Tensor:
    """What the mixed score of a head loses at each distance, sum_g talk[h, g] r1_g ln(1 + r2_g d), d < distances, as the
    attention kernels take it (`ops.pad_distances`)."""
    d = torch.arange(distances, dtype=torch.float64, device=talk.device)
    own = r1.double()[:, None] * torch.log1p(r2.double()[:, None] * d[None])
    return ops.pad_distances(talk.double() @ own)


class Projection:
    """Maps of one input as one product: blocks of output features with the places they go to."""

    def __init__(self, W: int):
        self.W, self.rows, self.bias, self.any_bias = W, [], [], False

    def add(self, w: torch.Tensor, bias: torch.Tensor | None = None) -> None:
        self.rows.append(_pad(w, 1, self.W))
        self.bias.append(torch.zeros(w.shape[0], device=w.device) if bias is None else bias.float())
        self.any_bias = self.any_bias or bias is not None

    def finish(self, dtype):
        w = torch.cat(self.rows).to(dtype).contiguous()
        return w, torch.cat(self.bias).contiguous() if self.any_bias else None


class GatedWeights:
    """One layer in run-time form (see the module docstring)."""

    def __init__(self, spec, t: dict[str, torch.Tensor], width: int, W: int, max_positions: int, device, dtype):
        m = spec.mixer

        def get(name):
            return t[name].to(device)

        def vec(x, to=None):
            x = x.float()
            return _pad(x, 0, to or x.shape[0]).contiguous()

        self.norm1 = vec(get("norm1"), W)
        proj = Projection(W)
        self.o_bias = None
        if isinstance(m, ParallelSpec):
            a, r = m.left, m.right
            self.Dk, self.Dv = _up(a.dim, 64), _up(a.vdim, 64)
            for name, heads, size, to in (("q", a.heads, a.dim, self.Dk), ("k", a.kv_heads, a.dim, self.Dk),
                                          ("v", a.kv_heads, a.vdim, self.Dv)):
                proj.add(_heads(get("mix.left." + name), heads, size, to), _heads(get(f"mix.left.{name}.b"), heads, size, to))
            talk = get("mix.left.talk").float()
            self.mix, self.talk = (talk * a.scale).contiguous(), talk.to(torch.bfloat16).contiguous()
            self.bias = distance_table(talk, get("mix.left.r1"), get("mix.left.r2"), min(a.window, max_positions))
            self.d, self.dv = _up(r.dim, 16), _up(r.vdim, 16)
            convs = []
            for name, heads, size, to in (("q", r.kv_heads, r.dim, self.d), ("k", r.kv_heads, r.dim, self.d),
                                          ("v", r.heads, r.vdim, self.dv)):
                proj.add(_heads(get("mix.right." + name), heads, size, to))
                convs.append(_heads(get(f"mix.right.{name}.conv"), heads, size, to))
            self.conv = torch.cat(convs).t().to(dtype).contiguous()  # [taps, channels]
            self.channels = self.conv.shape[1]
            proj.add(_heads(get("mix.right.g"), r.heads, r.vdim, self.dv))
            proj.add(_pad(get("rg1"), 0, W), _pad(get("rg1.b"), 0, W))
            proj.add(torch.cat([get("mix.right.b"), get("mix.right.a")]))
            self.a_log, self.dt_bias = vec(get("mix.right.A_log")), vec(get("mix.right.dt_bias"))
            self.head_norm = vec(get("mix.right.norm"), self.dv)
            wo = torch.cat([_heads(get("mix.left.o").t(), a.heads, a.vdim, self.Dv),
                            _heads(get("mix.right.o").t(), r.heads, r.vdim, self.dv)])
            self.o_bias = vec(get("mix.left.o.b").float() * m.left_scale, W)
            self.heads, self.qk_heads, self.blocked = r.heads, r.kv_heads, True
        else:
            self.d, self.dv = _up(m.dim, 16), _up(m.vdim, 16)
            for name, size, to in (("q", m.dim, self.d), ("k", m.dim, self.d), ("v", m.vdim, self.dv), ("g", m.vdim, self.dv)):
                proj.add(_heads(get("mix." + name), m.heads, size, to))
            proj.add(_pad(get("rg1"), 0, W), _pad(get("rg1.b"), 0, W))
            self.channels = m.heads * (2 * self.d + self.dv)
            self.decay = torch.tensor(m.decay, dtype=torch.float32, device=device)
            self.head_norm = vec(_heads(get("mix.norm"), m.heads, m.vdim, self.dv))
            wo = _heads(get("mix.o").t(), m.heads, m.vdim, self.dv)
            self.heads = self.qk_heads = m.heads
            self.blocked = min(m.decay) >= 0.0  # products of decays are summed logarithms there
        self.wproj, self.proj_bias = proj.finish(dtype)
        self.out_cols, self.out_ld = wo.shape[0], _up(wo.shape[0], 64)
        self.wo = _pad(_pad(wo, 0, self.out_ld), 1, W).t().to(dtype).contiguous()
        if spec.mlp is not None:
            e = spec.mlp
            self.norm2 = vec(get("norm2"), W)
            proj = Projection(W)
            proj.add(_pad(get("rg2"), 0, W), _pad(get("rg2.b"), 0, W))
            proj.add(get("mlp.router"))
            self.w_route, self.route_bias = proj.finish(dtype)
            F = _up(e.inner, 128)
            self.w_gate_up = torch.zeros(e.experts, F // 128, 2, 128, W, dtype=dtype, device=device)
            self.w_down = torch.zeros(e.experts, W, F, dtype=dtype, device=device)
            for i in range(e.experts):
                for j, name in enumerate(("gate", "up")):
                    self.w_gate_up[i, :, j] = _pad(_pad(get(f"mlp.e{i}.{name}"), 0, F), 1, W).view(F // 128, 128, W)
                self.w_down[i, :width, : e.inner] = get(f"mlp.e{i}.down")
            self.w_gate_up = self.w_gate_up.view(e.experts, 2 * F, W)


def launches(spec) -> int:
    """Kernels of one layer in a decode step: norm, projection, output projection; mixed queries, attention, its fold, gated delta
    rule, or recurrence and head norm; norm, projection, routing, ranks, scatter, two products of the experts."""
    return 3 + (4 if isinstance(spec.mixer, ParallelSpec) else 2) + (7 if spec.mlp is not None else 0)


# --------------------------------------------------------------------- passes


@dataclass
class Pending:
    """What a sublayer leaves for the residual stream; the norm after it adds it (``ops.residual_norm``)."""

    gate: torch.Tensor
    dense: torch.Tensor | None = None
    bias: torch.Tensor | None = None
    expert_rows: torch.Tensor | None = None
    row_of_pair: torch.Tensor | None = None
    pair_weight: torch.Tensor | None = None


@dataclass
class Rows:
    """The rows of one pass.  With `chunk` > 0 the first `chunk` rows are consecutive tokens, from position `first` on, of the
    sequence with pages table[0] and slot slots[0]; every other row is a decode row of its own sequence."""

    pos: torch.Tensor
    table: torch.Tensor
    slots: torch.Tensor | None
    first: int = 0
    chunk: int = 0

    def parts(self):
        """(lo, hi, is a chunk) of the row ranges."""
        n, R = self.chunk, self.pos.shape[0]
        return ([(0, n, True)] if n else []) + ([(n, R, False)] if n < R else [])


class GatedMechanisms:
    """Part of the engine (``layered.LayeredEngine``); uses its dtype, status word, pools, states and `_linear`."""

    def _init_states(self, num_slots: int) -> None:
        """Slots of the recurrent layers: `num_slots` for sequences, one more for the padding rows of a graph."""
        self.states, self.rings = [], []
        for spec, w in zip(self.cfg.layer_list, self.layers):
            self.states.append(torch.zeros(num_slots + 1, 2, w.heads, w.d, w.dv, dtype=torch.float32, device=self.device))
            taps = spec.mixer.right.taps if isinstance(spec.mixer, ParallelSpec) else 1
            self.rings.append(torch.zeros(num_slots + 1, taps, w.channels, dtype=self.dtype, device=self.device) if taps > 1 else None)
        self._moe_ws: list[torch.Tensor] = []
        self._mixed_ws: dict[tuple, tuple[int, torch.Tensor]] = {}

    def _add_norm(self, x, pending: Pending | None, weight, out=None):
        return ops.residual_norm(x, pending, weight, self.cfg.norm_eps, self.cfg.width, out=out, dtype=self.dtype)

    def _act(self, *shape, dtype=None):
        return torch.empty(*shape, dtype=dtype or self.dtype, device=self.device)

    def _recurrence(self, act, li: int, w: GatedWeights, rows: Rows, lo: int, hi: int, chunk: bool, o, ba=None, q_scale: float = 1.0):
        """Rows [lo, hi) of o [rows, heads, dv] fp32 from activated q, k, v: blocks of tokens on the tensor cores for a long enough
        chunk, token by token otherwise."""
        args = (act[lo:hi], w, self.states[li], rows.slots[lo:hi], rows.pos[lo:hi], o[lo:hi])
        more = dict(ba=None if ba is None else ba[lo:hi], q_scale=q_scale)
        if chunk and hi - lo >= BLOCKED_ROWS and w.blocked and ops.state_chunk_supported(w.d, w.dv, self.dtype):
            ops.state_chunk(*args, self.status, **more)
        elif not chunk and ba is None and ops.state_step_supported(w.d, w.dv):
            ops.state_step(*args, self.status)
        else:
            ops.state_scan(*args, chunk, self.status, **more)

    def _delta(self, pre, ba, g, li: int, r: DeltaSpec, w: GatedWeights, rows: Rows, scale: float, out) -> None:
        """Gated delta rule with its convolution in front and its head norm and gate behind: one kernel for decode rows."""
        q_scale, eps = r.dim ** -0.5, self.cfg.norm_eps
        for lo, hi, chunk in rows.parts():
            at = (rows.slots[lo:hi], rows.pos[lo:hi])
            if not chunk and ops.state_step_supported(w.d, w.dv):
                ops.state_step(pre[lo:hi], w, self.states[li], *at, None, self.status, ba=ba[lo:hi], q_scale=q_scale, ring=self.rings[li],
                               gate=g[lo:hi], eps=eps, size=r.vdim, scale=scale, out=out[lo:hi])
                continue
            act = ops.conv_silu(pre[lo:hi], w.conv, self.rings[li], *at, chunk, self.status)
            o = self._act(hi - lo, w.heads, w.dv, dtype=torch.float32)
            part = Rows(rows.pos[lo:hi], rows.table[lo:hi], rows.slots[lo:hi], rows.first, hi - lo if chunk else 0)
            self._recurrence(act, li, w, part, 0, hi - lo, chunk, o, ba[lo:hi], q_scale)
            ops.group_norm_gate(o, w.head_norm, g[lo:hi], eps, r.vdim, True, scale, out[lo:hi])

    def _parallel(self, h, li: int, m: ParallelSpec, w: GatedWeights, rows: Rows) -> Pending:
        a, r, R = m.left, m.right, h.shape[0]
        f32 = torch.float32
        q = self._act(R, a.heads, w.Dk)
        pre, g = self._act(R, w.channels), self._act(R, r.heads * w.dv)
        gate, ba = self._act(R, self.W), self._act(R, 2 * r.heads, dtype=f32)
        kp, vp = self.k_pools[li], self.v_pools[li]
        ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, q), (ops.SEG_PAGES, kp), (ops.SEG_PAGES, vp), (ops.SEG_ROWS, pre),
                                    (ops.SEG_ROWS, g, ops.ACT_SILU), (ops.SEG_ROWS, gate, ops.ACT_SIGMOID), (ops.SEG_F32, ba)],
                       positions=rows.pos, block_table=rows.table, status=self.status, col_bias=w.proj_bias)
        out = self._act(R, w.out_ld)
        if w.out_ld != w.out_cols:
            out[:, w.out_cols:].zero_()
        self._window_attention(q, kp, vp, a, w, rows, m.left_scale, out)
        self._delta(pre, ba, g, li, r, w, rows, m.right_scale, out[:, a.heads * w.Dv:])
        return Pending(gate, dense=self._linear(out, w.wo), bias=w.o_bias)

    def _window_attention(self, q, kp, vp, a: WindowAttentionSpec, w: GatedWeights, rows: Rows, scale: float, out) -> None:
        shape = (a.heads, a.kv_heads, w.Dk, w.Dv, self.dtype)
        form, decode_mixes = ops.mixed_attn_prefill_form(*shape), ops.mixed_attn_mixes(*shape)
        for lo, hi, chunk in rows.parts():
            if chunk and form:
                args = (kp, vp, a.kv_heads, rows.table[0], rows.first, w.bias, a.window, out[lo:hi], scale, self.status)
                if form == 2:
                    ops.mixed_attn_prefill(q[lo:hi], *args, talk=w.talk, scale=a.scale)
                else:
                    ops.mixed_attn_prefill(ops.mix_heads(q[lo:hi], w.mix, a.kv_heads), *args)
                continue
            split, ws = (None, None) if chunk and self.dtype == torch.bfloat16 else self._mixed_plan(hi - lo, a, w)
            args = (kp, vp, a.kv_heads, rows.table[lo:hi], rows.pos[lo:hi], w.bias, a.window, out[lo:hi], scale, self.status, split, ws)
            if decode_mixes:
                ops.mixed_attn(q[lo:hi], *args, mix=w.mix)
            else:
                ops.mixed_attn(ops.mix_heads(q[lo:hi], w.mix, a.kv_heads), *args)

    def _mixed_plan(self, rows: int, a: WindowAttentionSpec, w: GatedWeights):
        """(tokens per split, workspace) of the decode attention kernel; one workspace per shape and number of rows, kept for the
        graphs that use it."""
        if self.dtype != torch.bfloat16:
            return 0, None
        key = (rows, a, w.Dk, w.Dv)
        if key not in self._mixed_ws:
            split = self._fixed_split or ops.mixed_split_tokens(rows, a.window, self.max_pages * PAGE)
            self._mixed_ws[key] = (split, ops.mixed_attn_workspace(rows, a.heads, a.kv_heads, w.Dk, w.Dv, a.window, self.max_pages, split,
                                                                   self.device))
        return self._mixed_ws[key]

    def _lightning(self, h, li: int, m: LightningSpec, w: GatedWeights, rows: Rows) -> Pending:
        R = h.shape[0]
        act, g, gate = self._act(R, w.channels), self._act(R, m.heads * w.dv), self._act(R, self.W)
        ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, act, ops.ACT_SILU), (ops.SEG_ROWS, g, ops.ACT_SIGMOID),
                                    (ops.SEG_ROWS, gate, ops.ACT_SIGMOID)], status=self.status, col_bias=w.proj_bias)
        o = self._act(R, m.heads, w.dv, dtype=torch.float32)
        for lo, hi, chunk in rows.parts():
            self._recurrence(act, li, w, rows, lo, hi, chunk, o)
        out = self._act(R, w.out_ld)
        if w.out_ld != w.out_cols:
            out[:, w.out_cols:].zero_()
        ops.group_norm_gate(o.view(R, 1, -1), w.head_norm, g, self.cfg.norm_eps, m.heads * m.vdim, False, 1.0, out)
        return Pending(gate, dense=self._linear(out, w.wo))

    def _moe_workspace(self, rows: int, e: MoeSpec) -> torch.Tensor:
        """Grows; a workspace that a captured graph may use stays alive."""
        n = ops.moe_permute_workspace_bytes(rows, e.experts, e.top)
        if not self._moe_ws or self._moe_ws[-1].numel() < n:
            self._moe_ws.append(torch.zeros(n, dtype=torch.uint8, device=self.device))
        return self._moe_ws[-1]

    def _experts(self, h, e: MoeSpec, w: GatedWeights) -> Pending:
        R = h.shape[0]
        gate, logits = self._act(R, self.W), self._act(R, e.experts, dtype=torch.float32)
        ops.proj_split(h, w.w_route, [(ops.SEG_ROWS, gate, ops.ACT_SIGMOID), (ops.SEG_F32, logits)], status=self.status,
                       col_bias=w.route_bias)
        ids, weight = ops.moe_route_sigmoid(logits, e.top, e.scale)
        perm = ops.moe_permute_copy(ids, h, e.experts, self._moe_workspace(R, e))
        a = ops.moe_gate_up(perm, w.w_gate_up, self.status, **SILU_GLU)
        y = ops.moe_down(perm, a, w.w_down, self.status)
        return Pending(gate, expert_rows=y, row_of_pair=perm.row_of_pair, pair_weight=weight)
