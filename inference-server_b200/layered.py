"""Layer-list decoders: models whose config.json lists their layers one by one.  Two designs: Sulepel, described here, and
Sefalorn, whose mechanisms are in ``gated.py``; the engine, its step and its pass over the layers are the same.

    x_p = embed[token_p] + sinusoid(p)
    per layer   x += mixer(short_conv(norm1 x));   x += ff(norm2 x)        (a layer may have no ff)
    logits      = head norm(x)

(Sulepel) with a grouped RMSNorm, a short causal convolution in front of every mixer, mixers of two kinds in any order and of any
sizes - grouped-query attention over the position's own chunk, and latent attention whose cache is one vector per
token -, a sigmoid gate per head on either, and a dense feed-forward with a clamped gated unit.

The engine is a `PagedEngine`: step, CUDA graphs, prompt passes in chunks, merged passes and the page accounting are the
framework's own; here are the configuration, the weights in run-time form, the page pools and one pass over the layers.

State in pages.  Every layer's state is addressed by (page, slot) of the block table, like K/V:
  attention   k_pool, v_pool [blocks, kv_heads, 16, D]
  latent      c_pool [blocks, 16, rank]
  every layer hist [blocks, min(taps, 16), width]: the convolution's last inputs, kept per page (csrc/layer_glue.cu)
so a sequence's state is given back, and taken up by another sequence, with its pages alone.

Run-time form of the weights.  Sizes are padded at load so that the kernels see their granularity, with zero rows and
columns that change no result: width and inner sizes to multiples of 64 (128), per-head query/key and value sizes to one
common D (64 or 128 on the tensor-core attention kernels), the latent rank to a rank its kernel is built for.  All
projections that read the same input are one matrix.

Precision.  dtype bfloat16: matrix operands and the activations between kernels are bf16 with fp32 accumulation;
positions, norms, convolutions, scores, softmax, gates and the residual stream are fp32.  dtype float32: everything is
fp32, on kernels without tensor cores.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import gated, ops
from .engine import PAGE, PagedEngine

GLU_ALPHA = 1.702          # of the design's gated unit
SINUSOID_BASE = 10000.0
# Prompt chunks shorter than this run latent attention as decode rows (each over the latents themselves); longer ones
# form the chunk's keys and values once and use the prompt kernel.
LATENT_EXPAND_ROWS = 32


# -------------------------------------------------------------- configuration


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int  # positions per chunk; 0 = all earlier positions are seen


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    rank: int
    scale: float


@dataclass(frozen=True)
class GluSpec:
    inner: int
    limit: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec | LatentSpec | gated.ParallelSpec | gated.LightningSpec
    mlp: GluSpec | gated.MoeSpec | None


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    vocab_size: int
    width: int
    norm_groups: int
    norm_eps: float
    taps: int                   # of the convolution ahead of every mixer
    layer_list: tuple[LayerSpec, ...]
    gated: bool = False         # Sefalorn: layer norm, gated residual, no convolution ahead of a mixer, no positions added
    logit_scale: float = 1.0

    @property
    def hidden(self) -> int:
        return self.width

    @property
    def layers(self) -> int:
        return len(self.layer_list)

    @staticmethod
    def from_json(c: dict) -> "LayeredConfig":
        if c["architecture"] == "Sefalorn":
            layers = tuple(LayerSpec(gated.mixer_from_json(e["type"], e["mixer"]), gated.mlp_from_json(e.get("mlp")))
                           for e in c["layers"])
            return LayeredConfig(c["architecture"], c["vocab"], c["width"], 1, float(c["norm"]["eps"]), 1, layers, gated=True,
                                 logit_scale=float(c["logit_scale"]))

        def mixer(kind: str, m: dict):
            if kind == "attention":
                mask = m.get("mask")
                spec = AttentionSpec(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                                     mask["size"] if mask else 0)
                if spec.heads % spec.kv_heads:
                    raise ValueError(f"{spec.heads} query heads over {spec.kv_heads} kv heads")
                return spec
            if kind == "latent_attention":
                return LatentSpec(m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"]))
            raise ValueError(f"unknown mixer {kind!r}")

        def mlp(m: dict | None):
            if m is None:
                return None
            if m["kind"] != "dense":
                raise ValueError(f"unknown feed-forward {m['kind']!r}")
            return GluSpec(m["ff"], float(m["limit"]))

        cfg = LayeredConfig(c["architecture"], c["vocab"], c["width"], c["norm"]["groups"], float(c["norm"]["eps"]),
                            c["canon"]["taps"],
                            tuple(LayerSpec(mixer(e["type"], e["mixer"]), mlp(e.get("mlp"))) for e in c["layers"]))
        if cfg.width % cfg.norm_groups:
            raise ValueError(f"width {cfg.width} does not divide into {cfg.norm_groups} norm groups")
        if cfg.taps < 1:
            raise ValueError(f"a convolution of {cfg.taps} taps")
        return cfg

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Names and shapes of a checkpoint's tensors."""
        W = self.width
        out = {"embed": (self.vocab_size, W), "final.norm": (W,), "head": (self.vocab_size, W)}
        for i, layer in enumerate(self.layer_list):
            m, p = layer.mixer, f"l{i}."
            if self.gated:
                out.update({p + name: shape for name, shape in gated.layer_shapes(layer, W).items()})
                continue
            out[p + "norm1"] = (W,)
            out[p + "canon1"] = (W, self.taps)
            out[p + "mix.q"] = (m.heads * m.dim, W)
            if isinstance(m, AttentionSpec):
                out[p + "mix.k"] = (m.kv_heads * m.dim, W)
                out[p + "mix.v"] = (m.kv_heads * m.vdim, W)
                out[p + "mix.temp"] = (m.heads,)
            else:
                out[p + "mix.dkv"] = (m.rank, W)
                out[p + "mix.dkv.norm"] = (m.rank,)
                out[p + "mix.uk"] = (m.heads * m.dim, m.rank)
                out[p + "mix.uv"] = (m.heads * m.vdim, m.rank)
            out[p + "mix.g"] = (m.heads, W)
            out[p + "mix.o"] = (W, m.heads * m.vdim)
            if layer.mlp is not None:
                out[p + "norm2"] = (W,)
                out[p + "mlp.gate"] = (layer.mlp.inner, W)
                out[p + "mlp.up"] = (layer.mlp.inner, W)
                out[p + "mlp.down"] = (W, layer.mlp.inner)
        return out


def uniform_config(name: str, vocab: int, width: int, groups: int, taps: int, pattern: str, heads: int, kv_heads: int,
                   dim: int, chunk: int, latent_heads: int, rank: int, inner: int, limit: float) -> LayeredConfig:
    """A built-in shape: `pattern` has a letter per layer, a = attention, l = latent attention."""
    a = AttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, chunk)
    lat = LatentSpec(latent_heads, dim, dim, rank, dim ** -0.5)
    glu = GluSpec(inner, limit)
    return LayeredConfig(name, vocab, width, groups, 1e-6, taps,
                         tuple(LayerSpec(a if ch == "a" else lat, glu) for ch in pattern))


def gated_config(name: str, vocab: int, width: int, pattern: str, heads: int, kv_heads: int, dim: int, window: int,
                 state_heads: int, state_dim: int, taps: int, experts: int, top: int, inner: int) -> LayeredConfig:
    """A built-in Sefalorn shape: `pattern` has a letter per layer, p = parallel, l = lightning."""
    par = gated.ParallelSpec(gated.WindowAttentionSpec(heads, kv_heads, dim, dim, dim ** -0.5, window),
                             gated.DeltaSpec(state_heads, state_heads, state_dim, state_dim, taps), 1.0, 1.0)
    light = gated.LightningSpec(state_heads, state_dim, state_dim,
                                tuple(1.0 - 2.0 ** -(2 + 8 * i / max(1, state_heads - 1)) for i in range(state_heads)))
    moe = gated.MoeSpec(experts, top, inner, 1.0)
    return LayeredConfig(name, vocab, width, 1, 1e-6, 1, tuple(LayerSpec(par if ch == "p" else light, moe) for ch in pattern),
                         gated=True)


# Shapes for benchmarks with random weights.
CONFIGS = {
    # the width, heads and vocabulary of qwen3-30b-a3b, 12 layers
    "sulepel-2048": uniform_config("sulepel-2048", 151936, 2048, 4, 4, "aaal" * 3, 32, 4, 128, 2048, 16, 512, 6144, 7.0),
    # the width, attention heads, experts and vocabulary of qwen3-30b-a3b, 8 layers
    "sefalorn-2048": gated_config("sefalorn-2048", 151936, 2048, "plpl" * 2, 32, 4, 128, 1024, 16, 128, 4, 128, 8, 768),
    # the width, attention heads and experts of qwen3-235b-a22b, 4 layers
    "sefalorn-4096": gated_config("sefalorn-4096", 151936, 4096, "plpl", 64, 4, 128, 2048, 32, 128, 4, 128, 8, 1536),
    # the width and heads of qwen3-235b-a22b, 8 layers
    "sulepel-4096": uniform_config("sulepel-4096", 151936, 4096, 8, 4, "aaal" * 2, 64, 4, 128, 4096, 32, 512, 12288, 7.0),
}


# -------------------------------------------------------------------- weights


def _up(n: int, k: int) -> int:
    return -(-n // k) * k


def pad_width(n: int) -> int:
    return _up(n, 64)


def pad_head(n: int) -> int:
    """Common per-head size of queries, keys and values: what the tensor-core kernels are built for, else a multiple of 64
    for the generic one."""
    return 64 if n <= 64 else _up(n, 128) if n <= 128 else _up(n, 64)


def pad_rank(n: int) -> int:
    for r in (64, 128, 192, 256, 384, 512):
        if n <= r:
            return r
    return _up(n, 64)


def _rows(t: torch.Tensor, heads: int, size: int, to: int) -> torch.Tensor:
    """[heads * size, n] -> [heads * to, n], zero rows after each head's own."""
    if size == to:
        return t
    out = t.new_zeros(heads, to, t.shape[1])
    out[:, :size] = t.view(heads, size, -1)
    return out.view(heads * to, -1)


def _cols(t: torch.Tensor, to: int) -> torch.Tensor:
    if t.shape[-1] == to:
        return t
    out = t.new_zeros(*t.shape[:-1], to)
    out[..., : t.shape[-1]] = t
    return out


def interleave_glu(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[F, n] twice -> [2 * F', n], F' = F up to a multiple of 128: 128 gate rows, the 128 up rows of the same features, ..."""
    F, n = gate.shape
    Fp = _up(F, 128)
    out = gate.new_zeros(Fp // 128, 2, 128, n)
    for j, t in enumerate((gate, up)):
        p = t.new_zeros(Fp, n)
        p[:F] = t
        out[:, j] = p.view(-1, 128, n)
    return out.view(2 * Fp, n)


class LayeredWeights:
    """One layer in run-time form (see the module docstring)."""

    def __init__(self, spec: LayerSpec, t: dict[str, torch.Tensor], cfg: LayeredConfig, device, dtype):
        W, m = pad_width(cfg.width), spec.mixer

        def dev(x):
            return x.to(device=device, dtype=dtype).contiguous()

        def get(name):
            return t[name].to(device)

        self.norm1 = dev(_cols(get("norm1"), W))
        self.conv = dev(_cols(get("canon1").t().contiguous(), W))  # [taps, W]
        D = self.D = pad_head(max(m.dim, m.vdim))
        q = _rows(get("mix.q"), m.heads, m.dim, D)
        g = get("mix.g")
        # a negative scale goes into the queries, the kernels' running maximum wants a positive one
        sign = -1.0 if m.scale < 0 else 1.0
        self.scale = abs(m.scale)
        o = get("mix.o").t().contiguous()  # [heads * vdim, width]
        self.wo = dev(_cols(_rows(o, m.heads, m.vdim, D), W).t())
        if isinstance(m, AttentionSpec):
            k = _rows(get("mix.k"), m.kv_heads, m.dim, D)
            v = _rows(get("mix.v"), m.kv_heads, m.vdim, D)
            self.wproj = dev(_cols(torch.cat([q, k, v, g]), W))
            scale = torch.ones(self.wproj.shape[0], dtype=torch.float32, device=device)
            scale[: m.heads * D] = (get("mix.temp").float() * sign).repeat_interleave(D)
            self.col_scale = scale
        else:
            R = self.R = pad_rank(m.rank)
            dkv = _rows(get("mix.dkv"), 1, m.rank, R)
            self.wproj = dev(_cols(torch.cat([q, dkv, g]), W))
            self.col_scale = None
            if sign < 0:
                self.col_scale = torch.ones(self.wproj.shape[0], dtype=torch.float32, device=device)
                self.col_scale[: m.heads * D] = -1.0
            self.c_norm = dev(_cols(get("mix.dkv.norm"), R))
            uk = _cols(_rows(get("mix.uk"), m.heads, m.dim, D), R)  # [H * D, R]
            uv = _cols(_rows(get("mix.uv"), m.heads, m.vdim, D), R)
            self.wuk_t = dev(uk.view(m.heads, D, R).transpose(1, 2).contiguous())  # [H, R, D]
            self.wuv = dev(uv.view(m.heads, D, R))
            # both maps as one projection of the latents, for prompt chunks
            self.wukv = dev(torch.cat([uk, uv])) if dtype == torch.bfloat16 else None
        if spec.mlp is not None:
            self.norm2 = dev(_cols(get("norm2"), W))
            self.wgu = dev(_cols(interleave_glu(get("mlp.gate"), get("mlp.up")), W))
            self.wdown = dev(_rows(_cols(get("mlp.down"), _up(spec.mlp.inner, 128)), 1, cfg.width, W))


def sinusoid_tables(width: int, ld: int, max_pos: int, device) -> tuple[torch.Tensor, torch.Tensor]:
    """(lo [64, ld], hi [ceil(max_pos / 64), ld]) fp32, computed in fp64: columns 2i, 2i+1 hold sin and cos of
    p * base^(-2i/width) for p = 0..63 and for the multiples of 64.  sin and cos of any position follow by the addition
    theorem, so no table of max_pos rows is kept and no angle is rounded to fp32."""
    half = (width + 1) // 2
    freq = torch.pow(torch.tensor(SINUSOID_BASE, dtype=torch.float64), -2.0 * torch.arange(half, dtype=torch.float64) / width)

    def table(p: torch.Tensor) -> torch.Tensor:
        ang = p.double()[:, None] * freq[None]
        t = torch.zeros(len(p), ld, dtype=torch.float32)
        t[:, 0:2 * half:2] = ang.sin().float()
        t[:, 1:2 * half:2] = ang.cos().float()
        return t.to(device)

    return table(torch.arange(64)), table(torch.arange(-(-max_pos // 64)) * 64)


# --------------------------------------------------------------------- engine


class LayeredEngine(gated.GatedMechanisms, PagedEngine):
    """A layer-list decoder on the paged step: weights, pools and one pass over the layers."""

    logits_dtype = torch.float32
    prompt_chunk = 2048

    def __init__(self, cfg: LayeredConfig, num_blocks: int, max_batch: int, max_pages_per_seq: int, device="cuda", seed: int = 0,
                 tensors: dict[str, torch.Tensor] | None = None, dtype: torch.dtype = torch.bfloat16, use_graphs: bool = True,
                 graph_buckets: bool = True, keep_logits: bool = False, split_tokens: int | None = None,
                 num_slots: int | None = None):
        """`tensors`: a checkpoint's tensors (any device); random weights from `seed` without.  `num_slots`: sequences that may
        hold a recurrent state at a time, max_batch and a few whose prompts are under way unless given."""
        if cfg.gated:
            self.num_slots = max(max_batch, num_slots or max_batch + 4)
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"dtype {dtype}: bfloat16 or float32")
        self._init_step_state(num_blocks, max_batch, max_pages_per_seq, device, use_graphs, keep_logits, graph_buckets)
        self.cfg, self.dtype, self.vocab_size = cfg, dtype, cfg.vocab_size
        self.W = pad_width(cfg.width)
        if self.W > 8192:
            raise ValueError(f"width {cfg.width} is above the norm kernel's 8192")
        if tensors is not None:
            self._check_tensors(tensors)
        gen = torch.Generator(device=self.device).manual_seed(seed)
        shapes = cfg.tensor_shapes()

        def fetch(name):
            if tensors is not None:
                return tensors[name]
            shape = shapes[name]
            if len(shape) == 1:
                return torch.ones(shape, device=self.device, dtype=torch.bfloat16)
            return (torch.randn(shape, device=self.device, generator=gen) * 0.02).bfloat16()

        self.layers = []
        for i, spec in enumerate(cfg.layer_list):
            p = f"l{i}."
            t = {n[len(p):]: fetch(n) for n in shapes if n.startswith(p)}
            if cfg.gated:
                self.layers.append(gated.GatedWeights(spec, t, cfg.width, self.W, max_pages_per_seq * PAGE, self.device, dtype))
            else:
                self.layers.append(LayeredWeights(spec, t, cfg, self.device, dtype))

        def table(name):
            return _cols(fetch(name).to(self.device), self.W).to(dtype).contiguous()

        self.embed, self.lm_head = table("embed"), table("head")
        if cfg.gated:
            # the logits' factor goes with the norm's fp32 weight
            self.final_norm = (_cols(fetch("final.norm").to(self.device).float(), self.W) * cfg.logit_scale).contiguous()
            self.sinusoid = _up(max_pages_per_seq * PAGE, 64)
        else:
            self.final_norm = table("final.norm")
            self.sinusoid = sinusoid_tables(cfg.width, self.W, max_pages_per_seq * PAGE, self.device)

        nb = num_blocks + (1 if self.scratch_block is not None else 0)

        def pool(*shape):
            return torch.zeros(nb, *shape, device=self.device, dtype=dtype)

        self.k_pools, self.v_pools, self.c_pools, self.hist = [], [], [], []
        for spec, w in zip(cfg.layer_list, self.layers):
            if cfg.gated:
                a = getattr(spec.mixer, "left", None)
                # 64-wide columns of all heads, see csrc/mixed_attn.cu
                self.k_pools.append(pool(a.kv_heads * w.Dk // 64, PAGE, 64) if a else None)
                self.v_pools.append(pool(a.kv_heads * w.Dv // 64, PAGE, 64) if a else None)
                continue
            attn = isinstance(spec.mixer, AttentionSpec)
            self.k_pools.append(pool(spec.mixer.kv_heads, PAGE, w.D) if attn else None)
            self.v_pools.append(pool(spec.mixer.kv_heads, PAGE, w.D) if attn else None)
            self.c_pools.append(None if attn else pool(PAGE, w.R))
            self.hist.append(pool(min(cfg.taps, PAGE), self.W) if cfg.taps > 1 else None)

        if cfg.gated:
            self._init_states(self.num_slots)
        self._fixed_split = split_tokens
        self.status = torch.zeros(64, dtype=torch.int32, device=self.device)  # glue kernels, projections
        widest = max([self.W] + [w.wproj.shape[0] for w in self.layers])
        self.gemm_ws = ops.dense_gemm_workspace(min(max_batch, 256), widest, self.device) if dtype == torch.bfloat16 else None
        self.argmax_ws = ops.lm_head_argmax_workspace(self.device) if dtype == torch.bfloat16 else None
        self._row_ws: dict[int, tuple[dict, torch.Tensor]] = {}
        self._kv_scratch: dict[tuple[int, int], tuple] = {}
        if cfg.gated:
            self.kernel_launches_per_step = 4 + sum(gated.launches(s) for s in cfg.layer_list)
            return
        # kernels of one decode step: embedding, final norm, lm_head arg-max and its fold; per layer norm + convolution,
        # projection, attention, its fold, output projection (+ latents' norm, two maps per head), norm, two products
        self.kernel_launches_per_step = 4 + sum(
            5 + (0 if isinstance(s.mixer, AttentionSpec) else 3) + (3 if s.mlp is not None else 0) for s in cfg.layer_list)

    def _check_tensors(self, tensors) -> None:
        want = self.cfg.tensor_shapes()
        missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
        if missing or extra:
            raise ValueError(f"checkpoint does not fit its config: missing {missing[:5]}, not known {extra[:5]}")
        for name, shape in want.items():
            if tuple(tensors[name].shape) != shape:
                raise ValueError(f"{name} is {tuple(tensors[name].shape)}, the config says {shape}")

    # ------------------------------------------------------------ workspaces
    def _attn_for(self, rows: int) -> tuple[dict, torch.Tensor]:
        """({layer: tokens per split}, workspace) of the decode attention kernels for `rows` rows."""
        pair = self._row_ws.get(rows)
        if pair is None:
            splits, nbytes = {}, 256
            lib = ops._lib.load()
            max_ctx = self.max_pages * PAGE
            for li, (spec, w) in enumerate(zip(self.cfg.layer_list, self.layers)):
                m = spec.mixer
                if isinstance(m, AttentionSpec):
                    seen = min(max_ctx, m.chunk) if m.chunk else max_ctx
                    split, width = self._fixed_split or ops.default_split_tokens(rows, m.kv_heads, seen), w.D
                else:
                    split, width = self._fixed_split or ops.latent_split_tokens(rows, max_ctx), w.R
                splits[li] = split
                if self.dtype == torch.bfloat16:
                    nbytes = max(nbytes, lib.b200_paged_attn_workspace_bytes(rows, m.heads, width, self.max_pages, PAGE, split))
            pair = (splits, torch.zeros(nbytes, dtype=torch.uint8, device=self.device))
            self._row_ws[rows] = pair
        return pair

    def _expanded_kv(self, heads: int, D: int, pages: int):
        """Scratch pools [pages, heads, 16, D] for the keys and values of a latent layer's context, with the block table
        that lists their pages in order.  Zero where nothing has been written: the prompt kernel multiplies what lies
        past a context's end in its last page by 0."""
        have = self._kv_scratch.get((heads, D))
        if have is None or have[0].shape[0] < pages:
            n = min(self.max_pages, max(pages, 2 * (have[0].shape[0] if have else 0)))
            # the old scratch may still be read by queued kernels: the allocator hands it out again only in stream order
            have = tuple(torch.zeros(n, heads, PAGE, D, dtype=self.dtype, device=self.device) for _ in range(2)) + (
                torch.arange(n, dtype=torch.int32, device=self.device),)
            self._kv_scratch[(heads, D)] = have
        return have

    # ------------------------------------------------------------------ pass
    def _mixer_input(self, x, delta, w: LayeredWeights, hist, pos, table, chunk_of) -> torch.Tensor:
        """x += delta, norm, short convolution: consecutive rows of one sequence as norm then convolution, decode rows in one
        kernel."""
        c = self.cfg
        norm = dict(eps=c.norm_eps, width=c.width, groups=c.norm_groups, status=self.status)
        if chunk_of is None:
            return ops.group_rmsnorm(x, delta, w.norm1, conv_w=w.conv, hist=hist, positions=pos, block_table=table, page=PAGE, **norm)
        first, n = chunk_of
        R = x.shape[0]
        out = torch.empty(R, self.W, dtype=self.dtype, device=self.device)
        h = ops.group_rmsnorm(x[:n], None if delta is None else delta[:n], w.norm1, **norm)
        ops.short_conv(h, w.conv, hist, table[0], first, page=PAGE, status=self.status, out=out[:n])
        if n < R:
            ops.group_rmsnorm(x[n:], None if delta is None else delta[n:], w.norm1, conv_w=w.conv, hist=hist, positions=pos[n:],
                              block_table=table[n:], page=PAGE, out=out[n:], **norm)
        return out

    def _linear(self, x, w):
        if self.dtype == torch.float32:
            return ops.gemm_f32(x, w)
        return ops.dense_gemm(x, w, status=self.status, workspace=self.gemm_ws)

    def _attention(self, h, li: int, m: AttentionSpec, w: LayeredWeights, pos, new_len, table, chunk_of, plan) -> torch.Tensor:
        R, D = h.shape[0], w.D
        q = torch.empty(R, m.heads, D, dtype=self.dtype, device=self.device)
        gate = torch.empty(R, m.heads, dtype=torch.float32, device=self.device)
        kp, vp = self.k_pools[li], self.v_pools[li]
        ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, q), (ops.SEG_PAGES, kp), (ops.SEG_PAGES, vp), (ops.SEG_F32, gate)],
                       w.col_scale, pos, table, self.status)
        out = torch.empty_like(q)
        n = 0
        if chunk_of is not None and ops.paged_attn_prefill_chunked_supported(m.heads, m.kv_heads, D, self.dtype):
            first, n = chunk_of
            ops.paged_attn_prefill_chunked(q[:n], kp, vp, table[0], first, w.scale, self.status, m.chunk, gate[:n], out[:n])
        if n < R:
            splits, ws = plan if plan is not None and n else self._attn_for(R - n)
            ops.paged_attn_decode_chunked(q[n:], kp, vp, table[n:], new_len[n:], w.scale, splits[li], ws, m.chunk, gate[n:], out[n:])
        return self._linear(out.view(R, m.heads * D), w.wo)

    def _latent_rows(self, q, gate, li: int, m: LatentSpec, w: LayeredWeights, new_len, table, plan, out) -> None:
        """Latent attention of rows with a table row each: queries into the latents' space, attention over the latents,
        values of the weighted sums."""
        splits, ws = plan
        qc = ops.grouped_gemm(q, w.wuk_t, m.heads, status=self.status)
        pool = self.c_pools[li]
        if ops.latent_attn_supported(w.R, PAGE, self.dtype):
            oc = ops.latent_attn_decode(qc, pool, table, new_len, w.scale, splits[li], ws, gate)
        else:
            one = pool.view(pool.shape[0], 1, PAGE, w.R)
            oc = ops.paged_attn_decode_chunked(qc, one, one, table, new_len, w.scale, splits[li], ws, 0, gate)
        ops.grouped_gemm(oc, w.wuv, m.heads, out=out, status=self.status)

    def _latent(self, h, li: int, m: LatentSpec, w: LayeredWeights, pos, new_len, table, chunk_of, plan) -> torch.Tensor:
        R, D = h.shape[0], w.D
        q = torch.empty(R, m.heads, D, dtype=self.dtype, device=self.device)
        raw = torch.empty(R, w.R, dtype=torch.float32, device=self.device)
        gate = torch.empty(R, m.heads, dtype=torch.float32, device=self.device)
        ops.proj_split(h, w.wproj, [(ops.SEG_ROWS, q), (ops.SEG_F32, raw), (ops.SEG_F32, gate)], w.col_scale, status=self.status)
        ops.latent_norm_append(raw, w.c_norm, self.cfg.norm_eps, m.rank, self.c_pools[li], pos, table, self.status)
        out = torch.empty_like(q)
        n = 0
        if chunk_of is not None:
            first, n_chunk = chunk_of
            if n_chunk >= LATENT_EXPAND_ROWS and ops.paged_attn_prefill_chunked_supported(m.heads, m.heads, D, self.dtype):
                n = n_chunk
                ctx = first + n
                ks, vs, order = self._expanded_kv(m.heads, D, -(-ctx // PAGE))
                c = ops.gather_pages(self.c_pools[li], table[0], ctx, self.status)
                ops.proj_split(c, w.wukv, [(ops.SEG_PAGES, ks), (ops.SEG_PAGES, vs)], status=self.status)
                ops.paged_attn_prefill_chunked(q[:n], ks, vs, order, first, w.scale, self.status, 0, gate[:n], out[:n])
        if n < R:
            self._latent_rows(q[n:], gate[n:], li, m, w, new_len[n:], table[n:],
                              plan if plan is not None and n else self._attn_for(R - n), out[n:])
        return self._linear(out.view(R, m.heads * D), w.wo)

    def _forward(self, tokens, pos, table, chunk_of: tuple[int, int] | None = None, plan=None, slots=None) -> torch.Tensor:
        """One pass: row i is token `tokens[i]` at position `pos[i]` of the sequence with pages `table[i]` (and state slot
        `slots[i]`).  With `chunk_of` = (first position, n) the first n rows are consecutive tokens of one sequence; the others
        are decode rows of other sequences, with attention `plan` (see _attn_for).  Returns the final normed rows."""
        c = self.cfg
        if c.gated:
            rows = gated.Rows(pos, table, slots, *(chunk_of or (0, 0)))
            x, pending = ops.embed_sinusoid(tokens, pos, self.embed, self.sinusoid, c.width, self.status), None
            for li, (spec, w) in enumerate(zip(c.layer_list, self.layers)):
                h = self._add_norm(x, pending, w.norm1)
                mixer = self._parallel if isinstance(spec.mixer, gated.ParallelSpec) else self._lightning
                pending = mixer(h, li, spec.mixer, w, rows)
                if spec.mlp is not None:
                    pending = self._experts(self._add_norm(x, pending, w.norm2), spec.mlp, w)
            return self._add_norm(x, pending, self.final_norm)
        new_len = pos + 1
        x = ops.embed_sinusoid(tokens, pos, self.embed, self.sinusoid, c.width, self.status)
        delta = None
        for li, (spec, w) in enumerate(zip(c.layer_list, self.layers)):
            h = self._mixer_input(x, delta, w, self.hist[li], pos, table, chunk_of)
            mixer = self._attention if isinstance(spec.mixer, AttentionSpec) else self._latent
            delta = mixer(h, li, spec.mixer, w, pos, new_len, table, chunk_of, plan)
            if spec.mlp is not None:
                h = ops.group_rmsnorm(x, delta, w.norm2, c.norm_eps, c.width, c.norm_groups, status=self.status)
                a = ops.glu_proj(h, w.wgu, spec.mlp.limit, GLU_ALPHA, self.status)
                delta = self._linear(a, w.wdown)
        return ops.group_rmsnorm(x, delta, self.final_norm, c.norm_eps, c.width, c.norm_groups, status=self.status)

    # ----------------------------------------------------------------- hooks
    def _decode_hidden(self, B: int) -> torch.Tensor:
        if self.cfg.gated:
            return self._forward(self.tokens[:B], self.ctx_lens[:B], self.block_table[:B], slots=self.state_slots[:B])
        return self._forward(self.tokens[:B], self.ctx_lens[:B], self.block_table[:B], None, self._attn_for(B))

    def _begin_prompt(self, chunk: int) -> int:
        return chunk

    def _prompt_hidden(self, token_ids: list[int], row: torch.Tensor, lo: int, chunk: int, slot: int) -> torch.Tensor:
        n = len(token_ids)
        tokens = torch.tensor(token_ids, device=self.device)
        pos = torch.arange(lo, lo + n, device=self.device, dtype=torch.int32)
        return self._forward(tokens, pos, row.unsqueeze(0).expand(n, -1).contiguous(), (lo, n), slots=self._slots_of(slot, n))

    def _slots_of(self, slot: int, n: int):
        return torch.full((n,), slot, dtype=torch.int32, device=self.device) if self.num_slots else None

    def _mixed_hidden(self, tokens, pos, table, first_pos: int, n: int, B: int, slot: int) -> torch.Tensor:
        if self.cfg.gated:
            return self._forward(tokens, pos, table, (first_pos, n), slots=torch.cat([self._slots_of(slot, n), self.state_slots[:B]]))
        return self._forward(tokens, pos, table, (first_pos, n), self._attn_for(B))

    def _pick(self, h, out=None) -> torch.Tensor:
        if self.dtype == torch.bfloat16:
            return ops.lm_head_argmax(h, self.lm_head, self.argmax_ws, out=out, status=self.status)
        return ops.argmax_rows(ops.gemm_f32(h, self.lm_head), out)

    def _logits(self, h) -> torch.Tensor:
        if self.dtype == torch.bfloat16:
            return ops.dense_gemm_f32_out(h, self.lm_head, self.status)
        return ops.gemm_f32(h, self.lm_head)

    def check_status(self, where: str = "layered engine") -> None:
        """Synchronise and raise if a kernel has recorded a device-side finding."""
        ops.read_status(self.status, where)
        for rows, (_, ws) in self._row_ws.items():
            ops.read_status(ws, f"{where}: attention ({rows} rows)")
        for ws in getattr(self, "_moe_ws", ()):
            ops.read_status(ws, f"{where}: experts")

    # ------------------------------------------------------------ accounting
    def kv_bytes_per_token(self) -> int:
        """Cache bytes a token leaves behind, all layers (K/V or latents, and its share of the convolution history)."""
        size = torch.empty(0, dtype=self.dtype).element_size()
        total = 0
        for spec, w in zip(self.cfg.layer_list, self.layers):
            if self.cfg.gated:
                a = getattr(spec.mixer, "left", None)
                total += a.kv_heads * (w.Dk + w.Dv) if a else 0
                continue
            total += 2 * spec.mixer.kv_heads * w.D if isinstance(spec.mixer, AttentionSpec) else w.R
            total += min(self.cfg.taps, PAGE) * self.W // PAGE if self.cfg.taps > 1 else 0
        return total * size

    def state_bytes_per_sequence(self) -> int:
        """Bytes a sequence holds whatever its length (recurrent states, both halves, and convolution inputs)."""
        if not self.cfg.gated:
            return 0
        per = [t[0] for t in self.states + self.rings if t is not None]
        return sum(t.numel() * t.element_size() for t in per)
