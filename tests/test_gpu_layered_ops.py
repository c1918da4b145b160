"""Kernels of the layer-list decoders, each mechanism alone, against plain PyTorch (B200)."""
import pytest
import torch

from conftest import rel_err
from oracle import layered_ref as ref

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
TOL = {BF: 1e-2, F32: 2e-5}


def gen(seed):
    return torch.Generator().manual_seed(seed)


def randn(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=gen(seed)) * scale).to(dtype)


def status():
    return torch.zeros(64, dtype=torch.int32, device=DEV)


def paged(L, heads, D, dtype, seed, blocks_extra=5, dim_v=None):
    """Contiguous keys/values [L, heads, D] and the same in shuffled pages: (k, v, k_pool, v_pool, table row)."""
    k, v = randn(L, heads, D, seed=seed, dtype=dtype), randn(L, heads, D, seed=seed + 1, dtype=dtype)
    pages = -(-L // 16)
    order = torch.randperm(pages + blocks_extra, generator=gen(seed + 2))[:pages]
    kp, vp = (torch.full((pages + blocks_extra, heads, 16, D), 3.0, dtype=dtype) for _ in range(2))
    for t in range(L):
        kp[order[t // 16], :, t % 16] = k[t]
        vp[order[t // 16], :, t % 16] = v[t]
    return k, v, kp, vp, order.to(torch.int32)


# ------------------------------------------------------------------- glue


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,ld", [(200, 256), (1024, 1024), (33, 64)])
def test_embed_sinusoid(ops, dtype, width, ld):
    from conftest import pkg
    emb = torch.zeros(50, ld)
    emb[:, :width] = randn(50, width, seed=1)
    emb = emb.to(dtype)
    tok = torch.tensor([0, 49, 7, 7, 3, 12])
    pos = torch.tensor([0, 1, 63, 64, 700, 2999], dtype=torch.int32)
    tables = pkg("layered").sinusoid_tables(width, ld, 3000, DEV)
    st = status()
    x = ops.embed_sinusoid(tok.to(DEV), pos.to(DEV), emb.to(DEV), tables, width, st).cpu()
    want = emb[tok].double()[:, :width] + ref.sinusoid(pos, width)
    assert float((x[:, :width].double() - want).abs().max()) < 2e-6 and not x[:, width:].any()
    ops.read_status(st, "embed")
    ops.embed_sinusoid(torch.tensor([50], device=DEV), torch.tensor([5], dtype=torch.int32, device=DEV), emb.to(DEV), tables, width, st)
    with pytest.raises(RuntimeError):
        ops.read_status(st, "a token outside the vocabulary")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width,ld,groups", [(192, 192, 3), (204, 256, 6), (1024, 1024, 4), (2048, 2048, 1), (70, 128, 10),
                                              (4096, 4096, 8), (768, 768, 2), (8192, 8192, 4), (8100, 8128, 5)])
def test_group_rmsnorm(ops, dtype, width, ld, groups):
    x, d, w = torch.zeros(9, ld), torch.zeros(9, ld), torch.zeros(ld)
    # one group per row is far larger than the others, so a statistic over the wrong columns shows
    x[:, :width] = randn(9, width, seed=2)
    for r in range(9):
        gs = width // groups
        x[r, (r % groups) * gs:(r % groups + 1) * gs] *= 40
    d[:, :width] = randn(9, width, seed=3)
    w[:width] = 1 + randn(width, seed=4) * 0.3
    d, w = d.to(dtype), w.to(dtype)
    xg = x.to(DEV)
    out = ops.group_rmsnorm(xg, d.to(DEV), w.to(DEV), 1e-3, width, groups).cpu()
    total = x.double() + d.double()
    assert float((xg.cpu().double() - total).abs().max()) < 1e-4  # the residual stays fp32
    want = ref.group_rmsnorm(total[:, :width], w.double()[:width], 1e-3, groups)
    assert rel_err(out[:, :width], want) < TOL[dtype] and not out[:, width:].any()
    alone = ops.group_rmsnorm(x.to(DEV), None, w.to(DEV), 1e-3, width, groups).cpu()
    assert rel_err(alone[:, :width], ref.group_rmsnorm(x.double()[:, :width], w.double()[:width], 1e-3, groups)) < TOL[dtype]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("taps", [1, 2, 4, 18, 35])
def test_short_conv_in_portions_and_decoded(ops, taps, dtype):
    """Any cut of a sequence - portions of every size down to one token, decode rows in between - gives the whole
    sequence's convolution, and running a step twice changes nothing."""
    ld, T = 128, 75
    h = randn(T, ld, seed=5, dtype=dtype)
    w = randn(taps, ld, seed=6, dtype=dtype)
    want = ref.short_conv(h.double(), w.double().T.contiguous())
    rows = min(taps, 16)
    table = torch.tensor([4, 1, 7, 0, 5], dtype=torch.int32, device=DEV)
    ones = torch.ones(ld, dtype=dtype, device=DEV)
    for cuts in ([T], [2, 3, 1, 16, 14, 2, 37], [15, 1, 1, 1, 14, 43], [31, 2, 42]):
        hist = torch.full((8, rows, ld), 9.0, dtype=dtype, device=DEV) if taps > 1 else None  # what a page's last user left
        st, got, at = status(), [], 0
        for n in cuts:
            for _ in range(2 if n == 1 else 1):
                if n == 1 and at:
                    # a decode row; the norm is undone by giving it a row of unit mean square times a weight
                    x = h[at:at + 1].float()
                    ms = float(x.pow(2).mean().sqrt())
                    y = ops.group_rmsnorm(x.to(DEV), None, ones * ms, 0.0, ld, 1, conv_w=w.to(DEV), hist=hist,
                                          positions=torch.tensor([at], dtype=torch.int32, device=DEV), block_table=table[None],
                                          status=st)
                else:
                    y = ops.short_conv(h[at:at + n].to(DEV), w.to(DEV), hist, table, at, status=st)
            got.append(y.cpu())
            at += n
        ops.read_status(st, "short_conv")
        assert rel_err(torch.cat(got), want) < (2e-2 if dtype == BF else 2e-5), (taps, cuts)


@pytest.mark.parametrize("ld,taps", [(64, 4), (64, 7), (4160, 3)])
def test_decode_convolution_rows_are_independent(ops, ld, taps):
    """Rows of one step at their own positions and pages; a position at a sequence's start sees zeros."""
    w, g = randn(taps, ld, seed=1).to(DEV), torch.ones(ld, device=DEV)
    hist = torch.zeros(6, taps, ld, device=DEV)
    seqs = [randn(40, ld, seed=10 + i) for i in range(3)]
    seqs = [s / s.pow(2).mean(-1, keepdim=True).sqrt() for s in seqs]
    tables = torch.tensor([[0, 1, 2], [3, 4, 5], [5, 0, 0]], dtype=torch.int32, device=DEV)[:2]
    start = [17, 0]
    ops.short_conv(seqs[0][:17].to(DEV).contiguous(), w, hist, tables[0], 0)
    for t in range(20):
        x = torch.stack([seqs[i][start[i] + t] for i in range(2)]).to(DEV)
        pos = torch.tensor([start[i] + t for i in range(2)], dtype=torch.int32, device=DEV)
        y = ops.group_rmsnorm(x, None, g, 0.0, ld, 1, conv_w=w, hist=hist, positions=pos, block_table=tables).cpu()
        for i in range(2):
            want = ref.short_conv(seqs[i][: start[i] + t + 1].double(), w.cpu().double().T.contiguous())[-1]
            assert rel_err(y[i], want) < 1e-4, (t, i)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_norm_append_and_gather(ops, dtype):
    ld, rank, n = 192, 136, 37
    raw = torch.zeros(n, ld)
    raw[:, :rank] = randn(n, rank, seed=1, scale=3.0)
    w = torch.zeros(ld)
    w[:rank] = 1 + randn(rank, seed=2) * 0.2
    w = w.to(dtype)
    pool = torch.zeros(9, 16, ld, dtype=dtype, device=DEV)
    table = torch.tensor([[6, 2, 8]], dtype=torch.int32, device=DEV)
    st = status()
    ops.latent_norm_append(raw.to(DEV), w.to(DEV), 1e-2, rank, pool, torch.arange(n, dtype=torch.int32, device=DEV),
                           table.expand(n, -1).contiguous(), st)
    got = ops.gather_pages(pool, table[0], n, st).cpu()
    want = ref.group_rmsnorm(raw.double()[:, :rank], w.double()[:rank], 1e-2, 1)
    assert rel_err(got[:, :rank], want) < TOL[dtype] and not got[:, rank:].any()
    assert torch.equal(pool[2, 3].cpu(), got[19]) and not pool[[0, 1, 3, 4, 5, 7]].any()
    ops.read_status(st, "latent append")


# --------------------------------------------------------------- projections


@pytest.mark.parametrize("rows", [1, 3, 40, 300])
def test_split_projection(ops, rows):
    """Query rows, K and V page slots and gate logits out of one product, in bf16 (one kernel) and fp32, against plain
    products; per-feature factors apply to their own features."""
    K, Hq, Hkv, D, gates = 192, 3, 2, 64, 5
    N = Hq * D + 2 * Hkv * D + gates
    pages = -(-rows // 16) + 3
    table = torch.randperm(pages, generator=gen(1)).to(torch.int32)
    pos = torch.randperm(rows, generator=gen(2)).to(torch.int32)
    scale = 1 + randn(N, seed=3)
    for dtype in (BF, F32):
        x, w = randn(rows, K, seed=4, dtype=dtype), randn(N, K, seed=5, dtype=dtype, scale=0.1)
        q = torch.zeros(rows, Hq, D, dtype=dtype, device=DEV)
        kp, vp = (torch.zeros(pages, Hkv, 16, D, dtype=dtype, device=DEV) for _ in range(2))
        gate = torch.zeros(rows, gates, device=DEV)
        st = status()
        segs = [(ops.SEG_ROWS, q), (ops.SEG_PAGES, kp), (ops.SEG_PAGES, vp), (ops.SEG_F32, gate)]
        ops.proj_split(x.to(DEV), w.to(DEV), segs, scale.to(DEV), pos.to(DEV), table[None].expand(rows, -1).contiguous().to(DEV), st)
        ops.read_status(st, "split")
        y = (x.double() @ w.double().T) * scale.double()
        a, b, c = Hq * D, (Hq + Hkv) * D, (Hq + 2 * Hkv) * D
        assert rel_err(q.view(rows, -1), y[:, :a]) < TOL[dtype]
        assert rel_err(gate, y[:, c:]) < 2e-5
        slot_k = torch.stack([kp[table[p // 16], :, p % 16].cpu() for p in pos.tolist()])
        slot_v = torch.stack([vp[table[p // 16], :, p % 16].cpu() for p in pos.tolist()])
        assert rel_err(slot_k.view(rows, -1), y[:, a:b]) < TOL[dtype] and rel_err(slot_v.view(rows, -1), y[:, b:c]) < TOL[dtype]
        if dtype == BF:  # the unfused store writes the same
            q2, gate2 = torch.zeros_like(q), torch.zeros_like(gate)
            kp2, vp2 = torch.zeros_like(kp), torch.zeros_like(vp)
            ops.split_store(ops.dense_gemm_f32_out(x.to(DEV), w.to(DEV)),
                            [(ops.SEG_ROWS, q2), (ops.SEG_PAGES, kp2), (ops.SEG_PAGES, vp2), (ops.SEG_F32, gate2)], scale.to(DEV),
                            pos.to(DEV), table[None].expand(rows, -1).contiguous().to(DEV), st, BF)
            assert torch.equal(q, q2) and torch.equal(kp, kp2) and torch.equal(vp, vp2) and torch.equal(gate, gate2)
    # without positions and table: row m into slot m of pages in order
    kp, vp = (torch.zeros(pages, Hkv, 16, D, dtype=BF, device=DEV) for _ in range(2))
    x, w = randn(rows, K, seed=4, dtype=BF), randn(2 * Hkv * D, K, seed=6, dtype=BF)
    ops.proj_split(x.to(DEV), w.to(DEV), [(ops.SEG_PAGES, kp), (ops.SEG_PAGES, vp)])
    y = x.double() @ w.double().T
    flat = kp.permute(0, 2, 1, 3).reshape(pages * 16, -1)[:rows]
    assert rel_err(flat, y[:, : Hkv * D]) < 1e-2
    # a position outside the table is reported and not written
    st = status()
    ops.proj_split(x.to(DEV), w.to(DEV), [(ops.SEG_PAGES, kp), (ops.SEG_PAGES, vp)], None,
                   torch.full((rows,), pages * 16, dtype=torch.int32, device=DEV), table[None].expand(rows, -1).contiguous().to(DEV), st)
    with pytest.raises(RuntimeError):
        ops.read_status(st, "position outside")


@pytest.mark.parametrize("rows,K,F", [(1, 64, 128), (70, 192, 384), (300, 512, 1280)])
def test_gated_unit_projection(ops, rows, K, F):
    from conftest import pkg
    gate, up = randn(F, K, seed=1, scale=K ** -0.5), randn(F, K, seed=2, scale=K ** -0.5)
    for limit in (0.3, 1.5, 50.0):
        for dtype in (BF, F32):
            x = randn(rows, K, seed=3, dtype=dtype, scale=2.0)
            w = pkg("layered").interleave_glu(gate, up).to(dtype)
            y = ops.glu_proj(x.to(DEV), w.to(DEV), limit, 1.702)
            want = ref.clamped_glu(x.double() @ gate.to(dtype).double().T, x.double() @ up.to(dtype).double().T, limit)
            assert rel_err(y, want) < TOL[dtype], (limit, dtype)
    # the unit alone, the gate far below zero included
    gu = torch.tensor([[-200.0] * 128 + [3.0] * 128, [200.0] * 128 + [-3.0] * 128], device=DEV)
    assert torch.allclose(ops.clamped_glu(gu, 2.0, 1.702)[:, 0].cpu(), ref.clamped_glu(torch.tensor([-200.0, 200.0]), torch.tensor([3.0, -3.0]), 2.0))


@pytest.mark.parametrize("groups,K,N", [(1, 64, 128), (5, 72, 136), (16, 128, 512), (3, 512, 64), (7, 40, 200)])
def test_grouped_products(ops, groups, K, N):
    for rows in (1, 33, 270):
        for dtype in (BF, F32):
            x, w = randn(rows, groups, K, seed=1, dtype=dtype), randn(groups, N, K, seed=2, dtype=dtype)
            y = ops.grouped_gemm(x.to(DEV), w.to(DEV), groups)
            assert rel_err(y, torch.einsum("mgk,gnk->mgn", x.double(), w.double())) < TOL[dtype], (rows, dtype)


def test_fp32_products_do_not_depend_on_the_batch(ops):
    x, w = randn(200, 320, seed=1), randn(77, 320, seed=2)
    y = ops.gemm_f32(x.to(DEV), w.to(DEV))
    assert rel_err(y, x.double() @ w.double().T) < 2e-6  # a reduced-precision mode would be at 1e-3
    assert torch.equal(ops.gemm_f32(x[37:40].contiguous().to(DEV), w.to(DEV)), y[37:40])
    lg = ops.dense_gemm_f32_out(x.bfloat16().to(DEV), w.bfloat16().to(DEV))
    assert rel_err(lg, x.bfloat16().double() @ w.bfloat16().double().T) < 2e-5
    z = y.clone()
    z[5, 3] = z[5, 60] = 1e6
    assert ops.argmax_rows(z).tolist() == [3 if r == 5 else int(v) for r, v in enumerate(y.argmax(-1).tolist())]


# ------------------------------------------------------------------ attention


def reference_attention(q, k, v, positions, chunk, scale, gate):
    """q [n, Hq, D] at `positions` over k, v [L, Hkv, D]."""
    n, Hq, D = q.shape
    per = Hq // k.shape[1]
    out = torch.zeros(n, Hq, v.shape[2], dtype=torch.float64)
    for i, p in enumerate(positions):
        lo = p // chunk * chunk if chunk else 0
        for h in range(Hq):
            s = (k[lo:p + 1, h // per].double() @ q[i, h].double()) * scale
            out[i, h] = torch.softmax(s, -1) @ v[lo:p + 1, h // per].double()
    return out if gate is None else out * torch.sigmoid(gate.double())[..., None]


HEADS = [(8, 2, 64), (3, 3, 128), (32, 4, 128), (6, 1, 64), (12, 6, 64), (5, 1, 128), (34, 2, 64), (4, 2, 192)]


@pytest.mark.parametrize("hq,hkv,D", HEADS)
@pytest.mark.parametrize("chunk", [0, 1, 16, 37, 128, 200])
def test_chunked_gated_attention(ops, hq, hkv, D, chunk):
    """Decode rows at chunk and page edges and whole prompts / portions, bf16 and fp32, with and without gate.  The key just
    before every chunk's start is planted so that it would take all the weight, and so is the chunk's first key for
    half of the rows: a window one token off shows as a wrong value, not as a small difference."""
    L = 300
    for dtype in (BF, F32):
        k, v, kp, vp, table = paged(L, hkv, D, dtype, seed=hq + D)
        gate = randn(L, hq, seed=9)
        q = randn(L, hq, D, seed=8, dtype=dtype)
        mark = torch.ones(D) / D ** 0.5
        if chunk > 1:
            for j in range(chunk - 1, L, chunk):  # last key of every chunk: invisible from the next chunk on
                k[j] = (mark * 60).to(dtype)
                kp[table[j // 16], :, j % 16] = k[j]
            for j in range(0, L, chunk):
                k[j] = (mark * 40).to(dtype)
                kp[table[j // 16], :, j % 16] = k[j]
            q[::2] = (mark * 4 + q[::2].float() * 0.2).to(dtype)
        scale = 0.17
        want = reference_attention(q, k, v, range(L), chunk, scale, gate)
        plain = reference_attention(q, k, v, range(L), chunk, scale, None)
        kp, vp, table = kp.to(DEV), vp.to(DEV), table.to(DEV)
        edges = sorted({p for e in range(0, L, chunk or 64) for p in (e - 1, e, e + 1, e + 15) if 0 <= p < L} | {0, 15, 16, L - 1})
        rows = torch.tensor(edges)
        qd, gd = q[rows].to(DEV), gate[rows].to(DEV)
        tab = table[None].expand(len(edges), -1).contiguous()
        ctx = (rows + 1).to(torch.int32).to(DEV)
        for split in (16, 64, 1024):
            ws = ops.paged_attn_workspace(len(edges), hq, D, table.numel(), 16, split, DEV)
            got = ops.paged_attn_decode_chunked(qd, kp, vp, tab, ctx, scale, split, ws, chunk, gd)
            assert rel_err(got, want[rows]) < TOL[dtype], (dtype, split)
            got = ops.paged_attn_decode_chunked(qd, kp, vp, tab, ctx, scale, split, ws, chunk)
            assert rel_err(got, plain[rows]) < TOL[dtype]
            ops.read_status(ws, "decode")
        if ops.paged_attn_prefill_chunked_supported(hq, hkv, D, dtype):
            st = status()
            for first, n in ((0, L), (0, 1), (1, 2), (15, 2), (36, 3), (37, 100), (127, 130), (129, 171), (255, 45)):
                got = ops.paged_attn_prefill_chunked(q[first:first + n].to(DEV), kp, vp, table, first, scale, st, chunk,
                                                     gate[first:first + n].to(DEV).contiguous())
                assert rel_err(got, want[first:first + n]) < TOL[dtype], (first, n)
            ops.read_status(st, "prefill")


@pytest.mark.parametrize("rank", [64, 128, 192, 256, 384, 512])
@pytest.mark.parametrize("heads", [1, 5, 16, 20, 40])
def test_latent_decode_attention(ops, rank, heads):
    """Every rank and head grouping; contexts at tile, page and split edges; one far latent stands out for some rows."""
    L = 700
    c, _, pool, _, table = paged(L, 1, rank, BF, seed=rank + heads)
    c, pool = c[:, 0].clone(), pool[:, 0].clone()
    lens = [1, 2, 15, 16, 17, 63, 64, 65, 127, 128, 129, 192, 250, 256, 257, 640, 641, 700]
    q = randn(len(lens), heads, rank, seed=3, dtype=BF)
    for i in range(0, len(lens), 2):
        q[i] = (c[min(3, lens[i] - 1)].float() * 0.5 + q[i].float() * 0.1).bfloat16()  # looks for an early latent
    gate = randn(len(lens), heads, seed=4)
    scale = rank ** -0.5 * 2
    want = reference_attention(q, c[:, None], c[:, None], [n - 1 for n in lens], 0, scale, gate) if heads == 1 else \
        torch.stack([torch.cat([reference_attention(q[i:i + 1, h:h + 1], c[:, None], c[:, None], [lens[i] - 1], 0, scale,
                                                    gate[i:i + 1, h:h + 1]) for h in range(heads)], 1)[0] for i in range(len(lens))])
    tab = table[None].expand(len(lens), -1).contiguous().to(DEV)
    ctx = torch.tensor(lens, dtype=torch.int32, device=DEV)
    for split in (64, 208, 1024):
        ws = ops.paged_attn_workspace(len(lens), heads, rank, table.numel(), 16, split, DEV)
        got = ops.latent_attn_decode(q.to(DEV), pool.to(DEV), tab, ctx, scale, split, ws, gate.to(DEV))
        ops.read_status(ws, "latent decode")
        assert rel_err(got, want) < 1e-2, split
    # the generic kernel (fp32, and ranks without a kernel of their own) computes the same
    one = pool[:, None].float().to(DEV)
    got = ops.paged_attn_decode_chunked(q.float().to(DEV), one, one, tab, ctx, scale, 64, ws, 0, gate.to(DEV))
    assert rel_err(got, want) < 2e-5
    empty = ops.latent_attn_decode(q[:1].to(DEV), pool.to(DEV), tab[:1], torch.zeros(1, dtype=torch.int32, device=DEV), scale, 64, ws)
    assert not empty.any()
