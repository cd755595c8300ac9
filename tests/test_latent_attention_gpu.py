"""Latent attention one step at a time against tests/zigipel_oracle.py: the page rows, the products with a matrix per head, the expansion for
portions, the absorbed form of single tokens, and keys that stand out at window and page edges."""
import math

import pytest
import torch

from tests import zigipel_oracle as ZG
from tests.test_stack_kernels_gpu import batch, rand, rel

pytestmark = pytest.mark.gpu
BF = torch.bfloat16


def spec(H=3, dim=16, rot=8, vdim=24, rank=40, window=23, scale=0.3):
    from tunix_b200.models.mixers import LatentAttentionSpec, YarnScaling
    return LatentAttentionSpec(heads=H, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, scale=scale, window=window, rot_dims=rot, rot_base=100.0,
                               rot_scaling=YarnScaling(4.0, 50.0, 3.0, 0.5))


def rot_dict(sp):
    s = sp.rot_scaling
    return {"dims": sp.rot_dims, "base": sp.rot_base, "scaling": {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}}


SIZES = [(3, 16, 8, 24, 40), (3, 7, 6, 5, 13), (20, 96, 64, 128, 136), (2, 48, 16, 40, 264), (17, 104, 24, 64, 512), (1, 128, 128, 64, 72), (3, 64, 16, 56, 88),
         (2, 128, 64, 128, 320), (40, 32, 16, 48, 64)]


@pytest.mark.parametrize("dtype", [torch.float32, BF])
@pytest.mark.parametrize("sizes", SIZES)
def test_latents_and_rotated_parts_go_to_their_pages(sizes, dtype):
    from tunix_b200.models.stack_exec import rope_table
    from tunix_b200.ops import stack_kernels as SK
    sp = spec(*sizes)
    H, qd, R, W = sp.heads, sp.dim + sp.rot_dim, sp.kv_rank, sp.stored(dtype)[0]
    rb = batch([(1, 62, 4), (0, 0, 3), (2, 5, 1), (3, 700, 1)])
    rb.pos0[2] = -1
    n, eps = 9, 1e-2
    proj, w = rand(n, H * qd + R + sp.rot_dim, dtype=dtype, std=0.3), rand(R, dtype=dtype, seed=1)
    before = proj.clone()
    table = torch.full((4, 12), -1, dtype=torch.int32)
    table[0, 0], table[1, 0], table[1, 1], table[3, 10] = 4, 2, 0, 1
    pool = torch.full((5, 64, W), 3.0, device="cuda", dtype=dtype)
    cos, sin = rope_table(768, sp.rot_dims, sp.rot_base, "cuda", sp.rot_scaling)
    SK.latent_write(proj, H * qd, w, cos, sin, sp.rot_dims, eps, rb, table.cuda(), 64, H, sp.dim, sp.rot_dim, R, pool)
    pos, p = torch.tensor([62, 63, 64, 65, 0, 1, 2, 5, 700]), before.double().cpu()
    t, live = 2e-6 if dtype == torch.float32 else 5e-3, [0, 1, 2, 3, 4, 5, 6, 8]
    q = p[:, :H * qd].view(n, H, qd)
    turned = ZG.rotate(q[..., sp.dim:], pos, rot_dict(sp))
    got = proj[:, :H * qd].view(n, H, qd)
    assert torch.equal(got[..., :sp.dim], before[:, :H * qd].view(n, H, qd)[..., :sp.dim])
    assert rel(got[live][..., sp.dim:], turned[live]) < t and torch.equal(proj[7], before[7])
    c = ZG.rms(p[:, H * qd:H * qd + R], eps) * w.double().cpu()
    kr = ZG.rotate(p[:, H * qd + R:], pos, rot_dict(sp))
    for row, (pg, o) in zip(live, [(2, 62), (2, 63), (0, 0), (0, 1), (4, 0), (4, 1), (4, 2), (1, 60)]):
        assert rel(pool[pg, o, :R], c[row]) < t and rel(pool[pg, o, R:sp.width], kr[row]) < t
        assert pool[pg, o, sp.width:].eq(3).all()                       # nobody writes what lies behind a row
    assert (pool != 3).any(-1).sum() == 8


@pytest.mark.parametrize("transposed", [False, True])
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 16, 40), (64, 2, 128, 512), (70, 5, 104, 136), (130, 1, 512, 128), (9, 4, 264, 24)])
def test_products_with_a_matrix_per_head(T, H, K, N, transposed):
    """Rows by name, columns of wider rows, what lies behind a head copied along."""
    from tunix_b200.ops import stack_kernels as SK
    tail, pad = (0, 0) if transposed else (16, 40)
    x = rand(T + 3, H * (K + 16) + 8, dtype=BF)[:, :H * (K + 16)].unflatten(1, (H, K + 16))
    w = rand(H, *((N, K) if transposed else (K, N)), dtype=BF, std=K ** -0.5, seed=3)
    want = torch.einsum("thk,hnk->thn" if transposed else "thk,hkn->thn", x[..., :K].double(), w.double())
    perm = torch.randperm(T + 3, generator=torch.Generator().manual_seed(0)).int().cuda()[:T]
    out = torch.full((T + 3, H * (N + pad) + 8), 9.0, dtype=BF, device="cuda")
    view = out[:, 8:].unflatten(1, (H, N + pad))
    SK.head_product(x, w, view, transposed=transposed, rows=T, tail=tail)
    assert rel(view[:T, :, :N], want[:T]) < 5e-3 and out[:, :8].eq(9).all() and out[T:].eq(9).all()
    if tail:
        assert torch.equal(view[:T, :, N:N + tail], x[:T, :, K:K + tail]) and view[:T, :, N + tail:].eq(0).all()
    out.fill_(9.0)
    SK.head_product(x, w, view, transposed=transposed, rows=T, tail=tail, x_rows=perm, out_rows=perm)
    live = perm.long()
    assert rel(view[live][..., :N], want[live]) < 5e-3
    rest = torch.ones(T + 3, dtype=torch.bool, device="cuda")
    rest[live] = False
    assert out[rest].eq(9).all()
    if not transposed:
        SK.head_product(x, w, view, rows=T, tail=tail, x_rows=perm)
        assert rel(view[:T, :, :N], want[live]) < 5e-3 and torch.equal(view[:T, :, N:N + tail], x[live][..., K:K + tail])


class Latents:
    """Cached rows of unequal sequences over shuffled pages; what no sequence owns holds large finite values."""

    def __init__(self, lens, sp, seed=0, page=64):
        g = torch.Generator("cuda").manual_seed(seed)
        self.sp, self.page, self.W = sp, page, sp.stored(BF)[0]
        pages = [-(-n // page) for n in lens]
        perm = torch.randperm(sum(pages) + 2, generator=torch.Generator().manual_seed(seed)).tolist()
        self.pool = torch.full((sum(pages) + 2, page, self.W), 50.0, device="cuda", dtype=BF)
        self.pool[..., sp.width:] = 0
        self.table = torch.full((len(lens) + 1, max(pages) + 2), -1, dtype=torch.int32)
        self.rows = []
        for s, n in enumerate(lens):
            own = [perm.pop() for _ in range(pages[s])]
            self.table[s, :len(own)] = torch.tensor(own)
            r = torch.randn(n, sp.width, device="cuda", generator=g).to(BF)
            self.rows.append(r)
            for j in range(n):
                self.pool[own[j // page], j % page, :sp.width] = r[j]
        self.table = self.table.cuda()

    def dense(self, q, s, i0, uk, uv, sink):
        """The oracle's attention of queries q [T, H, dim + rot] at positions i0 .. of sequence s -> [T, H, vdim]."""
        sp = self.sp
        q, uk, uv, sink = (t.double().cpu() for t in (q, uk, uv, sink))
        P = i0 + q.shape[0]
        r = self.rows[s][:P].double().cpu()
        c, kr = r[:, :sp.kv_rank], r[:, sp.kv_rank:]
        k, v = torch.einsum("tr,hdr->thd", c, uk), torch.einsum("tr,hvr->thv", c, uv)
        pad = torch.zeros(P, *q.shape[1:], dtype=torch.float64)
        pad[i0:] = q
        m = {"heads": sp.heads, "scale": sp.scale, "mask": {"size": sp.window or 10 ** 9}}
        return ZG.latent_attend(pad[..., :sp.dim], pad[..., sp.dim:], k, kr, v, m, sink)[i0:]


def weights(sp):
    uk = rand(sp.heads, sp.dim, sp.kv_rank, dtype=BF, std=sp.kv_rank ** -0.5, seed=21)
    uv = rand(sp.heads, sp.vdim, sp.kv_rank, dtype=BF, std=sp.kv_rank ** -0.5, seed=22)
    return uk, uv, rand(sp.heads, std=1.5, seed=23)


def absorbed(c, q, uk, uv, sink, slots, lens, split=0):
    from tunix_b200.ops import stack_kernels as SK
    sp, n = c.sp, q.shape[0]
    q1 = SK.head_product(q, uk, torch.empty(n, sp.heads, c.W, dtype=BF, device="cuda"), tail=sp.rot_dim)
    a = SK.latent_decode(q1, c.pool, c.table, c.page, slots, lens, rank=sp.kv_rank, scale=sp.scale, window=sp.window, sinks=sink,
                         max_ctx=c.table.shape[1] * c.page, split_tokens=split)
    return SK.head_product(a, uv, torch.empty(n, sp.heads, sp.vdim, dtype=BF, device="cuda"), transposed=True)


def expanded(c, q, parts, uk, uv, sink):
    """What the model does for portions: gather, expand, flash attention."""
    from tunix_b200.models.mixers import LatentAttention
    from tunix_b200.ops import kernels as K
    from tunix_b200.ops import stack_kernels as SK
    sp = c.sp
    m = LatentAttention(sp, 8, 1e-5, BF, "cuda")
    m.uk_proj.weight.data.copy_(uk.reshape(m.uk_proj.weight.shape))
    m.uv_proj.weight.data.copy_(uv.reshape(m.uv_proj.weight.shape))
    wide, wide_v = sp.tile_heads()
    rb = batch(parts)
    plan = rb.latent_plan(sp.window)
    assert plan.blocks is not None
    rows, w = SK.latent_gather(c.pool, *plan.blocks, c.table, c.page), m.expansion(c.W)
    kv, keys = K.gemm(rows[:, :w.shape[1]], w), sp.heads * (sp.dim if sp.split_keys else wide)
    qd = sp.dim + sp.rot_dim
    row = torch.cat([q.reshape(q.shape[0], -1), torch.full((q.shape[0], wide + 8), 2.0, dtype=BF, device="cuda")], 1)
    out = K.attn_fwd_paged(row.as_strided((q.shape[0], sp.heads, wide), (row.stride(0), qd, 1)), kv[:, :keys], kv[:, keys:], rb,
                           plan.table, 64, num_heads=sp.heads, num_kv_heads=sp.heads, head_dim=wide, scale=sp.scale, window=sp.window, sinks=sink,
                           value_dim=sp.vdim, tiles=plan.tiles, slots=plan.entries, shared_keys=(rows, sp.kv_rank) if sp.split_keys else None)
    return out.view(q.shape[0], sp.heads, sp.vdim), plan


TILED = [s for s in SIZES if all(x % 8 == 0 for x in s[1:])]
WINDOWS = [20, 64, 65, 63, 200, 0, 1, 129]


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("sizes", TILED)
def test_absorbed_single_tokens(sizes, window):
    """Positions around page and window edges, every split of the context, an idle slot."""
    sp = spec(*sizes, window=window, scale=0.2)
    assert sp.tiled(BF)
    lens = [1, 20, 21, 63, 64, 65, 66, 129, 140, 200, 201, 300]
    c = Latents(lens, sp, seed=1)
    uk, uv, sink = weights(sp)
    n = len(lens) + 1
    q = rand(n, sp.heads, sp.dim + sp.rot_dim, dtype=BF, std=0.6)
    slots, seen = torch.arange(n, dtype=torch.int32, device="cuda"), torch.tensor(lens + [0], dtype=torch.int32, device="cuda")
    want = torch.cat([c.dense(q[s:s + 1], s, m - 1, uk, uv, sink) for s, m in enumerate(lens)])
    for split in (0, 64, 128, 512):
        out = absorbed(c, q, uk, uv, sink, slots, seen, split)
        assert rel(out[:-1], want) < 1.5e-2, split
        worst = (out[:-1].double().cpu() - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1)
        assert worst.max() < 3e-2 and out[-1].abs().max() == 0


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("sizes", TILED)
def test_expanded_portions(sizes, window):
    """Portions of unequal requests behind prefixes that fill windows, from the first token and across pages; tokens of short
    entries are left to the other form."""
    sp = spec(*sizes, window=window, scale=0.2)
    lens = [300, 64, 130, 7, 200]
    c = Latents(lens, sp, seed=2)
    uk, uv, sink = weights(sp)
    parts = [(0, 120, 180), (1, 0, 64), (2, 128, 2), (3, 0, 7), (4, 69, 131), (2, 100, 28)]
    n = sum(p[2] for p in parts)
    q = rand(n, sp.heads, sp.dim + sp.rot_dim, dtype=BF, std=0.6)
    out, plan = expanded(c, q, parts, uk, uv, sink)
    left, at = set(plan.rows.tolist()), 0
    for s, p, m in parts:
        if at in left:
            assert set(range(at, at + m)) <= left
        else:
            assert rel(out[at:at + m], c.dense(q[at:at + m], s, p, uk, uv, sink)) < 1.5e-2, s
        at += m
    rows = plan.rows.long()
    got = absorbed(c, q[rows].contiguous(), uk, uv, sink, plan.slots, plan.lens)
    want = torch.cat([c.dense(q[at:at + m], s, p, uk, uv, sink) for (s, p, m), at in
                      zip(parts, [0, 180, 244, 246, 253, 384]) if at in left])
    assert rel(got, want) < 1.5e-2


@pytest.mark.parametrize("window", [20, 64, 70, 129, 128])
@pytest.mark.parametrize("form", ["absorbed", "expanded"])
@pytest.mark.parametrize("sizes", [(3, 16, 16, 24, 64), (20, 96, 64, 128, 136), (4, 128, 64, 104, 200)])
def test_one_key_at_a_window_edge(sizes, form, window):
    """The rotated part singles out one key: seen, the output is its value; just outside, it is something else."""
    sp = spec(*sizes, window=window, scale=0.5)
    c = Latents([330], sp, seed=3)
    uk, uv, _ = weights(sp)
    sink = torch.zeros(sp.heads, device="cuda")
    R, r = sp.kv_rank, c.rows[0]
    own = c.table[0].tolist()
    kr = r[:, R:].float()
    r[:, R:] = (kr / kr.norm(dim=-1, keepdim=True)).to(BF)
    for j in range(330):
        c.pool[own[j // 64], j % 64, R:sp.width] = r[j, R:]
    pairs = sorted({(i, j) for i in (63, 64, 127, 128, 191, 200, 255, 256, 320, 329)
                    for j in (i, i - 1, i - window + 1, i - window, 0, 63, 64, 127, 128) if 0 <= j <= i})
    q = torch.zeros(len(pairs), sp.heads, sp.dim + sp.rot_dim, dtype=BF, device="cuda")
    for t, (i, j) in enumerate(pairs):
        q[t, :, sp.dim:] = 240 * r[j, R:]
    if form == "absorbed":
        got = absorbed(c, q, uk, uv, sink, torch.zeros(len(pairs), dtype=torch.int32, device="cuda"),
                       torch.tensor([i + 1 for i, _ in pairs], dtype=torch.int32, device="cuda"))
    else:                                               # the last of 20 rows asks, the others ask for themselves
        rows = []
        for t, (i, j) in enumerate(pairs):
            lo = max(0, i - 19)
            qq = torch.zeros(i + 1 - lo, sp.heads, sp.dim + sp.rot_dim, dtype=BF, device="cuda")
            qq[:, :, sp.dim:] = 240 * r[lo:i + 1, None, R:]
            qq[-1] = q[t]
            rows.append(expanded(c, qq, [(0, lo, i + 1 - lo)], uk, uv, sink)[0][-1:])
        got = torch.cat(rows)
    vals = torch.einsum("tr,hvr->thv", r[:, :R].double(), uv.double()).cpu()
    for (i, j), o in zip(pairs, got):
        err = ((o.double().cpu() - vals[j]).norm() / vals[j].norm()).item()
        assert err < 0.05 if ZG.visible(i, j, {"size": window}) else err > 0.3, (i, j, err)


@pytest.mark.parametrize("score", [-60.0, -8.0, 0.0, 12.0, 60.0])
def test_sinks_of_the_absorbed_form(score):
    """All keys score the same: every head's sink takes its exact share, whatever the split."""
    window, n = 150, 320
    sp = spec(20, 16, 16, 24, 64, window=window, scale=1.0)
    c = Latents([n], sp, seed=4)
    c.pool[..., sp.kv_rank] = 1.0
    uk, uv, _ = weights(sp)
    sink = torch.linspace(-70.0, 70.0, sp.heads, device="cuda")
    q = torch.zeros(1, sp.heads, sp.dim + sp.rot_dim, dtype=BF, device="cuda")
    q[..., sp.dim] = score
    v = torch.einsum("tr,hvr->thv", c.rows[0][n - window:, :sp.kv_rank].double(), uv.double()).sum(0).cpu()
    want = torch.stack([v[h] / (math.exp(sink[h].item() - score) + window) for h in range(sp.heads)])
    for split in (64, 128, 512):
        out = absorbed(c, q, uk, uv, sink, torch.zeros(1, dtype=torch.int32, device="cuda"), torch.tensor([n], dtype=torch.int32, device="cuda"),
                       split)[0].double().cpu()
        for h in range(sp.heads):
            assert torch.allclose(out[h], want[h], rtol=2e-2, atol=2e-2 * want[h].abs().max().item() + 1e-30), h


def test_pages_of_several_blocks():
    """Pages of 128 tokens: tiles and expanded blocks are halves of pages."""
    sp = spec(4, 32, 16, 40, 72, window=100)
    c = Latents([300, 130], sp, seed=5, page=128)
    uk, uv, sink = weights(sp)
    parts = [(0, 170, 130), (1, 0, 130)]
    q = rand(260, 4, 48, dtype=BF, std=0.6)
    out, _ = expanded(c, q, parts, uk, uv, sink)
    one = absorbed(c, q[[129, 259]].contiguous(), uk, uv, sink, torch.tensor([0, 1], dtype=torch.int32, device="cuda"),
                   torch.tensor([300, 130], dtype=torch.int32, device="cuda"))
    for k, (s, p, m) in enumerate(parts):
        want = c.dense(q[130 * k:130 * k + m], s, p, uk, uv, sink)
        assert rel(out[130 * k:130 * k + m], want) < 1.5e-2 and rel(one[k], want[-1]) < 2e-2
