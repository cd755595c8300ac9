"""Attention of layer-stack models over the paged cache (distance-biased sliding windows with kept first tokens; rotary, capped
attention inside chunks), in its three kernels (general, flash attention over pages, paged decode): against a dense restatement, with queries whose scores single out one key at an edge."""
import math

import pytest
import torch

from tests import roluzen_oracle as O
from tests import tovalix_oracle as TO
from tests import zigipel_oracle as ZG
from tests import zikezen_oracle as ZO
from tests.test_stack_kernels_gpu import batch, rand, rel

pytestmark = pytest.mark.gpu


def dense(q, k, v, i0, scale, bias, size, keep):
    """q [T, H, d] at positions i0.., k / v [P, G, *] of the whole sequence, bias [H, far + 1] -> [T, H, dv] in fp64."""
    q, k, v, bias = (t.double().cpu() for t in (q, k, v, bias))
    T, H, _ = q.shape
    P, G, _ = k.shape
    far = bias.shape[1] - 1
    out = torch.zeros(T, H, v.shape[2], dtype=torch.float64)
    for t in range(T):
        i = i0 + t
        js = [j for j in range(P) if O.visible(i, j, size or 10 ** 9, keep)]
        dist = torch.tensor([min(i - j, far) for j in js])
        for h in range(H):
            g = h // (H // G)
            s = k[js, g] @ q[t, h] * scale + bias[h, dist]
            out[t, h] = torch.softmax(s, -1) @ v[js, g]
    return out


class Cache:
    """Sequences of unequal length scattered over shuffled pages; what no sequence owns holds large values."""

    def __init__(self, lens, G, dq, dv, dtype, page=64, seed=0, unit=False):
        g = torch.Generator("cuda").manual_seed(seed)
        pages = [-(-n // page) for n in lens]
        total = sum(pages) + 2
        self.k = torch.full((total, page, G * dq), 50.0, device="cuda", dtype=dtype)
        self.v = torch.full((total, page, G * dv), 50.0, device="cuda", dtype=dtype)
        perm = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
        self.table = torch.full((len(lens) + 1, max(pages) + 1), -1, dtype=torch.int32)
        self.seqs = []
        for s, n in enumerate(lens):
            own = [perm.pop() for _ in range(pages[s])]
            self.table[s, :len(own)] = torch.tensor(own)
            k = torch.randn(n, G, dq, device="cuda", generator=g)
            k = (k / k.norm(dim=-1, keepdim=True) if unit else k).to(dtype)
            v = torch.randn(n, G, dv, device="cuda", generator=g).to(dtype)
            self.seqs.append((k, v))
            for j in range(n):
                self.k[own[j // page], j % page] = k[j].reshape(-1)
                self.v[own[j // page], j % page] = v[j].reshape(-1)
        self.table = self.table.cuda()
        self.page = page


def run(kind, cache, rb, q, sp, bias, split=0, **kw):
    from tunix_b200.ops import kernels as K
    from tunix_b200.ops import stack_kernels as SK
    n = q.shape[0]
    if kind == "general":
        return SK.window_attn(q if q.stride(0) != q.shape[1] * q.shape[2] else q.reshape(n, -1), cache.k, cache.v, rb, cache.table, cache.page, sp, bias, **kw).view(n, sp.heads, sp.vdim)
    kw = dict(scale=sp.scale, softcap=sp.softcap, window=sp.window, chunk=sp.chunk, keep_first=sp.keep_first, sink=sp.sink, bias=bias,
              value_dim=sp.vdim, **kw)
    if kind == "decode":
        return K.paged_decode(q, cache.k, cache.v, cache.table, rb.slot, rb.pos0 + 1, num_kv_heads=sp.kv_heads, page_size=cache.page,
                              max_ctx=cache.table.shape[1] * cache.page, split_tokens=split, **kw).view(n, sp.heads, sp.vdim)
    return K.attn_fwd_paged(q if q.stride(0) != q.shape[1] * q.shape[2] else q.reshape(n, -1).contiguous(), cache.k, cache.v, rb, cache.table, cache.page, num_heads=sp.heads,
                            num_kv_heads=sp.kv_heads, head_dim=sp.stored(q.dtype)[0], **kw).view(n, sp.heads, sp.vdim)


def spec(H, G, dq, dv, window, keep, scale=0.2):
    from tunix_b200.models.mixers import WindowAttentionSpec
    return WindowAttentionSpec(heads=H, kv_heads=G, dim=dq, vdim=dv, scale=scale, bias_max=1, window=window, keep_first=keep)


GENERAL = [("general", torch.float32, 4, 2, 12, 20), ("general", torch.bfloat16, 3, 1, 17, 9), ("general", torch.float32, 2, 2, 64, 512)]
FLASH = [("flash", torch.bfloat16, 4, 2, 64, 64), ("flash", torch.bfloat16, 3, 1, 128, 128), ("flash", torch.bfloat16, 2, 2, 256, 256)]
DECODE = [("decode", torch.bfloat16, 6, 2, 64, 64), ("decode", torch.bfloat16, 16, 1, 128, 128), ("decode", torch.bfloat16, 3, 3, 256, 256)]
MASKS = [(20, 3), (64, 5), (65, 64), (63, 70), (200, 0), (0, 0), (1, 1), (130, 130)]


def tol(dtype):
    return 2e-6 if dtype == torch.float32 else 1.2e-2


@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", GENERAL + FLASH)
def test_portions(kind, dtype, H, G, dq, dv, window, keep):
    """Portions of unequal requests at page and tile edges, down to two tokens, with a wide bias table."""
    sp = spec(H, G, dq, dv, window, keep)
    cache = Cache([300, 64, 130, 7], G, dq, dv, dtype)
    bias = rand(H, 91, std=2.0)
    parts = [(0, 120, 180), (1, 0, 64), (2, 128, 2), (3, 0, 7)]
    rb = batch(parts)
    q = rand(sum(n for _, _, n in parts), H, dq, dtype=dtype)
    out = run(kind, cache, rb, q, sp, bias)
    at = 0
    for s, p, n in parts:
        k, v = cache.seqs[s]
        assert rel(out[at:at + n], dense(q[at:at + n], k[:p + n], v[:p + n], p, sp.scale, bias, window, keep)) < tol(dtype), s
        at += n


@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", GENERAL[:2] + DECODE)
def test_single_tokens(kind, dtype, H, G, dq, dv, window, keep):
    """Decoded tokens at positions around page edges, in every split of the context over CTAs; an idle slot gives zeros."""
    sp = spec(H, G, dq, dv, window, keep)
    lens = [1, 63, 64, 65, 129, 300, 22]
    cache = Cache(lens, G, dq, dv, dtype, seed=3)
    bias = rand(H, 91, std=2.0)
    rb = batch([(s, n - 1, 1) for s, n in enumerate(lens)] + [(len(lens), 0, 1)])
    rb.pos0[-1] = -1                                                    # idle
    q = rand(len(lens) + 1, H, dq, dtype=dtype)
    want = [dense(q[s:s + 1], k, v, lens[s] - 1, sp.scale, bias, window, keep) for s, (k, v) in enumerate(cache.seqs)]
    for split in (0, 64, 128, 512):
        out = run(kind, cache, rb, q, sp, bias, split)
        for s, w in enumerate(want):
            assert rel(out[s:s + 1], w) < tol(dtype), (s, split)
        assert out[-1].abs().max() == 0
        if kind == "general":
            break


def outstanding(cache, s, positions, targets, H, dq):
    """Queries at `positions` that score far above everything else with the key at `targets`."""
    k, _ = cache.seqs[s]
    G = k.shape[1]
    q = torch.stack([torch.stack([k[j, h // (H // G)].float() / k[j, h // (H // G)].float().norm() for h in range(H)]) for j in targets])
    return (q * 300.0).to(k.dtype)


EDGES = [(20, 3), (64, 5), (70, 64), (129, 66), (128, 1)]


@pytest.mark.parametrize("window,keep", EDGES)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv,decoded", [(*c, d) for d, cs in ((False, GENERAL[:2] + FLASH[:2]), (True, GENERAL[:2] + DECODE[:2]))
                                                          for c in cs])
def test_one_key_at_an_edge(kind, dtype, H, G, dq, dv, window, keep, decoded):
    """Every query asks for one key: just inside and just outside the window, the last kept and the first dropped token, the
    sequence's first token, page edges, itself. Seen, the output is that key's value; unseen, it must be something else."""
    P = 330
    sp = spec(H, G, dq, dv, window, keep, scale=0.3)
    cache = Cache([P], G, dq, dv, dtype, seed=5, unit=True)
    k, v = cache.seqs[0]
    bias = torch.zeros(H, 40, device="cuda")
    pairs = []
    for i in (63, 64, 127, 128, 191, 200, 255, 256, 320, 329):
        for j in {i, i - 1, i - window + 1, i - window, 0, keep - 1, keep, 63, 64, 127, 128}:
            if 0 <= j <= i:
                pairs.append((i, j))
    if decoded:
        got = torch.cat([run(kind, cache, batch([(0, i, 1)]), outstanding(cache, 0, [i], [j], H, dq), sp, bias) for i, j in pairs])
    else:                                    # one portion that reaches each position; the other rows ask for themselves
        rows = []
        for i, j in pairs:
            lo = max(0, i - 2)
            q = outstanding(cache, 0, range(lo, i + 1), [*range(lo, i), j], H, dq)
            rows.append(run(kind, cache, batch([(0, lo, i + 1 - lo)]), q, sp, bias)[-1:])
        got = torch.cat(rows)
    for (i, j), o in zip(pairs, got):
        val = torch.stack([v[j, h // (H // G)] for h in range(H)]).double().cpu()
        err = ((o.double().cpu() - val).norm() / val.norm()).item()
        if O.visible(i, j, window, keep):
            assert err < 0.05, (i, j, err)
        else:
            assert err > 0.3, (i, j, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dq,dv", [(4, 2, 16, 24), (3, 1, 10, 6), (8, 8, 64, 64)])
def test_query_key_norm_and_page_write(H, G, dq, dv, dtype):
    """The norm runs over all heads at once; keys and values land in their pages, idle rows nowhere."""
    from tunix_b200.ops import stack_kernels as SK
    NQ, NK, NV, eps = H * dq, G * dq, G * dv, 1e-2
    rb = batch([(1, 62, 4), (0, 0, 3), (2, 5, 1)])
    rb.pos0[2] = -1
    n = 8
    proj = rand(n, 2 + NQ + NK + NV, dtype=dtype, std=0.3)
    qw, kw = rand(NQ, dtype=dtype, seed=1), rand(NK, dtype=dtype, seed=2)
    table = torch.tensor([[4, -1], [2, 0], [3, 3]], dtype=torch.int32, device="cuda")
    kp, vp = torch.zeros(5, 64, NK, device="cuda", dtype=dtype), torch.zeros(5, 64, NV, device="cuda", dtype=dtype)
    q = SK.qk_norm_write(proj, 2, 2 + NQ, 2 + NQ + NK, qw, kw, eps, rb, table, 64, kp, vp, NQ)
    d = proj.double()
    t = 2e-6 if dtype == torch.float32 else 5e-3
    assert rel(q[:7], O.rms(d[:7, 2:2 + NQ], eps) * qw.double()) < t and q[7].abs().max() == 0
    kn = O.rms(d[:, 2 + NQ:2 + NQ + NK], eps) * kw.double()
    where = [(2, 62), (2, 63), (0, 0), (0, 1), (4, 0), (4, 1), (4, 2)]
    for row, (pg, o) in enumerate(where):
        assert rel(kp[pg, o], kn[row]) < t and torch.equal(vp[pg, o], proj[row, 2 + NQ + NK:])
    assert (kp.abs().sum(-1) > 0).sum() == 7 and (vp.abs().sum(-1) > 0).sum() == 7


def test_existing_decode_attention_without_bias_is_unchanged_by_the_tile_walk():
    """Windowed decode without bias or kept tokens, many splits: the walk over visible tiles equals the dense result."""
    sp = spec(8, 2, 64, 64, 100, 0, scale=1 / math.sqrt(64))
    cache = Cache([640, 100, 101, 1], 2, 64, 64, torch.bfloat16, seed=9)
    rb = batch([(s, n - 1, 1) for s, n in enumerate([640, 100, 101, 1])])
    q = rand(4, 8, 64, dtype=torch.bfloat16)
    zero = torch.zeros(8, 2, device="cuda")
    for split in (64, 128, 256):
        out = run("decode", cache, rb, q, sp, None, split)
        for s, (k, v) in enumerate(cache.seqs):
            assert rel(out[s:s + 1], dense(q[s:s + 1], k, v, k.shape[0] - 1, sp.scale, zero, 100, 0)) < 1.2e-2


# ------------------------------------------------------------------------------------------------ rotary, capped, in chunks
def rotary(H, G, dq, dv, chunk, cap=0.0, scale=0.2, rot=0):
    from tunix_b200.models.mixers import RotaryAttentionSpec
    return RotaryAttentionSpec(heads=H, kv_heads=G, dim=dq, vdim=dv, scale=scale, rot_dims=rot, rot_base=100.0, softcap=cap, chunk=chunk)


def dense_chunks(q, k, v, i0, sp):
    q, k, v = (t.double().cpu() for t in (q, k, v))
    out = torch.zeros(*q.shape[:2], v.shape[2], dtype=torch.float64)
    for t in range(q.shape[0]):
        js = [j for j in range(k.shape[0]) if TO.visible(i0 + t, j, sp.chunk or 10 ** 9)]
        for h in range(sp.heads):
            g = h // (sp.heads // sp.kv_heads)
            s = k[js, g] @ q[t, h] * sp.scale
            if sp.softcap:
                s = sp.softcap * torch.tanh(s / sp.softcap)
            out[t, h] = torch.softmax(s, -1) @ v[js, g]
    return out


CHUNKS = [(20, 3.0), (64, 0.0), (65, 8.0), (70, 50.0), (200, 1.5), (1, 4.0), (0, 2.0)]


@pytest.mark.parametrize("chunk,cap", CHUNKS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", GENERAL + FLASH)
def test_chunked_portions(kind, dtype, H, G, dq, dv, chunk, cap):
    sp = rotary(H, G, dq, dv, chunk, cap)
    cache = Cache([300, 64, 130, 7], G, dq, dv, dtype, seed=21)
    parts = [(0, 120, 180), (1, 0, 64), (2, 128, 2), (3, 0, 7), (0, 69, 131)]
    q = rand(sum(n for _, _, n in parts), H, dq, dtype=dtype, std=2.0)
    out, at = run(kind, cache, batch(parts), q, sp, None), 0
    for s, p, n in parts:
        k, v = cache.seqs[s]
        assert rel(out[at:at + n], dense_chunks(q[at:at + n], k[:p + n], v[:p + n], p, sp)) < tol(dtype), s
        at += n


@pytest.mark.parametrize("chunk,cap", CHUNKS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", GENERAL[:2] + DECODE)
def test_chunked_single_tokens(kind, dtype, H, G, dq, dv, chunk, cap):
    sp = rotary(H, G, dq, dv, chunk, cap)
    lens = [1, 20, 21, 63, 64, 65, 66, 129, 140, 141, 300]
    cache = Cache(lens, G, dq, dv, dtype, seed=22)
    rb = batch([(s, n - 1, 1) for s, n in enumerate(lens)] + [(len(lens), 0, 1)])
    rb.pos0[-1] = -1                                                    # idle
    q = rand(len(lens) + 1, H, dq, dtype=dtype, std=2.0)
    want = [dense_chunks(q[s:s + 1], k, v, lens[s] - 1, sp) for s, (k, v) in enumerate(cache.seqs)]
    for split in (0, 64, 128, 512):
        out = run(kind, cache, rb, q, sp, None, split)
        for s, w in enumerate(want):
            assert rel(out[s:s + 1], w) < tol(dtype), (s, split)
        assert out[-1].abs().max() == 0
        if kind == "general":
            break


@pytest.mark.parametrize("chunk", [20, 64, 70, 129, 200])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv,decoded", [(*c, d) for d, cs in ((False, GENERAL[:2] + FLASH[:2]), (True, GENERAL[:2] + DECODE[:2]))
                                                          for c in cs])
def test_one_key_at_a_chunk_edge(kind, dtype, H, G, dq, dv, chunk, decoded):
    """Every query asks for one key: the first of its chunk, the one before it, page edges, the sequence's first token, itself."""
    sp = rotary(H, G, dq, dv, chunk, cap=60.0, scale=0.3)
    cache = Cache([330], G, dq, dv, dtype, seed=23, unit=True)
    k, v = cache.seqs[0]
    pairs = sorted({(i, j) for i in (chunk - 1, chunk, chunk + 1, 63, 64, 128, 2 * chunk, 3 * chunk + 7, 255, 256, 329) if i < 330
                    for j in (i, i - 1, i - i % chunk, i - i % chunk - 1, 0, 63, 64, 127, 128) if 0 <= j <= i})
    if decoded:
        got = torch.cat([run(kind, cache, batch([(0, i, 1)]), outstanding(cache, 0, [i], [j], H, dq), sp, None) for i, j in pairs])
    else:
        rows = []
        for i, j in pairs:
            lo = max(0, i - 2)
            q = outstanding(cache, 0, range(lo, i + 1), [*range(lo, i), j], H, dq)
            rows.append(run(kind, cache, batch([(0, lo, i + 1 - lo)]), q, sp, None)[-1:])
        got = torch.cat(rows)
    for (i, j), o in zip(pairs, got):
        val = torch.stack([v[j, h // (H // G)] for h in range(H)]).double().cpu()
        err = ((o.double().cpu() - val).norm() / val.norm()).item()
        assert err < 0.05 if TO.visible(i, j, chunk) else err > 0.3, (i, j, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dq,dv,rot", [(4, 2, 16, 24, 16), (3, 1, 10, 6, 6), (8, 4, 64, 64, 64), (2, 2, 128, 128, 32), (5, 1, 24, 8, 0),
                                           (1, 1, 300, 20, 200), (4, 2, 256, 128, 256), (2, 1, 72, 200, 48)])
def test_rotation_norm_and_page_write(H, G, dq, dv, rot, dtype):
    """Rotation before the norm, far positions, pass-through dimensions, pages; queries alone for a layer that shares its keys."""
    from tunix_b200.models.stack_exec import rope_table
    from tunix_b200.ops import stack_kernels as SK
    NQ, NK, NV, eps = H * dq, G * dq, G * dv, 1e-2
    rb = batch([(1, 62, 4), (0, 0, 3), (2, 5, 1), (3, 700, 1)])
    rb.pos0[2] = -1
    off, n = 8, 9
    proj = rand(n, off + NQ + NK + NV, dtype=dtype, std=0.3)
    table = torch.full((4, 12), -1, dtype=torch.int32)
    table[0, 0], table[1, 0], table[1, 1], table[3, 10] = 4, 2, 0, 1
    table = table.cuda()
    kp, vp = torch.zeros(5, 64, NK, device="cuda", dtype=dtype), torch.zeros(5, 64, NV, device="cuda", dtype=dtype)
    cos, sin = rope_table(768, rot, 100.0, "cuda")
    args = (cos, sin, rot, eps, rb, table, 64)
    q = SK.rope_norm_write(proj, off, off + NQ, off + NQ + NK, *args, H, G, dq, dv, kp, vp)
    pos = torch.tensor([62, 63, 64, 65, 0, 1, 2, 5, 700])
    d = proj.double().cpu()
    turn = lambda x, heads: TO.rms(TO.rotate(x.reshape(n, heads, dq), pos, rot, 100.0), eps).reshape(n, -1)  # noqa: E731
    wq, wk = turn(d[:, off:off + NQ], H), turn(d[:, off + NQ:off + NQ + NK], G)
    t, live = 2e-6 if dtype == torch.float32 else 5e-3, [0, 1, 2, 3, 4, 5, 6, 8]
    assert rel(q[live], wq[live]) < t and q[7].abs().max() == 0
    for row, (pg, o) in zip(live, [(2, 62), (2, 63), (0, 0), (0, 1), (4, 0), (4, 1), (4, 2), (1, 60)]):
        assert rel(kp[pg, o], wk[row]) < t and torch.equal(vp[pg, o], proj[row, off + NQ + NK:])
    assert (kp.abs().sum(-1) > 0).sum() == 8 and (vp.abs().sum(-1) > 0).sum() == 8
    alone = proj[:, off:off + NQ].contiguous()
    before = kp.clone()
    assert torch.equal(SK.rope_norm_write(alone, 0, NQ, NQ, *args, H, 0, dq, dv, kp, vp), q) and torch.equal(kp, before)


# ------------------------------------------------------------------------------------------------ windows with a sink, wider stored heads
def sinking(H, G, dq, dv, window, scale=0.2, sink=0.0, rot=0, fit=True, **kw):
    from tunix_b200.models.mixers import RotaryAttentionSpec
    return RotaryAttentionSpec(heads=H, kv_heads=G, dim=dq, vdim=dv, scale=scale, rot_dims=rot, rot_base=100.0, window=window, sink=sink,
                               fit_heads=fit, **kw)


class Widened(Cache):
    """The cache of a spec whose heads may be stored wider than they are, zeros behind them."""

    def __init__(self, lens, sp, dtype, **kw):
        wk, wv = sp.stored(dtype)
        G = sp.kv_heads
        super().__init__(lens, G, wk, wv, dtype, **kw)
        for t, width, w in ((self.k, sp.dim, wk), (self.v, sp.vdim, wv)):
            t.view(*t.shape[:2], G, w)[..., width:] = 0
        seqs = []
        for k, v in self.seqs:
            k, v = k[..., :sp.dim].clone(), v[..., :sp.vdim].clone()
            if kw.get("unit"):
                k = (k / k.float().norm(dim=-1, keepdim=True)).to(dtype)
            seqs.append((k, v))
        if kw.get("unit"):                                 # cut to the heads' size and scaled again
            for s, (k, _) in enumerate(seqs):
                own = self.table[s].tolist()
                for j in range(k.shape[0]):
                    self.k[own[j // self.page], j % self.page].view(G, wk)[:, :sp.dim] = k[j]
        self.seqs = seqs


def widen(q, sp):
    return torch.nn.functional.pad(q, (0, sp.stored(q.dtype)[0] - sp.dim)).contiguous()


def dense_sink(q, k, v, i0, sp):
    """The oracle's attention of the last rows of a sequence."""
    q, k, v = (t.double().cpu() for t in (q, k, v))
    T, P = q.shape[0], k.shape[0]
    pad = torch.zeros(P, *q.shape[1:], dtype=torch.float64)
    pad[i0:i0 + T] = q
    m = {"heads": sp.heads, "kv_heads": sp.kv_heads, "vdim": sp.vdim, "scale": sp.scale, "mask": {"size": sp.window or 10 ** 9}}
    return ZO.attend(pad, k, v, m)[i0:i0 + T].view(T, sp.heads, sp.vdim)


SINK_GENERAL = [("general", torch.float32, 4, 2, 12, 20), ("general", torch.bfloat16, 3, 1, 17, 9), ("general", torch.bfloat16, 4, 2, 40, 56)]
SINK_FLASH = [("flash", torch.bfloat16, 4, 2, 64, 48), ("flash", torch.bfloat16, 3, 1, 72, 128), ("flash", torch.bfloat16, 2, 2, 256, 256),
              ("flash", torch.bfloat16, 6, 3, 40, 64)]
SINK_DECODE = [("decode", torch.bfloat16, 6, 2, 64, 48), ("decode", torch.bfloat16, 16, 1, 128, 128), ("decode", torch.bfloat16, 3, 3, 96, 200)]
WINDOWS = [20, 64, 65, 63, 200, 0, 1, 129]


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", SINK_GENERAL + SINK_FLASH)
def test_sink_in_portions(kind, dtype, H, G, dq, dv, window):
    """Weights that the sink takes a large part of, heads stored wider, the result in columns of a wider row and scaled."""
    sp = sinking(H, G, dq, dv, window)
    cache = Widened([300, 64, 130, 7], sp, dtype, seed=31)
    parts = [(0, 120, 180), (1, 0, 64), (2, 128, 2), (3, 0, 7), (0, 69, 131)]
    n = sum(p[2] for p in parts)
    q = rand(n, H, dq, dtype=dtype, std=0.5)
    rows = torch.full((n, 8 + H * dv + 8 + (-H * dv) % 8), 9.0, dtype=dtype, device="cuda")
    out, at = run(kind, cache, batch(parts), widen(q, sp), sp, None, out=rows[:, 8:8 + H * dv], out_scale=0.5), 0
    assert rows[:, :8].eq(9).all() and rows[:, 8 + H * dv:].eq(9).all()
    for s, p, m in parts:
        k, v = cache.seqs[s]
        assert rel(out[at:at + m], 0.5 * dense_sink(q[at:at + m], k[:p + m], v[:p + m], p, sp)) < tol(dtype), s
        at += m


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", SINK_GENERAL[:2] + SINK_DECODE)
def test_sink_in_single_tokens(kind, dtype, H, G, dq, dv, window):
    sp = sinking(H, G, dq, dv, window)
    lens = [1, 20, 21, 63, 64, 65, 66, 129, 140, 200, 201, 300]
    cache = Widened(lens, sp, dtype, seed=32)
    rb = batch([(s, n - 1, 1) for s, n in enumerate(lens)] + [(len(lens), 0, 1)])
    rb.pos0[-1] = -1                                                    # idle
    n = len(lens) + 1
    q = rand(n, H, dq, dtype=dtype, std=0.5)
    want = [-3.0 * dense_sink(q[s:s + 1], k, v, lens[s] - 1, sp) for s, (k, v) in enumerate(cache.seqs)]
    for split in (0, 64, 128, 512):
        rows = torch.full((n, 3 + H * dv + 2), 9.0, dtype=dtype, device="cuda")
        out = run(kind, cache, rb, widen(q, sp), sp, None, split, out=rows[:, 3:3 + H * dv], out_scale=-3.0)
        assert rows[:, :3].eq(9).all() and rows[:, 3 + H * dv:].eq(9).all()
        for s, w in enumerate(want):
            assert rel(out[s:s + 1], w) < tol(dtype), (s, split)
        assert out[-1].abs().max() == 0
        if kind == "general":
            break


@pytest.mark.parametrize("score", [-60.0, -8.0, 0.0, 12.0, 60.0])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", SINK_GENERAL[:2] + SINK_FLASH[:2] + SINK_DECODE[:2])
def test_sink_against_scores_of_every_size(kind, dtype, H, G, dq, dv, score):
    """All keys score the same: the sink takes everything, its exact share, or nothing."""
    window, n = 40, 100
    sp = sinking(H, G, dq, dv, window, scale=1.0)
    cache = Widened([n], sp, dtype, seed=33)
    wk, _ = sp.stored(dtype)
    cache.k.view(*cache.k.shape[:2], G, wk)[..., 0] = 1.0
    q = torch.zeros(1, H, dq, dtype=dtype, device="cuda")
    q[..., 0] = score
    out = run(kind, cache, batch([(0, n - 1, 1)]), widen(q, sp), sp, None)[0].double().cpu()
    v = cache.seqs[0][1].double().cpu()[n - window:]
    share = 1 / (math.exp(-score) + window)                             # e^s / (1 + window e^s)
    want = torch.stack([v[:, h // (H // G)].sum(0) * share for h in range(H)])
    if score == -60.0:
        assert out.abs().max() < 1e-20
    else:
        assert rel(out, want) < tol(dtype)


@pytest.mark.parametrize("window", [20, 64, 70, 129, 128])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv,decoded", [(*c, d) for d, cs in ((False, SINK_GENERAL + SINK_FLASH), (True, SINK_GENERAL[:2] + SINK_DECODE))
                                                          for c in cs])
def test_one_key_at_a_window_edge_beside_the_sink(kind, dtype, H, G, dq, dv, window, decoded):
    """Every query asks for one key: seen, the output is its value; just outside, it must be something else, also when nothing
    else scores above the sink."""
    sp = sinking(H, G, dq, dv, window, scale=0.3)
    cache = Widened([330], sp, dtype, seed=34, unit=True)
    k, v = cache.seqs[0]
    pairs = sorted({(i, j) for i in (63, 64, 127, 128, 191, 200, 255, 256, 320, 329)
                    for j in (i, i - 1, i - window + 1, i - window, 0, 63, 64, 127, 128) if 0 <= j <= i})
    ask = lambda ps, js: widen(outstanding(cache, 0, ps, js, H, dq), sp)  # noqa: E731
    if decoded:
        got = torch.cat([run(kind, cache, batch([(0, i, 1)]), ask([i], [j]), sp, None) for i, j in pairs])
    else:
        rows = []
        for i, j in pairs:
            lo = max(0, i - 2)
            rows.append(run(kind, cache, batch([(0, lo, i + 1 - lo)]), ask(range(lo, i + 1), [*range(lo, i), j]), sp, None)[-1:])
        got = torch.cat(rows)
    for (i, j), o in zip(pairs, got):
        val = torch.stack([v[j, h // (H // G)] for h in range(H)]).double().cpu()
        err = ((o.double().cpu() - val).norm() / val.norm()).item()
        assert err < 0.05 if ZO.visible(i, j, window) else err > 0.3, (i, j, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dq,dv,rot", [(4, 2, 16, 24, 16), (3, 1, 10, 6, 6), (8, 4, 64, 64, 64), (2, 2, 72, 128, 8), (5, 1, 24, 8, 0),
                                           (6, 2, 40, 48, 24), (4, 2, 256, 128, 128), (2, 1, 96, 200, 2), (1, 1, 300, 20, 200),
                                           (4, 2, 52, 40, 12), (3, 3, 40, 64, 10)])
def test_weighted_norm_interleaved_rotation_and_wider_pages(H, G, dq, dv, rot, dtype):
    """Norm with weights before the rotation of neighbours, scaled frequencies; what lies behind a head is zero."""
    from tunix_b200.models.stack_exec import rope_table
    from tunix_b200.ops import stack_kernels as SK
    sp = sinking(H, G, dq, dv, 0, rot=rot)
    wk, wv = sp.stored(dtype)
    NQ, NK, NV, eps = H * dq, G * dq, G * dv, 1e-2
    rb = batch([(1, 62, 4), (0, 0, 3), (2, 5, 1), (3, 700, 1)])
    rb.pos0[2] = -1
    off, n = 8, 9
    proj = rand(n, off + NQ + NK + NV, dtype=dtype, std=0.3)
    qw, kw = rand(dq, dtype=dtype, seed=1), rand(dq, dtype=dtype, seed=2)
    table = torch.full((4, 12), -1, dtype=torch.int32)
    table[0, 0], table[1, 0], table[1, 1], table[3, 10] = 4, 2, 0, 1
    kp, vp = torch.full((5, 64, G * wk), 3.0, device="cuda", dtype=dtype), torch.full((5, 64, G * wv), 3.0, device="cuda", dtype=dtype)
    scaling = {"factor": 6.0, "low": 1.0, "high": 4.0, "original": 400}
    cos, sin = rope_table(768, rot, 100.0, "cuda", tuple(scaling.values()))
    q = SK.rope_norm_write(proj, off, off + NQ, off + NQ + NK, cos, sin, rot, eps, rb, table.cuda(), 64, H, G, dq, dv, kp, vp, q_w=qw,
                           k_w=kw, interleaved=True, stored=(wk, wv))
    pos = torch.tensor([62, 63, 64, 65, 0, 1, 2, 5, 700])
    p, rt = proj.double().cpu(), {"dims": rot, "base": 100.0, "scaling": scaling}

    def turn(x, heads, w):
        x = ZO.rotate(ZO.rms(x.reshape(n, heads, dq), eps) * w.double().cpu(), pos, rt)
        return torch.nn.functional.pad(x, (0, wk - dq)).reshape(n, -1)
    wantq, wantk = turn(p[:, off:off + NQ], H, qw), turn(p[:, off + NQ:off + NQ + NK], G, kw)
    wantv = torch.nn.functional.pad(p[:, off + NQ + NK:].reshape(n, G, dv), (0, wv - dv)).reshape(n, -1)
    t, live = 2e-6 if dtype == torch.float32 else 5e-3, [0, 1, 2, 3, 4, 5, 6, 8]
    assert rel(q[live], wantq[live]) < t and q[7].abs().max() == 0
    assert q[live].view(8, H, wk)[..., dq:].abs().sum() == 0
    for row, (pg, o) in zip(live, [(2, 62), (2, 63), (0, 0), (0, 1), (4, 0), (4, 1), (4, 2), (1, 60)]):
        assert rel(kp[pg, o], wantk[row]) < t and torch.equal(vp[pg, o].double().cpu(), wantv[row])
        assert kp[pg, o].view(G, wk)[:, dq:].abs().sum() == 0
    assert (kp != 3).any(-1).sum() == 8 and (vp != 3).any(-1).sum() == 8


# ------------------------------------------------------------------------------------------------ distance, learned sinks, gates
def distant(H, G, dq, dv, window, keep, scale=0.3):
    from tunix_b200.models.mixers import DistanceAttentionSpec
    return DistanceAttentionSpec(heads=H, kv_heads=G, dim=dq, vdim=dv, scale=scale, window=window, keep_first=keep)


def learned(sp, positions, seed=0):
    """(r1, r2, sinks, distance bias) of a module with drawn numbers."""
    from tunix_b200.models.mixers import DistanceAttention
    m = DistanceAttention(sp, 8, 1e-5, torch.float32, "cuda")
    g = torch.Generator("cuda").manual_seed(seed)
    m.r1.data.uniform_(0.1, 0.9, generator=g)
    m.r2.data.uniform_(0.1, 2.0, generator=g)
    m.sink.data.normal_(0.5, 1.5, generator=g)
    return m.r1.data, m.r2.data, m.sink.data, m.bias_table(positions)


def dense_distance(q, k, v, i0, sp, r1, r2, sink, gate):
    q, k, v, r1, r2, sink, gate = (t.double().cpu() for t in (q, k, v, r1, r2, sink, gate))
    T, P = q.shape[0], k.shape[0]
    pad = torch.zeros(P, *q.shape[1:], dtype=torch.float64)
    pad[i0:i0 + T] = q
    m = {"heads": sp.heads, "kv_heads": sp.kv_heads, "scale": sp.scale, "mask": {"size": sp.window or 10 ** 9, "keep_first": sp.keep_first}}
    return ZG.attend(pad, k, v, m, r1, r2, sink)[i0:i0 + T] * torch.sigmoid(gate)[:, :, None]


def apart(q, sp, extra=16):
    """The same queries in rows that hold more behind them (and between heads nothing), read at the stored width."""
    n, H, d = q.shape
    wk = sp.stored(q.dtype)[0]
    row = torch.full((n, H * d + max(wk - d, 0) + extra), 3.0, dtype=q.dtype, device="cuda")
    row = torch.cat([q.reshape(n, -1), row[:, H * d:]], 1)
    return row.as_strided((n, H, wk), (row.stride(0), d, 1)) if d % 8 == 0 and row.shape[1] % 8 == 0 else widen(q, sp)


FAR = [("general", torch.float32, 4, 2, 12, 20), ("general", torch.bfloat16, 3, 1, 17, 9), ("general", torch.float32, 2, 1, 24, 600)]
FAR_FLASH = [("flash", torch.bfloat16, 6, 2, 40, 56), ("flash", torch.bfloat16, 3, 1, 128, 128), ("flash", torch.bfloat16, 4, 4, 72, 80)]
FAR_DECODE = [("decode", torch.bfloat16, 6, 2, 40, 56), ("decode", torch.bfloat16, 16, 1, 128, 128), ("decode", torch.bfloat16, 3, 3, 72, 80)]


@pytest.mark.parametrize("window,keep", [(20, 3), (64, 5), (65, 64), (63, 70), (200, 0), (0, 0), (1, 1), (130, 129)])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", FAR + FAR_FLASH)
def test_distance_sinks_and_gates_in_portions(kind, dtype, H, G, dq, dv, window, keep):
    sp = distant(H, G, dq, dv, window, keep)
    r1, r2, sink, bias = learned(sp, 384)
    cache = Widened([300, 64, 130, 7], sp, dtype, seed=41)
    parts = [(0, 120, 180), (1, 0, 64), (2, 128, 2), (3, 0, 7), (0, 69, 131)]
    n = sum(p[2] for p in parts)
    q, rows = rand(n, H, dq, dtype=dtype), torch.full((n, 8 + H * dv + 8 + (-H * dv) % 8), 9.0, dtype=dtype, device="cuda")
    gate = rand(n, 3 + H, dtype=dtype, std=2.0, seed=4)[:, 3:]
    out, at = run(kind, cache, batch(parts), apart(q, sp), sp, bias, out=rows[:, 8:8 + H * dv], sinks=sink, gate=gate), 0
    assert rows[:, :8].eq(9).all() and rows[:, 8 + H * dv:].eq(9).all()
    for s, p, m in parts:
        k, v = cache.seqs[s]
        want = dense_distance(q[at:at + m], k[:p + m], v[:p + m], p, sp, r1, r2, sink, gate[at:at + m])
        assert rel(out[at:at + m], want) < tol(dtype), s
        at += m


@pytest.mark.parametrize("window,keep", [(20, 3), (64, 5), (65, 64), (63, 70), (200, 0), (0, 0), (1, 1), (130, 129)])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", FAR[:2] + FAR_DECODE)
def test_distance_sinks_and_gates_in_single_tokens(kind, dtype, H, G, dq, dv, window, keep):
    sp = distant(H, G, dq, dv, window, keep)
    r1, r2, sink, bias = learned(sp, 384, seed=1)
    lens = [1, 20, 21, 63, 64, 65, 66, 129, 140, 200, 201, 300]
    cache = Widened(lens, sp, dtype, seed=42)
    rb = batch([(s, n - 1, 1) for s, n in enumerate(lens)] + [(len(lens), 0, 1)])
    rb.pos0[-1] = -1                                                    # idle
    n = len(lens) + 1
    q, gate = rand(n, H, dq, dtype=dtype), rand(n, H, dtype=dtype, std=2.0, seed=4)
    want = [dense_distance(q[s:s + 1], k, v, lens[s] - 1, sp, r1, r2, sink, gate[s:s + 1]) for s, (k, v) in enumerate(cache.seqs)]
    for split in (0, 64, 128, 512):
        out = run(kind, cache, rb, apart(q, sp), sp, bias, split, sinks=sink, gate=gate)
        for s, w in enumerate(want):
            assert rel(out[s:s + 1], w) < tol(dtype), (s, split)
        assert out[-1].abs().max() == 0
        if kind == "general":
            break


@pytest.mark.parametrize("score", [-60.0, -8.0, 0.0, 12.0, 60.0])
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv", FAR[:2] + FAR_FLASH[:2] + FAR_DECODE[:2])
def test_every_head_has_its_own_sink(kind, dtype, H, G, dq, dv, score):
    """All keys score the same: a head's sink takes its exact share of the weights, also far below and above them."""
    window, n = 40, 100
    sp = distant(H, G, dq, dv, window, 0, scale=1.0)
    cache = Widened([n], sp, dtype, seed=43)
    wk, _ = sp.stored(dtype)
    cache.k.view(*cache.k.shape[:2], G, wk)[..., 0] = 1.0
    q = torch.zeros(1, H, dq, dtype=dtype, device="cuda")
    q[..., 0] = score
    sink = torch.linspace(-70.0, 70.0, H, device="cuda") if H > 1 else torch.zeros(1, device="cuda")
    out = run(kind, cache, batch([(0, n - 1, 1)]), widen(q, sp), sp, None, sinks=sink)[0].double().cpu()
    v = cache.seqs[0][1].double().cpu()[n - window:]
    for h in range(H):
        share = 1 / (math.exp(sink[h].item() - score) + window)
        want = v[:, h // (H // G)].sum(0) * share
        assert torch.allclose(out[h], want, rtol=tol(dtype), atol=tol(dtype) * want.abs().max().item() + 1e-30), h


@pytest.mark.parametrize("window,keep", EDGES)
@pytest.mark.parametrize("kind,dtype,H,G,dq,dv,decoded", [(*c, d) for d, cs in ((False, FAR[:2] + FAR_FLASH), (True, FAR[:2] + FAR_DECODE)) for c in cs])
def test_one_key_at_an_edge_against_distance_and_sinks(kind, dtype, H, G, dq, dv, window, keep, decoded):
    """Queries that ask for one key, whose score stands above what the distance takes off: seen, the output is its value."""
    sp = distant(H, G, dq, dv, window, keep, scale=0.3)
    r1, r2, sink, bias = learned(sp, 384, seed=2)
    cache = Widened([330], sp, dtype, seed=44, unit=True)
    k, v = cache.seqs[0]
    pairs = sorted({(i, j) for i in (63, 64, 127, 128, 191, 200, 255, 256, 320, 329)
                    for j in (i, i - 1, i - window + 1, i - window, 0, keep - 1, keep, 63, 64, 127, 128) if 0 <= j <= i})
    ask = lambda ps, js: widen(outstanding(cache, 0, ps, js, H, dq), sp)  # noqa: E731
    rows = []
    for i, j in pairs:
        lo = i if decoded else max(0, i - 2)
        rows.append(run(kind, cache, batch([(0, lo, i + 1 - lo)]), ask(range(lo, i + 1), [*range(lo, i), j]), sp, bias, sinks=sink)[-1:])
    for (i, j), o in zip(pairs, torch.cat(rows)):
        val = torch.stack([v[j, h // (H // G)] for h in range(H)]).double().cpu()
        err = ((o.double().cpu() - val).norm() / val.norm()).item()
        assert err < 0.05 if ZG.visible(i, j, {"size": window, "keep_first": keep}) else err > 0.3, (i, j, err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dq,dv", [(4, 2, 16, 24), (3, 1, 10, 6), (8, 4, 64, 64), (2, 2, 72, 128), (6, 2, 40, 48), (4, 2, 52, 40), (3, 3, 24, 256)])
def test_value_norm_and_page_write(H, G, dq, dv, dtype):
    """Queries and keys as they are, value heads divided by their root mean square; with queries or without."""
    from tunix_b200.ops import stack_kernels as SK
    sp = distant(H, G, dq, dv, 0, 0)
    wk, wv = sp.stored(dtype)
    NQ, NK, NV, eps = H * dq, G * dq, G * dv, 1e-2
    rb = batch([(1, 62, 4), (0, 0, 3), (2, 5, 1)])
    rb.pos0[2] = -1
    n = 8
    proj = rand(n, 8 + NQ + NK + NV, dtype=dtype, std=0.3)
    table = torch.tensor([[4, -1], [2, 0], [3, 3]], dtype=torch.int32, device="cuda")
    t = 2e-6 if dtype == torch.float32 else 5e-3
    p = proj.double().cpu()
    wide = lambda x, heads, w: torch.nn.functional.pad(x.reshape(n, heads, -1), (0, w - x.shape[1] // heads)).reshape(n, -1)  # noqa: E731
    wantk = wide(p[:, 8 + NQ:8 + NQ + NK], G, wk)
    wantv = wide(ZG.rms(p[:, 8 + NQ + NK:].reshape(n, G, dv), eps).reshape(n, -1), G, wv)
    for heads in (H, 0):
        kp, vp = torch.full((5, 64, G * wk), 3.0, device="cuda", dtype=dtype), torch.full((5, 64, G * wv), 3.0, device="cuda", dtype=dtype)
        q = SK.rope_norm_write(proj, 8, 8 + NQ, 8 + NQ + NK, None, None, 0, eps, rb, table, 64, heads, G, dq, dv, kp, vp, stored=(wk, wv),
                               norm_qk=False, norm_v=True)
        if heads:
            assert torch.equal(q[:7].double().cpu(), wide(p[:, 8:8 + NQ], H, wk)[:7]) and q[7].abs().max() == 0
        for row, (pg, o) in enumerate([(2, 62), (2, 63), (0, 0), (0, 1), (4, 0), (4, 1), (4, 2)]):
            assert torch.equal(kp[pg, o].double().cpu(), wantk[row]) and rel(vp[pg, o], wantv[row]) < t
        assert (kp != 3).any(-1).sum() == 7 and (vp != 3).any(-1).sum() == 7
