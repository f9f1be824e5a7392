"""The mechanisms of the Folivik layers alone, on the device, against float64 statements of the same: windowed attention with a penalty
on distance and factors on the query heads, attention over latents in both of its forms with the append in front of it, the Mamba-2 state
space, and the mixture of experts."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from oracle import folivik as oracle
from tests.test_vozozen_mechanisms import LL, SHAPES, TOL, Pool, i32, stream

pytestmark = pytest.mark.gpu
LL = LL | {torch.float16: llaisys.DataType.F16}
BOTH = [torch.float32, torch.bfloat16]


def sync():
    llaisys.RuntimeAPI(llaisys.DeviceType.NVIDIA).stream_synchronize(stream())


# ---- attention with a penalty on distance -----------------------------------------------------------------------------------


class FadePool(Pool):
    def fade(self, q, q_lens, kv_lens, nh, scale, window, a, b, decode):
        n, rows = len(q_lens), sum(q_lens)
        width = nh * self.dv + 24
        out = torch.full((rows, width), 7.0, dtype=self.dtype, device="cuda")
        starts = i32([0, *np.cumsum(q_lens).tolist()])
        self.cache.fade_dev(0, out, q.cuda().contiguous(), i32(self.seqs[:n]), None if decode else starts, i32(kv_lens), n_seqs=n,
                            total_q=rows, max_q_len=max(q_lens), max_kv_len=max(kv_lens), nh=nh, scale=scale, stream=stream(), window=window,
                            fade_a=a.float().cuda(), fade_b=b.float().cuda(), row_stride=width)
        self.cache.check()
        assert torch.all(out[:, nh * self.dv:] == 7.0), "columns behind the heads were written"
        return out[:, :nh * self.dv].reshape(rows, nh, self.dv).cpu()

    def expect_fade(self, q, q_lens, kv_lens, scale, window, a, b):
        outs = []
        for i, (n, kv) in enumerate(zip(q_lens, kv_lens)):
            part = q[sum(q_lens[:i]):sum(q_lens[:i + 1])].double()
            outs.append(oracle.softmax_attention(part, self.k[i][:kv].double(), self.v[i][:kv].double(), scale, first=kv - n, window=window or None,
                                                 bias=(a.double(), b.double())))
        return torch.cat(outs)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", SHAPES)
@pytest.mark.parametrize("window", [1, 17, 64, 100000])
def test_fading_attention_decode_and_portions(cuda_device, dtype, nkvh, nh, d, dv, window):
    lens = [1, 16, 17, 130, 64, 65]
    pool = FadePool(dtype, nkvh, d, dv, lens, seed=window)
    pool.append([0] * len(lens), lens)
    g = torch.Generator().manual_seed(3)
    scale = 1.3 * d ** -0.5
    a, b = torch.randn(nh, generator=g).float(), torch.rand(nh, generator=g).float() * 3
    for q_lens in ([1] * len(lens), [min(n, 3 + 40 * (i % 3)) for i, n in enumerate(lens)]):
        q = torch.randn(sum(q_lens), nh, d, generator=g).to(dtype)
        want = pool.expect_fade(q, q_lens, lens, scale, window, a, b)
        for decode in ([True, False] if max(q_lens) == 1 else [False]):
            got = pool.fade(q, q_lens, lens, nh, scale, window, a, b, decode)
            assert (got.double() - want).abs().max().item() <= TOL[dtype] * max(1.0, want.abs().max().item()), (q_lens, decode)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", [SHAPES[1], SHAPES[3], SHAPES[4]])
@pytest.mark.parametrize("window", [2, 16, 48, 300])
def test_the_edge_of_a_window_and_how_far_the_penalty_reaches(cuda_device, dtype, nkvh, nh, d, dv, window):
    """One key stands out so far that it wins every softmax until the window has passed it: queries around that edge, in a prompt and
    decoded alone. Then the penalty is made to outweigh it at a certain distance, inside the window."""
    for place in (0, 15, 33):
        n = place + window + 40
        pool = FadePool(dtype, nkvh, d, dv, [n], seed=place)
        pool.k[0] *= 0.05
        direction = torch.ones(d) / d ** 0.5
        pool.k[0][place] = (direction * 30).to(dtype)
        pool.append([0], [n])
        q = (direction.expand(n, nh, d) * 2.0).to(dtype).contiguous()
        value = pool.v[0][place].double().repeat_interleave(nh // nkvh, 0)
        for a, b in ((0.01, 0.5), (25.0, 0.3)):  # 25 ln(1 + 0.3 distance) passes the key's 60 at a distance of 34
            fa, fb = torch.full((nh,), a), torch.full((nh,), b)
            got = pool.fade(q, [n], [n], nh, 1.0, window, fa, fb, False)
            want = pool.expect_fade(q, [n], [n], 1.0, window, fa, fb)
            assert (got.double() - want).abs().max().item() <= TOL[dtype] * 4
            for at in (place + window - 1, place + window, min(place + 60, n - 1)):
                one = pool.fade(q[:1], [1], [at + 1], nh, 1.0, window, fa, fb, True)
                assert (one[0].double() - want[at]).abs().max().item() <= TOL[dtype] * 4
                seen = at < place + window and (a < 1 or at - place < 20)
                lost = at >= place + window or (a > 1 and at - place > 50)
                distance = (got[at].double() - value).abs().max().item()
                assert not seen or distance <= 0.02 * max(1.0, value.abs().max().item()), (place, at)
                assert not lost or distance > 0.1, (place, at)


def test_fading_on_the_fast_kernels_over_long_sequences(cuda_device):
    lens, nh = [3000, 1700, 500], 8
    for window in (700, 0):
        pool = FadePool(torch.bfloat16, 2, 128, 128, lens)
        pool.append([0, 0, 0], lens)
        g = torch.Generator().manual_seed(1)
        a, b = torch.rand(nh, generator=g) * 2, torch.rand(nh, generator=g)
        q_lens = [200, 133, 140]
        q = torch.randn(sum(q_lens), nh, 128, generator=g).to(torch.bfloat16)
        got = pool.fade(q, q_lens, lens, nh, 0.09, window, a, b, False)
        assert pool.cache.last_kernel() == llaisys.Kernel.PREFILL_TC
        assert (got.double() - pool.expect_fade(q, q_lens, lens, 0.09, window, a, b)).abs().max().item() <= 1.2e-2
        one = pool.fade(q[:3], [1, 1, 1], lens, nh, 0.09, window, a, b, True)
        assert pool.cache.last_kernel() == llaisys.Kernel.DECODE_TMA
        assert (one.double() - pool.expect_fade(q[:3], [1, 1, 1], lens, 0.09, window, a, b)).abs().max().item() <= 1.2e-2


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("rows", [5, 1100])
def test_factors_on_the_query_heads(cuda_device, dtype, rows):
    """Norm, then a factor per query head; keys get the norm alone."""
    nh, nkvh, d, dv = 6, 2, 64, 48
    g = torch.Generator().manual_seed(rows)
    pages = rows // 16 + 2
    cache = llaisys.PagedKVCache.with_layers(pages, [(nkvh, d, dv)], dtype=LL[dtype], max_seqs=1, max_pages_per_seq=pages)
    seq = cache.add_seq()
    cache.reserve(seq, rows)
    cache.flush()
    width = (nh + nkvh) * d + nkvh * dv
    proj, wq, wk = (torch.randn(*s, generator=g).to(dtype) for s in ((rows, width), (d,), (d,)))
    temp = torch.randn(nh, generator=g)
    q_out = torch.zeros(rows, nh, d, dtype=dtype, device="cuda")
    cache.norm_append_dev(0, stream(), proj=proj.cuda(), row_stride=width, q_at=0, k_at=nh * d, v_at=(nh + nkvh) * d, gate_at=-1,
                          q_norm=wq.cuda(), k_norm=wk.cuda(), eps=1e-4, gate_scale=1.0, q_out=q_out, row_scale=None,
                          seq_ids_dev=i32([seq] * rows), positions_dev=i32(list(range(rows))), n_rows=rows, nh=nh, head_scale=temp.cuda())
    cache.check()
    want = oracle.rms(proj[:, :nh * d].double().view(rows, nh, d), 1e-4) * wq.double() * temp.double().unsqueeze(1)
    tol = 1e-5 if dtype == torch.float32 else 2 ** -7
    assert (q_out.cpu().double() - want).abs().max().item() <= tol * want.abs().max().item()
    # the keys, through attention: a query along one key's direction scores |k|^2 / |k| = |k| there
    k = oracle.rms(proj[:, nh * d:(nh + nkvh) * d].double().view(rows, nkvh, d), 1e-4) * wk.double()
    v = proj[:, (nh + nkvh) * d:].double().view(rows, nkvh, dv)
    q = torch.randn(1, nh, d, generator=g).to(dtype)
    out = torch.zeros(1, nh, dv, dtype=dtype, device="cuda")
    cache.attention_dev(0, out, q.cuda(), i32([seq]), None, i32([rows]), n_seqs=1, total_q=1, max_q_len=1, max_kv_len=rows, nh=nh, scale=0.3,
                        stream=stream())
    want = oracle.softmax_attention(q.double(), k, v, 0.3, first=rows - 1)
    assert (out.cpu().double() - want).abs().max().item() <= (2e-5 if dtype == torch.float32 else 2e-2) * max(1.0, want.abs().max().item())


# ---- latents ----------------------------------------------------------------------------------------------------------------


class Latents:
    """A one-layer cache of latents for several sequences, on shuffled pages."""

    def __init__(self, dtype, rank, rot, lens, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.rank, self.rot, self.lens = dtype, rank, rot, lens
        pages = [-(-n // 16) for n in lens]
        self.cache = llaisys.PagedKVCache.with_latents(sum(pages) + 5, [(rank, rot)], dtype=LL[dtype], max_seqs=len(lens) + 2,
                                                       max_pages_per_seq=max(pages) + 3)
        junk = self.cache.add_seq()
        self.cache.reserve(junk, 40)
        self.seqs = [self.cache.add_seq() for _ in lens]
        order = list(np.random.default_rng(seed).permutation(sum(pages) + 2) + 3)
        self.cache.free_seq(junk)
        for s, n in zip(self.seqs, pages):
            self.cache.assign_pages(s, [int(order.pop()) for _ in range(n)])
        self.cache.flush()
        self.down = [torch.randn(n, rank + rot, generator=g).to(dtype) for n in lens]
        self.norm = (1 + 0.3 * torch.randn(rank, generator=g)).to(dtype)
        self.q_norm = (1 + 0.3 * torch.randn(24, generator=g)).to(dtype)

    def append(self, lo, hi, base=50.0, nh=3):
        """-> normed query latents and gate factors of the rows"""
        ids, pos, rows = [], [], []
        for i, (a, b) in enumerate(zip(lo, hi)):
            rows.append(self.down[i][a:b])
            ids += [self.seqs[i]] * (b - a)
            pos += list(range(a, b))
        kv = torch.cat(rows)
        g = torch.Generator().manual_seed(len(pos))
        q, gate = torch.randn(len(pos), 24, generator=g).to(self.dtype), torch.randn(len(pos), nh, generator=g).to(self.dtype)
        proj = torch.cat([gate, q, kv, gate], dim=1).contiguous().cuda()
        table = torch.empty(len(pos), max(self.rot // 2, 1), 2, device="cuda")
        if self.rot:
            freq = torch.tensor([base ** (-2.0 * i / self.rot) for i in range(self.rot // 2)], dtype=torch.float64, device="cuda")
            llaisys.rotary_table_wide_dev(table, i32(pos), freq, len(pos), self.rot // 2, stream=stream())
        latent = torch.full((len(pos), 32), 3.0, dtype=self.dtype, device="cuda")
        factor = torch.empty(len(pos), nh, device="cuda")
        self.cache.latent_append_dev(0, stream(), proj=proj, row_stride=proj.shape[1], q_at=nh, kv_at=nh + 24, gate_at=0, q_rank=24,
                                     rank=self.rank, rot_dims=self.rot, nh=nh, q_norm=self.q_norm.cuda(), kv_norm=self.norm.cuda(), eps=1e-4,
                                     rot_table=table, q_latent=latent, q_latent_stride=32, row_scale=factor, seq_ids_dev=i32(ids),
                                     positions_dev=i32(pos), n_rows=len(pos))
        self.cache.check()
        tol = 1e-5 if self.dtype == torch.float32 else 2 ** -7
        want = oracle.rms(q.double(), 1e-4) * self.q_norm.double()
        assert (latent[:, :24].cpu().double() - want).abs().max().item() <= tol * 4 and torch.all(latent[:, 24:] == 3.0)
        assert (factor.cpu().double() - torch.sigmoid(gate.double())).abs().max().item() <= 1e-6
        return table, pos

    def rows(self, i, base=50.0):
        """What the pages hold, in float64 (rounded as they are)."""
        c = oracle.rms(self.down[i][:, :self.rank].double(), 1e-4) * self.norm.double()
        z = oracle.turn_pairs(self.down[i][:, self.rank:].double(), range(self.lens[i]), base) if self.rot else self.down[i][:, self.rank:].double()
        return torch.cat([c, z], dim=1).to(self.dtype).double()

    def attend(self, q, q_lens, kv_lens, nh, scale, factor, decode):
        n, rows = len(q_lens), sum(q_lens)
        out = torch.full((rows, nh * self.rank + 8), 7.0, dtype=self.dtype, device="cuda")
        starts = i32([0, *np.cumsum(q_lens).tolist()])
        self.cache.attention_dev(0, out, q.cuda().contiguous(), i32(self.seqs[:n]), None if decode else starts, i32(kv_lens), n_seqs=n,
                                 total_q=rows, max_q_len=max(q_lens), max_kv_len=max(kv_lens), nh=nh, scale=scale, stream=stream(),
                                 row_scale=factor.cuda() if factor is not None else None, row_stride=nh * self.rank + 8)
        self.cache.check()
        assert torch.all(out[:, nh * self.rank:] == 7.0)
        return out[:, :nh * self.rank].reshape(rows, nh, self.rank).cpu()

    def expect(self, q, q_lens, kv_lens, scale, factor):
        outs = []
        for i, (n, kv) in enumerate(zip(q_lens, kv_lens)):
            part, rows = q[sum(q_lens[:i]):sum(q_lens[:i + 1])].double(), self.rows(i)[:kv]
            outs.append(oracle.softmax_attention(part, rows.unsqueeze(1), rows[:, :self.rank].unsqueeze(1), scale, first=kv - n))
        return torch.cat(outs) * (factor.double().unsqueeze(-1) if factor is not None else 1.0)


# dtype, heads, rank, turned dims
LATENT_SHAPES = [(torch.float32, 3, 40, 16), (torch.bfloat16, 6, 88, 40), (torch.bfloat16, 16, 512, 64), (torch.bfloat16, 5, 64, 64),
                 (torch.bfloat16, 40, 256, 64), (torch.bfloat16, 1, 128, 0), (torch.float16, 12, 384, 24), (torch.bfloat16, 3, 13, 6),
                 (torch.bfloat16, 32, 200, 8), (torch.bfloat16, 7, 72, 56)]
LATENT_TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2, torch.float16: 3e-3}


@pytest.mark.parametrize("dtype,nh,rank,rot", LATENT_SHAPES)
def test_latent_attention_decode_and_portions(cuda_device, dtype, nh, rank, rot):
    lens = [1, 15, 16, 17, 127, 128, 129, 300]
    x = Latents(dtype, rank, rot, lens, seed=rank)
    half = [n // 2 for n in lens]
    x.append([0] * len(lens), half)
    x.append(half, lens)
    g = torch.Generator().manual_seed(3)
    scale = 1.5 * (rank + rot) ** -0.5
    for q_lens in ([1] * len(lens), [1, 2, 1, 17, 40, 1, 3, 64]):
        q = torch.randn(sum(q_lens), nh, rank + rot, generator=g).to(dtype)
        factor = torch.rand(sum(q_lens), nh, generator=g) * 2 - 0.5
        want = x.expect(q, q_lens, lens, scale, factor)
        for decode in ([True, False] if max(q_lens) == 1 else [False]):
            got = x.attend(q, q_lens, lens, nh, scale, factor, decode)
            kernel = x.cache.last_kernel()
            assert kernel == (llaisys.Kernel.GENERIC if dtype == torch.float32 or rank % 8 or rot % 8 else llaisys.Kernel.LATENT_TC)
            assert (got.double() - want).abs().max().item() <= LATENT_TOL[dtype] * max(1.0, want.abs().max().item()), (q_lens, decode)


@pytest.mark.parametrize("dtype,nh,rank,rot", [LATENT_SHAPES[1], LATENT_SHAPES[2], LATENT_SHAPES[0]])
def test_one_latent_far_away_wins(cuda_device, dtype, nh, rank, rot):
    """A row that stands out, at the first token, at page and tile borders and in the middle, against a thousand others: seen by every query
    from its own position on and by none before."""
    n = 1100
    for place in (0, 15, 16, 127, 128, 500, 1023):
        x = Latents(dtype, rank, rot, [n], seed=place)
        x.norm = torch.ones(rank).to(dtype)
        x.down[0][place, :rank] = 0.0
        x.down[0][place, 0] = 1.0  # after the norm: sqrt(rank) in one place
        x.append([0], [n])
        q = torch.zeros(n, nh, rank + rot)
        q[..., 0] = 60.0 / rank ** 0.5
        q = q.to(dtype)
        value = x.rows(0)[place, :rank]
        for q_len, kv in ((1, place + 1), (1, n), (40, min(n, place + 20)), (70, n)):
            q_len = min(q_len, kv)
            got = x.attend(q[:q_len], [q_len], [kv], nh, 1.0, None, False)
            want = x.expect(q[:q_len], [q_len], [kv], 1.0, None)
            assert (got.double() - want).abs().max().item() <= LATENT_TOL[dtype] * max(1.0, want.abs().max().item()), (place, q_len, kv)
            if kv - 1 >= place:
                assert (got[-1].double() - value).abs().max().item() <= 0.02 * value.abs().max().item(), (place, kv)
            if kv - q_len < place:
                assert (got[0].double() - value).abs().max().item() > 0.5 * value.abs().max().item()


def test_latent_units_cut_over_many_pieces(cuda_device):
    """One long sequence over all SMs, and many unequal ones: the same results twice, and against the oracle."""
    for lens, nh in (([5000], 16), ([4000, 30, 1500, 2, 700, 129, 64], 6)):
        x = Latents(torch.bfloat16, 128, 64, lens, seed=len(lens))
        x.append([0] * len(lens), lens)
        q = torch.randn(len(lens), nh, 192, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16)
        want = x.expect(q, [1] * len(lens), lens, 0.1, None)
        first = x.attend(q, [1] * len(lens), lens, nh, 0.1, None, True)
        assert x.cache.last_kernel() == llaisys.Kernel.LATENT_TC
        assert (first.double() - want).abs().max().item() <= 2e-2
        assert torch.equal(first, x.attend(q, [1] * len(lens), lens, nh, 0.1, None, True))


@pytest.mark.parametrize("dtype,nh,dim,rot,dv", [(torch.bfloat16, 4, 128, 64, 128), (torch.bfloat16, 6, 64, 64, 64), (torch.float16, 3, 40, 24, 128),
                                                 (torch.bfloat16, 2, 104, 8, 64), (torch.bfloat16, 1, 8, 64, 128)])
def test_expanded_attention(cuda_device, dtype, nh, dim, rot, dv):
    """Gathered rows and chunk attention over keys in two parts: unequal chunks, some left out, contexts in front of some."""
    rank = 48
    lens, q_lens, left_out = [300, 17, 64, 1000, 129, 5], [130, 17, 1, 257, 100, 3], {2, 5}
    x = Latents(dtype, rank, rot, lens, seed=dim)
    x.append([0] * 6, lens)
    starts, at = [], 0
    for i, n in enumerate(lens):
        starts.append(-1 if i in left_out else at // 16)
        at += 0 if i in left_out else (n + 15) // 16 * 16
    context = torch.full((at + 64, rank + rot), float("nan"), dtype=dtype, device="cuda")
    context[at:] = 0
    x.cache.latent_gather_dev(0, context, rank + rot, i32(x.seqs), i32(starts), i32(lens), 6, max(lens), stream())
    x.cache.check()
    held = context.cpu().double()
    assert torch.isfinite(held).all()
    g = torch.Generator().manual_seed(2)
    uk, uv = torch.randn(nh * dim, rank, generator=g).to(dtype) / rank ** 0.5, torch.randn(nh * dv, rank, generator=g).to(dtype) / rank ** 0.5
    keys, values = (context[:, :rank] @ uk.cuda().T).contiguous(), (context[:, :rank] @ uv.cuda().T).contiguous()
    rows = sum(q_lens)
    q = torch.randn(rows, nh, dim + rot, generator=g).to(dtype)
    factor = torch.rand(rows, nh, generator=g)
    out = torch.full((rows, nh * dv + 16), 7.0, dtype=dtype, device="cuda")
    scale = 1.4 * (dim + rot) ** -0.5
    torch.cuda.synchronize()
    x.cache.expanded_dev(stream(), q=q.cuda(), k=keys, k_shared=context.data_ptr() + rank * 2, v=values, shared_stride=rank + rot, tokens=at + 64,
                         nh=nh, dim=dim, rot_dim=rot, vdim=dv, page_starts_dev=i32(starts), q_starts_dev=i32([0, *np.cumsum(q_lens).tolist()]),
                         kv_lens_dev=i32(lens), n_seqs=6, scale=scale, out=out, out_stride=nh * dv + 16, row_scale=factor.cuda())
    x.cache.check()
    assert x.cache.last_kernel() == llaisys.Kernel.EXPANDED_TC and torch.all(out[:, nh * dv:] == 7.0)
    got = out[:, :nh * dv].reshape(rows, nh, dv).cpu()
    for i in range(6):
        lo = sum(q_lens[:i])
        if i in left_out:
            assert torch.all(got[lo:lo + q_lens[i]] == 7.0)
            continue
        s = starts[i] * 16
        assert torch.equal(held[s:s + lens[i]], x.rows(i)) or (held[s:s + lens[i]] - x.rows(i)).abs().max() <= 2 ** -6
        c = held[s:s + lens[i]]
        k = torch.cat([keys[s:s + lens[i]].cpu().double().view(-1, nh, dim), c[:, rank:].unsqueeze(1).expand(-1, nh, rot)], dim=-1)
        v = values[s:s + lens[i]].cpu().double().view(-1, nh, dv)
        want = oracle.softmax_attention(q[lo:lo + q_lens[i]].double(), k, v, scale, first=lens[i] - q_lens[i]) * factor[lo:lo + q_lens[i]].double().unsqueeze(-1)
        assert (got[lo:lo + q_lens[i]].double() - want).abs().max().item() <= LATENT_TOL[dtype] * max(1.0, want.abs().max().item()), i


@pytest.mark.parametrize("dtype", BOTH)
def test_rotation_of_neighbouring_dims(cuda_device, dtype):
    """Far positions, other dims untouched, in place and into wider rows."""
    rows, nh, dim, rot, base = 9, 3, 10, 12, 1e4
    pos = [0, 1, 2, 15, 16, 1000, 70000, 131071, 5]
    q = torch.randn(rows, nh, dim + rot).to(dtype)
    freq = torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64, device="cuda")
    table = torch.empty(rows, rot // 2, 2, device="cuda")
    llaisys.rotary_table_wide_dev(table, i32(pos), freq, rows, rot // 2, stream=stream())
    wide = torch.full((rows, nh, 40), 7.0, dtype=dtype, device="cuda")
    on = q.cuda()
    llaisys.rotate_pairs_dev(LL[dtype], wide, 40, 20, on, dim, rot, table, rows, nh, stream=stream())
    llaisys.rotate_pairs_dev(LL[dtype], on, dim + rot, dim, on, dim, rot, table, rows, nh, stream=stream())
    sync()
    want = oracle.turn_pairs(q[..., dim:].double(), pos, base)
    tol = 1e-6 if dtype == torch.float32 else 2 ** -7
    assert (on[..., dim:].cpu().double() - want).abs().max().item() <= tol * 4
    assert torch.equal(on[..., :dim].cpu(), q[..., :dim]) and torch.equal(wide[..., 20:32], on[..., dim:])
    assert torch.all(wide[..., :20] == 7.0) and torch.all(wide[..., 32:] == 7.0)


# ---- state space ------------------------------------------------------------------------------------------------------------


class States:
    """Inputs of one state-space layer for several sequences, and both ways to run them."""

    def __init__(self, dtype, heads, groups, dk, dv, taps, parts, lens, *, bias=-2.0, spread=1.5, a_spread=0.7, seed=0):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.dtype, self.heads, self.groups, self.dk, self.dv, self.taps, self.parts, self.lens = dtype, heads, groups, dk, dv, taps, parts, lens
        inner, up8 = heads * dv, lambda n: (n + 7) // 8 * 8
        self.inner, self.channels = inner, inner + 2 * groups * dk
        self.z_at = 8
        self.x_at = self.z_at + up8(inner)
        self.dt_at = self.x_at + up8(self.channels)
        self.width = self.dt_at + up8(heads) + 8
        self.proj = [rand(t, self.width).to(dtype) for t in lens]
        self.conv_w, self.conv_b = (rand(self.channels, taps) / taps ** 0.5).to(dtype), (0.3 * rand(self.channels)).to(dtype)
        self.norm_w = (1 + 0.3 * rand(inner)).to(dtype)
        self.a_log, self.dt_bias, self.d_skip = a_spread * rand(heads), bias + spread * rand(heads), rand(heads)
        state, _, self.segment_floats = llaisys.state_space_sizes(LL[dtype], 1, heads, groups, dk, dv, taps)
        self.stride = (state + 3) // 4 * 4 + 8
        self.slots = len(lens) + 3
        # slots start with garbage: a sequence's first token must not see it
        self.state = torch.full((self.slots, self.stride), float("nan"), device="cuda")
        self.slot_of = [int(s) for s in torch.randperm(self.slots, generator=g)[:len(lens)]]
        self.out_width = up8(inner) + 16

    def inputs(self, p):
        """What enters the recurrence, in float64; convolutions rounded where the device rounds them."""
        T, p = p.shape[0], p.double()
        xbc = oracle.convolve(p[:, self.x_at:self.x_at + self.channels], self.conv_w.double(), self.conv_b.double()).to(self.dtype).double()
        x, B, C = xbc.split([self.inner, self.groups * self.dk, self.groups * self.dk], dim=1)
        dt = oracle.softplus(p[:, self.dt_at:self.dt_at + self.heads] + self.dt_bias.double())
        return x.reshape(T, self.heads, self.dv), B.reshape(T, self.groups, -1), C.reshape(T, self.groups, -1), dt, self.a_log.double(), self.d_skip.double()

    def expect(self):
        outs, states = [], []
        for p in self.proj:
            y, S = oracle.state_space(*self.inputs(p))
            z = p[:, self.z_at:self.z_at + self.inner].double()
            outs.append(oracle.gated_parts_norm(y.reshape(len(p), -1), z, self.norm_w.double(), self.parts, 1e-4))
            states.append(S)
        return outs, states

    def run(self, lo, hi, decode=False, segments=True):
        """Rows [lo_i, hi_i) of every sequence with any -> their outputs"""
        who = [i for i in range(len(self.lens)) if hi[i] > lo[i]]
        counts = [hi[i] - lo[i] for i in who]
        rows = sum(counts)
        proj = torch.cat([self.proj[i][lo[i]:hi[i]] for i in who]).cuda().contiguous()
        out = torch.full((rows, self.out_width), 5.0, dtype=self.dtype, device="cuda")
        n_scratch = llaisys.state_space_sizes(LL[self.dtype], rows, self.heads, self.groups, self.dk, self.dv, self.taps)[1]
        scratch = torch.full((n_scratch,), float("nan"), device="cuda")
        seg = torch.full((self.segment_floats,), float("nan"), device="cuda") if self.segment_floats and segments else None
        dev = {n: getattr(self, n).cuda().contiguous() for n in ("conv_w", "conv_b", "norm_w", "a_log", "dt_bias", "d_skip")}
        torch.cuda.synchronize()
        llaisys.state_space_dev(
            LL[self.dtype], decode=decode, stream=stream(), proj=proj, row_stride=self.width, z_at=self.z_at, x_at=self.x_at, dt_at=self.dt_at,
            **dev, taps=self.taps, heads=self.heads, groups=self.groups, dk=self.dk, dv=self.dv, norm_groups=self.parts, eps=1e-4,
            state=self.state, slot_stride=self.stride, seq_ids_dev=i32([self.slot_of[i] for i in who]),
            q_starts_dev=i32([0, *np.cumsum(counts).tolist()]), kv_lens_dev=i32([hi[i] for i in who]), n_seqs=len(who), n_rows=rows,
            max_q_len=max(counts), out=out, out_stride=self.out_width, scratch=scratch, scratch_floats=n_scratch, scratch_segments=seg,
            scratch_segment_floats=self.segment_floats if seg is not None else 0)
        sync()
        assert torch.all(out[:, self.inner:] == 5.0)
        return list(out[:, :self.inner].cpu().split(counts))

    def check(self, got, want, what=""):
        tol = 3e-5 if self.dtype == torch.float32 else 1.5e-2
        for i, (a, b) in enumerate(zip(got, want)):
            err = ((a.double() - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt()).max().item()
            assert err <= tol, f"{what} sequence {i}: {err:.2e}"

    def check_states(self, states):
        # the state is f32 in both; in bfloat16 a convolution at a rounding boundary may fall to the other side
        tol = 1e-5 if self.dtype == torch.float32 else 4e-3
        for i, S in enumerate(states):
            got = self.state[self.slot_of[i]][:S.numel()].view_as(S).cpu().double()
            scale = S.abs().amax(dim=(1, 2), keepdim=True)
            assert ((got - S).abs() / scale).max().item() <= tol, f"state of sequence {i}"


# dtype, heads, groups, state size, value size, taps, parts of the norm
STATE_SHAPES = [(torch.float32, 2, 1, 24, 20, 3, 1), (torch.float32, 6, 3, 64, 64, 4, 2), (torch.float32, 1, 1, 300, 33, 2, 3),
                (torch.bfloat16, 4, 2, 64, 64, 4, 1), (torch.bfloat16, 4, 1, 128, 64, 4, 4), (torch.bfloat16, 3, 3, 128, 128, 2, 1),
                (torch.bfloat16, 2, 1, 16, 32, 1, 2), (torch.bfloat16, 2, 2, 40, 24, 5, 1), (torch.bfloat16, 2, 1, 13, 9, 3, 6),
                (torch.bfloat16, 1, 1, 96, 200, 4, 1), (torch.bfloat16, 2, 1, 144, 48, 4, 2), (torch.bfloat16, 8, 4, 32, 8, 4, 8)]


@pytest.mark.parametrize("shape", STATE_SHAPES)
def test_states_whole_and_carried(cuda_device, shape):
    lens = [1, 2, 31, 63, 64, 65, 130]
    n = len(lens)
    x = States(*shape, lens)
    want, states = x.expect()
    x.check(x.run([0] * n, lens), want, "whole")
    x.check_states(states)
    # the same in portions that end anywhere, sequences joining and pausing, single tokens in between
    y = States(*shape, lens)
    at, got = [0] * n, [[] for _ in lens]
    sizes = [7, 1, 40, 2, 64, 33, 3]
    step = 0
    while any(a < m for a, m in zip(at, lens)):
        hi = [min(m, a + sizes[(i + step) % 7]) if (i + step) % 3 else a for i, (a, m) in enumerate(zip(at, lens))]
        if hi != at:
            outs = iter(y.run(at, hi))
            for i in range(n):
                if hi[i] > at[i]:
                    got[i].append(next(outs))
        at, step = hi, step + 1
    y.check([torch.cat(o) for o in got], want, "portions")
    y.check_states(states)


@pytest.mark.parametrize("shape", STATE_SHAPES)
def test_states_token_by_token_and_in_two_token_portions(cuda_device, shape):
    """(Portions of two tokens are shorter than most convolutions: their inputs come from several portions back.)"""
    lens = [20, 9, 20]
    x = States(*shape, lens, seed=1)
    want, states = x.expect()
    got = [[] for _ in lens]
    for t in range(20):
        lo, hi = [min(t, n) for n in lens], [min(t + 1, n) for n in lens]
        outs = iter(x.run(lo, hi, decode=True))
        for i in range(3):
            if hi[i] > lo[i]:
                got[i].append(next(outs))
    x.check([torch.cat(o) for o in got], want, "decode")
    x.check_states(states)
    y = States(*shape, [23], seed=6)
    want, states = y.expect()
    y.check([torch.cat([y.run([t], [min(t + 2, 23)])[0] for t in range(0, 23, 2)])], want, "pairs")
    y.check_states(states)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("bias,spread,a_spread", [(3.0, 3.0, 1.0), (0.0, 8.0, 2.0), (30.0, 40.0, 0.5), (-9.0, 1.0, 0.2)])
def test_states_strong_and_weak_decay(cuda_device, dtype, bias, spread, a_spread):
    """Heads that forget everything within a token beside heads that keep it for the whole sequence."""
    lens = [200, 77]
    x = States(dtype, 6, 2, 64, 64, 3, 1, lens, bias=bias, spread=spread, a_spread=a_spread, seed=2)
    want, states = x.expect()
    x.check(x.run([0, 0], lens), want, f"bias {bias}")
    x.check_states(states)


@pytest.mark.parametrize("shape", [(torch.bfloat16, 1, 1, 128, 64, 4, 1), (torch.bfloat16, 2, 1, 64, 128, 4, 1), (torch.bfloat16, 3, 3, 40, 24, 2, 1),
                                   (torch.bfloat16, 1, 1, 32, 200, 4, 1), (torch.float32, 1, 1, 64, 64, 4, 1)])
def test_states_long_runs(cuda_device, shape):
    """Runs long enough to be cut into segments: the same outputs and states as uncut, from a fresh and from a carried state."""
    lens = [1500, 700, 3, 1]
    make = lambda: States(*shape, lens, bias=-5.0, seed=3)  # noqa: E731
    x = make()
    want, states = x.expect()
    x.check(x.run([0] * 4, lens), want, "cut")
    x.check_states(states)
    y = make()
    y.check(y.run([0] * 4, lens, segments=False), want, "uncut")
    y.check_states(states)
    z = make()
    first = z.run([0] * 4, [410, 5, 1, 1])
    rest = z.run([410, 5, 1, 1], lens)
    z.check([torch.cat(p) for p in zip(first, [*rest, torch.empty(0, z.inner)])], want, "carried over")
    z.check_states(states)


@pytest.mark.parametrize("dtype", BOTH)
def test_one_far_write_stays_in_the_state(cuda_device, dtype):
    """One token's step is large, all others' next to nothing, through heads that hardly decay: hundreds of tokens later its x is what every
    read along its B returns, so a state lost between portions or tiles shows."""
    lens = [400]
    x = States(dtype, 1, 1, 64, 64, 2, 1, lens, bias=-6.0, spread=0.0, a_spread=0.0, seed=4)
    x.a_log[:] = -9.0
    x.d_skip[:] = 0.0
    x.proj[0][:, x.dt_at] = -8.0
    x.proj[0][30, x.dt_at] = 9.0
    B_at = x.x_at + x.inner
    x.proj[0][29:31, B_at:B_at + 64] = 1.0
    x.proj[0][31:, B_at + 64:B_at + 128] = 1.0
    want, states = x.expect()
    xs, B, C, dt, _, _ = x.inputs(x.proj[0])
    y = oracle.state_space(*x.inputs(x.proj[0]))[0][399, 0]
    assert torch.nn.functional.cosine_similarity(y, xs[30, 0] * (B[30, 0] @ C[399, 0]).sign(), dim=0).item() > 0.95  # as it claims to be
    a = x.run([0], [31])
    b = x.run([31], [32], decode=True)
    c = x.run([32], [395])
    d = [x.run([t], [t + 1], decode=True)[0] for t in range(395, 400)]
    x.check([torch.cat([a[0], b[0], c[0], *d])], want)
    x.check_states(states)


# ---- experts ----------------------------------------------------------------------------------------------------------------


class Experts:
    def __init__(self, dtype, experts, identity, top, groups, keep, width, ff, rows, seed=0, scale=1.3):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.dtype, self.rows, self.ff = dtype, rows, ff
        self.sizes = dict(experts=experts, identity=identity, top=top, groups=groups, keep=keep, width=width, ff=ff)
        self.scale = scale
        self.h, self.x, self.logits = rand(rows, width).to(dtype), rand(rows, width), 2.0 * rand(rows, experts + identity)
        self.correction = 0.1 * rand(experts + identity)
        self.gate, self.up = ((rand(experts, ff, width) / width ** 0.5).to(dtype) for _ in range(2))
        self.down = (rand(experts, width, ff) / ff ** 0.5).to(dtype)
        self.gain = torch.tensor(0.8)
        self.counts = torch.zeros(experts, dtype=torch.int32, device="cuda")

    def router(self):
        s = self.sizes
        return {"top": s["top"], "scale": self.scale, "groups": {"count": s["groups"], "keep": s["keep"]}}

    def run(self):
        s = self.sizes
        n, top, width = self.rows, s["top"], s["width"]
        ints = lambda: torch.full((n, top), -7, dtype=torch.int32, device="cuda")  # noqa: E731
        buf = lambda w: torch.full((n * top, w), float("nan"), dtype=self.dtype, device="cuda")  # noqa: E731
        gate_up = torch.cat([self.gate, self.up], dim=1).contiguous().cuda()
        x, h, chosen, weights = self.x.cuda(), self.h.cuda(), ints(), torch.zeros(n, top, device="cuda")
        keep = [self.down.cuda().contiguous(), self.correction.cuda(), self.logits.cuda(), self.gain.cuda(), ints(), ints(), buf(width), buf(self.ff),
                buf(width)]
        torch.cuda.synchronize()
        llaisys.experts_dev(LL[self.dtype], stream=stream(), **s, n_rows=n, scale=self.scale, eps=1e-4, gate_up=gate_up, down=keep[0],
                            correction=keep[1], logits=keep[2], gain=keep[3], h=h, chosen=chosen, weights=weights, place=keep[4],
                            counts=self.counts, line=keep[5], rows=keep[6], act=keep[7], out=keep[8], x=x, next=h)
        sync()
        assert torch.all(self.counts == 0)
        return x.cpu(), h.cpu(), chosen.cpu(), weights.cpu()

    def expect(self, chosen):
        """The sum with the device's own choice (compared on its own) in float64."""
        s, out = self.sizes, self.x.double().clone()
        h = self.h.double()
        for t in range(self.rows):
            score = torch.softmax(self.logits[t].double(), 0)[chosen[t].long()]
            weight = score / (score.sum() + 1e-20) * self.scale
            for e, w in zip(chosen[t].tolist(), weight):
                if e < s["experts"]:
                    a = h[t] @ self.gate[e].double().T
                    out[t] += w * ((a * torch.sigmoid(a) * (h[t] @ self.up[e].double().T)) @ self.down[e].double().T)
                else:
                    out[t] += w * h[t]
        return out

    def check(self):
        x, nxt, chosen, weights = self.run()
        for t in range(self.rows):
            want, weight = oracle.route(self.logits[t].double(), self.correction.double(), self.router())
            order = {int(e): float(w) for e, w in zip(want, weight)}
            assert sorted(order) == sorted(chosen[t].tolist()), f"row {t}"
            assert all(abs(order[int(e)] - float(w)) <= 2e-6 * max(1.0, self.scale) for e, w in zip(chosen[t], weights[t]))
        want = self.expect(chosen)
        spread = (want - self.x.double()).pow(2).mean().sqrt().item()
        tol = {torch.float32: 2e-5, torch.float16: 4e-3, torch.bfloat16: 2e-2}[self.dtype]
        assert (x.double() - want).pow(2).mean(-1).sqrt().max().item() <= tol * spread
        norm = oracle.rms(want, 1e-4) * float(self.gain)
        assert (nxt.double() - norm).abs().max().item() <= {torch.float32: 1e-4, torch.float16: 0.01, torch.bfloat16: 0.06}[self.dtype]


# dtype, experts, identity, top, groups, keep, width, ff, rows
EXPERT_SHAPES = [(torch.float32, 6, 2, 2, 4, 3, 48, 40, 33), (torch.float32, 5, 0, 1, 1, 1, 51, 19, 7), (torch.bfloat16, 8, 4, 3, 3, 2, 64, 64, 100),
                 (torch.bfloat16, 16, 0, 4, 4, 4, 128, 256, 1), (torch.bfloat16, 3, 3, 2, 2, 1, 320, 72, 65), (torch.float16, 12, 3, 4, 5, 2, 192, 136, 50),
                 (torch.bfloat16, 4, 0, 2, 1, 1, 520, 200, 700), (torch.bfloat16, 1, 0, 1, 1, 1, 64, 24, 300), (torch.bfloat16, 2, 6, 2, 4, 4, 40, 48, 90),
                 (torch.bfloat16, 64, 8, 6, 8, 3, 128, 64, 40), (torch.bfloat16, 5, 1, 2, 1, 1, 51, 33, 20), (torch.float16, 3, 0, 3, 3, 3, 256, 384, 260)]


@pytest.mark.parametrize("shape", EXPERT_SHAPES)
def test_experts(cuda_device, shape):
    Experts(*shape).check()


def test_experts_all_rows_to_one_and_none_to_any(cuda_device):
    """Every row to the same expert (one line of one expert); every choice an identity expert (no row at all)."""
    for dtype in BOTH:
        e = Experts(dtype, 8, 2, 1, 1, 1, 64, 32, 300, seed=3)
        e.logits[:, 5] = 30.0
        e.check()
        e = Experts(dtype, 4, 4, 2, 2, 1, 64, 32, 70, seed=4)
        e.logits[:, 4:] += 20.0
        x, _, chosen, weights = e.run()
        assert (chosen >= 4).all()
        want = e.x.double() + 1.3 * e.h.double()
        assert (x.double() - want).abs().max().item() <= 1e-5 * want.abs().max().item()


def test_choice_scores_below_zero_and_groups(cuda_device):
    """Corrections below zero: outputs of refused groups must not win as if they stood at zero; the correction decides the choice but not the
    weight."""
    e = Experts(torch.float32, 6, 3, 2, 3, 1, 32, 16, 50, seed=5)
    e.correction = torch.full((9,), -3.0)
    e.check()
    e.correction = torch.tensor([-5.0, -5.0, -1.0, -3.0, -3.0, -3.0, -3.0, -3.0, -3.0])
    x, _, chosen, weights = e.run()
    assert all(2 in row for row in chosen.tolist()) and all(set(row) <= {0, 1, 2} for row in chosen.tolist())
    e.check()
