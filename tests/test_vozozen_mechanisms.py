"""The mechanisms of the Vozozen layers alone, on the device, against float64 statements of the same: sliding-window
attention with an output factor per head, the norm + append in front of it, and gated linear attention."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from oracle import vozozen as oracle

pytestmark = pytest.mark.gpu
LL = {torch.float32: llaisys.DataType.F32, torch.bfloat16: llaisys.DataType.BF16}
TOL = {torch.float32: 2e-5, torch.bfloat16: 1.2e-2}


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


def stream():
    return llaisys.context_stream()


class Pool:
    """A one-layer cache of several sequences filled through norm_append (norms of ones would still divide by the rms, so
    keys go in without a norm)."""

    def __init__(self, dtype, nkvh, d, dv, lens, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.nkvh, self.d, self.dv, self.lens = dtype, nkvh, d, dv, lens
        pages = [-(-n // 16) for n in lens]
        self.cache = llaisys.PagedKVCache.with_layers(sum(pages) + 5, [(nkvh, d, dv)], dtype=LL[dtype], max_seqs=len(lens) + 2,
                                                      max_pages_per_seq=max(pages) + 3)
        junk = self.cache.add_seq()  # shifts slots and pages, then goes away
        self.cache.reserve(junk, 40)
        self.seqs = [self.cache.add_seq() for _ in lens]
        order = list(np.random.default_rng(seed).permutation(sum(pages) + 2) + 3)
        self.cache.free_seq(junk)
        for s, n in zip(self.seqs, pages):
            self.cache.assign_pages(s, [int(order.pop()) for _ in range(n)])
        self.k = [torch.randn(n, nkvh, d, generator=g).to(dtype) for n in lens]
        self.v = [torch.randn(n, nkvh, dv, generator=g).to(dtype) for n in lens]

    def append(self, lo, hi):
        rows, ids, pos = [], [], []
        for i, (a, b) in enumerate(zip(lo, hi)):
            rows.append(torch.cat([self.k[i][a:b].reshape(b - a, -1), self.v[i][a:b].reshape(b - a, -1)], dim=1))
            ids += [self.seqs[i]] * (b - a)
            pos += list(range(a, b))
        proj = torch.nn.functional.pad(torch.cat(rows), (self.d, 8)).cuda().contiguous()
        q_sink = torch.empty(len(ids), 1, self.d, dtype=self.dtype, device="cuda")
        self.cache.flush()
        self.cache.norm_append_dev(0, stream(), proj=proj, row_stride=proj.shape[1], q_at=0, k_at=self.d,
                                   v_at=self.d + self.nkvh * self.d, gate_at=-1, q_norm=None, k_norm=None, eps=0.0,
                                   gate_scale=1.0, q_out=q_sink, row_scale=None, seq_ids_dev=i32(ids), positions_dev=i32(pos),
                                   n_rows=len(ids), nh=1)
        self.cache.check()

    def attend(self, q, q_lens, kv_lens, nh, scale, window, factor, decode, keep_first=0):
        n = len(q_lens)
        rows = sum(q_lens)
        width = nh * self.dv + 24
        out = torch.full((rows, width), 7.0, dtype=self.dtype, device="cuda")
        starts = i32([0, *np.cumsum(q_lens).tolist()])
        self.cache.attention_dev(0, out, q.cuda().contiguous(), i32(self.seqs[:n]), None if decode else starts, i32(kv_lens),
                                 n_seqs=n, total_q=rows, max_q_len=max(q_lens), max_kv_len=max(kv_lens), nh=nh, scale=scale,
                                 stream=stream(), window=window, keep_first=keep_first, row_scale=factor.cuda() if factor is not None else None,
                                 row_stride=width)
        self.cache.check()
        assert torch.all(out[:, nh * self.dv:] == 7.0), "columns behind the heads were written"
        return out[:, :nh * self.dv].reshape(rows, nh, self.dv).cpu()

    def expect(self, q, q_lens, kv_lens, scale, window, factor, keep_first=0):
        outs, at = [], 0
        for i, (n, kv) in enumerate(zip(q_lens, kv_lens)):
            share = q.shape[1] // self.nkvh
            for t in range(n):
                last = kv - n + t
                first = max(0, last - window + 1) if window else 0
                seen = [*range(min(keep_first, first)), *range(first, last + 1)]
                k = self.k[i][seen].double().repeat_interleave(share, 1)
                v = self.v[i][seen].double().repeat_interleave(share, 1)
                s = torch.einsum("jhd,hd->hj", k, q[at].double()) * scale
                o = torch.einsum("hj,jhd->hd", s.softmax(-1), v)
                outs.append(o * (factor[at].double().unsqueeze(1) if factor is not None else 1.0))
                at += 1
        return torch.stack(outs)


SHAPES = [(torch.float32, 2, 6, 20, 12), (torch.float32, 1, 3, 64, 64), (torch.bfloat16, 2, 4, 64, 32), (torch.bfloat16, 3, 3, 40, 72),
          (torch.bfloat16, 2, 12, 128, 128), (torch.bfloat16, 1, 8, 128, 128)]


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", SHAPES)
@pytest.mark.parametrize("window", [1, 5, 16, 33, 64, 200, 100000])
def test_window_attention_decode_and_portions(cuda_device, dtype, nkvh, nh, d, dv, window):
    lens = [1, 15, 16, 17, 130, 300, 64, 65]
    pool = Pool(dtype, nkvh, d, dv, lens, seed=window)
    pool.append([0] * len(lens), lens)
    g = torch.Generator().manual_seed(3)
    scale = 1.3 * d ** -0.5
    for q_lens, kv_lens in (([1] * len(lens), lens), ([min(n, 3 + 40 * (i % 4)) for i, n in enumerate(lens)], lens),
                            (lens, lens), ([1, 2, 1, 17, 129, 1, 2, 64], lens)):
        q = torch.randn(sum(q_lens), nh, d, generator=g).to(dtype)
        factor = torch.rand(sum(q_lens), nh, generator=g) * 2 - 0.5
        want = pool.expect(q, q_lens, kv_lens, scale, window, factor)
        for decode in ([True, False] if max(q_lens) == 1 else [False]):
            got = pool.attend(q, q_lens, kv_lens, nh, scale, window, factor, decode)
            assert (got.double() - want).abs().max().item() <= TOL[dtype] * max(1.0, want.abs().max().item()), (q_lens, decode)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", [SHAPES[1], SHAPES[3], SHAPES[4]])
@pytest.mark.parametrize("window", [2, 16, 17, 48, 64, 129])
def test_a_key_just_inside_and_just_outside_the_window(cuda_device, dtype, nkvh, nh, d, dv, window):
    """One key is made to win every softmax it takes part in. Queries at every distance around the window's edge either
    return its value or do not notice it, in prompts and decoded alone, for places at and beside page borders."""
    for place in (0, 15, 16, 31, 40):
        n = place + window + 3
        pool = Pool(dtype, nkvh, d, dv, [n], seed=place)
        pool.k[0] *= 0.05
        direction = torch.ones(d) / d ** 0.5
        pool.k[0][place] = (direction * 30).to(dtype)
        pool.append([0], [n])
        q = (direction.expand(n, nh, d) * 2.0).to(dtype).contiguous()
        got = pool.attend(q, [n], [n], nh, 1.0, window, None, False)
        want = pool.expect(q, [n], [n], 1.0, window, None)
        assert (got.double() - want).abs().max().item() <= TOL[dtype] * 4
        value = pool.v[0][place].double().repeat_interleave(nh // nkvh, 0)
        inside, outside = got[place + window - 1].double(), got[place + window].double()
        assert (inside - value).abs().max().item() <= 0.02 * max(1.0, value.abs().max().item())
        assert (outside - value).abs().max().item() > 0.1
        for last in (place + window - 1, place + window):
            one = pool.attend(q[:1], [1], [last + 1], nh, 1.0, window, None, True)
            assert (one[0].double() - want[last]).abs().max().item() <= TOL[dtype] * 4


def test_the_fast_kernels_serve_windows(cuda_device):
    pool = Pool(torch.bfloat16, 2, 128, 128, [100])
    pool.append([0], [100])
    q = torch.randn(100, 8, 128).to(torch.bfloat16)
    pool.attend(q, [100], [100], 8, 0.1, 30, None, False)
    assert pool.cache.last_kernel() == llaisys.Kernel.PREFILL_TC
    pool.attend(q[:1], [1], [100], 8, 0.1, 30, None, True)
    assert pool.cache.last_kernel() == llaisys.Kernel.DECODE_TMA


def test_window_over_a_long_sequence_on_the_fast_kernels(cuda_device):
    """Thousands of tokens, so that tiles are cut over CTAs and pairs over spans."""
    lens, window, nh = [4000, 2500], 700, 8
    pool = Pool(torch.bfloat16, 1, 128, 128, lens)
    pool.append([0, 0], lens)
    q_lens = [600, 333]
    q = torch.randn(sum(q_lens), nh, 128).to(torch.bfloat16)
    got = pool.attend(q, q_lens, lens, nh, 0.09, window, None, False)
    want = pool.expect(q, q_lens, lens, 0.09, window, None)
    assert (got.double() - want).abs().max().item() <= 1.2e-2
    one = pool.attend(q[:2], [1, 1], lens, nh, 0.09, window, None, True)
    assert (one.double() - pool.expect(q[:2], [1, 1], lens, 0.09, window, None)).abs().max().item() <= 1.2e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,dv", [(64, 64), (20, 12), (128, 128), (13, 9), (24, 40), (256, 8)])
@pytest.mark.parametrize("rows", [37, 1100])
def test_norm_append(cuda_device, dtype, d, dv, rows):
    """q and k per head over their own root mean square, gates to factors, v untouched; k and v arrive in their pages."""
    nh, nkvh, eps = 4, 2, 1e-3
    g = torch.Generator().manual_seed(d)
    cache = llaisys.PagedKVCache.with_layers(rows // 16 + 3, [(1, 8, 8), (nkvh, d, dv)], dtype=LL[dtype], max_seqs=2)
    seq = cache.add_seq()
    cache.reserve(seq, rows)
    cache.flush()
    width = (nh * d + nkvh * d + nkvh * dv + nh + 10) // 8 * 8
    proj = (torch.randn(rows, width, generator=g) * 0.3).to(dtype)
    qn, kn = ((1 + 0.3 * torch.randn(d, generator=g)).to(dtype) for _ in range(2))
    q_out = torch.zeros(rows, nh, d, dtype=dtype, device="cuda")
    factor = torch.zeros(rows, nh, device="cuda")
    cache.norm_append_dev(1, stream(), proj=proj.cuda(), row_stride=width, q_at=0, k_at=nh * d, v_at=(nh + nkvh) * d,
                          gate_at=(nh + nkvh) * d + nkvh * dv, q_norm=qn.cuda(), k_norm=kn.cuda(), eps=eps, gate_scale=0.37,
                          q_out=q_out, row_scale=factor, seq_ids_dev=i32([seq] * rows), positions_dev=i32(range(rows)),
                          n_rows=rows, nh=nh)
    cache.check()
    p = proj.double()
    want_q = oracle.rms_norm(p[:, :nh * d].view(rows, nh, d), qn.double(), eps)
    want_k = oracle.rms_norm(p[:, nh * d:(nh + nkvh) * d].view(rows, nkvh, d), kn.double(), eps)
    tol = 1e-6 if dtype == torch.float32 else 2 ** -8
    assert ((q_out.cpu().double() - want_q).abs() <= tol * want_q.abs() + 1e-6).all()
    gates = p[:, (nh + nkvh) * d + nkvh * dv:][:, :nh]
    assert (factor.cpu().double() - 0.37 * torch.sigmoid(gates)).abs().max().item() <= 1e-6
    # k and v as attention sees them: a query of one huge coordinate picks one key, whose value comes back
    for row in (0, 15, 16, rows - 1):
        q = torch.zeros(1, nh, d, dtype=dtype)
        out = torch.zeros(1, nh, dv, dtype=dtype, device="cuda")
        cache.attention_dev(1, out, q.cuda(), i32([seq]), None, i32([row + 1]), n_seqs=1, total_q=1, max_q_len=1,
                            max_kv_len=rows, nh=nh, scale=1.0, stream=stream(), window=1)
        v = proj[row, (nh + nkvh) * d:(nh + nkvh) * d + nkvh * dv].view(nkvh, dv).repeat_interleave(2, 0)
        assert torch.equal(out[0].cpu(), v)
    if d == dv and d * proj.element_size() % 16 == 0:
        k_out, v_out = (torch.zeros(rows, nkvh, d, dtype=dtype, device="cuda") for _ in range(2))
        cache.gather(1, seq, rows, k_out, v_out)
        assert ((k_out.cpu().double() - want_k).abs() <= tol * want_k.abs() + 1e-6).all()


# ---- gated linear attention -----------------------------------------------------------------------------------------------


class Gla:
    """Inputs of one gated-linear layer for several sequences, and both ways to run them."""

    def __init__(self, dtype, heads, dk, dv, rank, lens, tau, bias=2.0, spread=2.0, seed=0, k_size=1.0):
        g = torch.Generator().manual_seed(seed)
        self.dtype, self.heads, self.dk, self.dv, self.rank, self.lens, self.tau = dtype, heads, dk, dv, rank, lens, tau
        n = heads * dk
        self.at = dict(q_at=8, k_at=8 + n, v_at=8 + 2 * n, g_at=8 + 2 * n + heads * dv, z_at=8 + 2 * n + 2 * heads * dv)
        self.width = self.at["z_at"] + rank + 5
        self.proj = [torch.randn(t, self.width, generator=g) * 0.7 for t in lens]
        for p in self.proj:
            p[:, self.at["k_at"]:self.at["v_at"]] *= k_size
        self.proj = [p.to(dtype) for p in self.proj]
        self.w = (torch.randn(n, rank, generator=g) * 0.5).to(dtype)
        self.b = (bias + spread * torch.randn(n, generator=g)).to(dtype)
        self.norm = (1 + 0.3 * torch.randn(dv, generator=g)).to(dtype)
        self.slots = len(lens) + 3
        self.stride = (heads * dk * dv + 3) // 4 * 4 + 8
        # slots start with garbage: a sequence's first token must not see it
        self.state = torch.full((self.slots, self.stride), float("nan"), device="cuda")
        self.slot_of = [int(s) for s in torch.randperm(self.slots, generator=g)[:len(lens)]]
        self.out_width = heads * dv + 16

    def expect(self):
        outs, states = [], []
        for p in self.proj:
            p = p.double()
            T, a, n, m = p.shape[0], self.at, self.heads * self.dk, self.heads * self.dv
            q = p[:, a["q_at"]:][:, :n].view(T, self.heads, self.dk) * self.dk ** -0.5
            k = p[:, a["k_at"]:][:, :n].view(T, self.heads, self.dk)
            v = p[:, a["v_at"]:][:, :m].view(T, self.heads, self.dv)
            z = p[:, a["z_at"]:][:, :self.rank] @ self.w.double().T + self.b.double()
            y, S = oracle.gated_linear(q, k, v, oracle.key_decay(z, self.tau).view(T, self.heads, self.dk))
            gate = oracle.silu(p[:, a["g_at"]:][:, :m]).view(T, self.heads, self.dv)
            outs.append(1.7 * oracle.rms_norm(y, self.norm.double(), 1e-4) * gate)
            states.append(S)
        return outs, states

    def run(self, lo, hi, decode=False, segments=True):
        """Rows [lo_i, hi_i) of every sequence with any; -> their outputs"""
        who = [i for i in range(len(self.lens)) if hi[i] > lo[i]]
        counts = [hi[i] - lo[i] for i in who]
        rows = sum(counts)
        proj = torch.cat([self.proj[i][lo[i]:hi[i]] for i in who]).cuda().contiguous()
        out = torch.full((rows, self.out_width), 5.0, dtype=self.dtype, device="cuda")
        raw = torch.empty(rows, self.heads * self.dv, device="cuda")
        decay = torch.empty(rows, self.heads * self.dk, device="cuda")
        n_seg = llaisys.gated_linear_segment_floats(LL[self.dtype], self.heads, self.dk, self.dv)
        seg = torch.full((n_seg,), float("nan"), device="cuda") if n_seg and segments else None
        torch.cuda.synchronize()
        llaisys.gated_linear_dev(
            LL[self.dtype], decode=decode, stream=stream(), proj=proj, row_stride=self.width, **self.at, decay_w=self.w.cuda(),
            decay_b=self.b.cuda(), norm_w=self.norm.cuda(), tau=self.tau, q_scale=self.dk ** -0.5, eps=1e-4, out_scale=1.7,
            heads=self.heads, dk=self.dk, dv=self.dv, rank=self.rank, state=self.state, slot_stride=self.stride,
            seq_ids_dev=i32([self.slot_of[i] for i in who]), q_starts_dev=i32([0, *np.cumsum(counts).tolist()]),
            kv_lens_dev=i32([hi[i] for i in who]), n_seqs=len(who), n_rows=rows, max_q_len=max(counts), out=out,
            out_stride=self.out_width, scratch_raw=raw, scratch_decay=decay, scratch_segments=seg, scratch_segment_floats=n_seg if seg is not None else 0)
        llaisys.RuntimeAPI(llaisys.DeviceType.NVIDIA).stream_synchronize(stream())
        assert torch.all(out[:, self.heads * self.dv:] == 5.0)
        return list(out[:, :self.heads * self.dv].reshape(rows, self.heads, self.dv).cpu().split(counts))

    def check(self, got, want, what=""):
        tol = 3e-5 if self.dtype == torch.float32 else 1.5e-2
        for i, (a, b) in enumerate(zip(got, want)):
            err = ((a.double() - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt()).max().item()
            assert err <= tol, f"{what} sequence {i}: {err:.2e}"

    def check_states(self, states):
        tol = 1e-5 if self.dtype == torch.float32 else 2e-4  # (the state is f32 in both; its inputs are the same)
        for i, S in enumerate(states):
            got = self.state[self.slot_of[i]][:S.numel()].view_as(S).cpu().double()
            scale = S.abs().amax(dim=(1, 2), keepdim=True)
            assert ((got - S).abs() / scale).max().item() <= tol, f"state of sequence {i}"


GLA_SHAPES = [(torch.float32, 2, 24, 20, 5, 4.0), (torch.float32, 3, 64, 64, 16, 16.0), (torch.bfloat16, 3, 64, 64, 16, 16.0),
              (torch.bfloat16, 2, 128, 128, 16, 8.0), (torch.bfloat16, 1, 48, 72, 7, 2.0), (torch.bfloat16, 2, 13, 9, 3, 1.0),
              (torch.bfloat16, 1, 144, 256, 20, 16.0), (torch.float32, 1, 300, 33, 4, 2.0), (torch.bfloat16, 2, 96, 128, 33, 5.0)]


@pytest.mark.parametrize("dtype,heads,dk,dv,rank,tau", GLA_SHAPES)
def test_gated_linear_whole_and_carried(cuda_device, dtype, heads, dk, dv, rank, tau):
    lens = [1, 2, 63, 64, 65, 150]
    x = Gla(dtype, heads, dk, dv, rank, lens, tau)
    want, states = x.expect()
    x.check(x.run([0] * 6, lens), want, "whole")
    x.check_states(states)
    # the same in portions that end anywhere, sequences joining and pausing, single tokens in between
    y = Gla(dtype, heads, dk, dv, rank, lens, tau)
    at, got = [0] * 6, [[] for _ in lens]
    sizes = [7, 1, 40, 64, 2, 33]
    step = 0
    while any(a < n for a, n in zip(at, lens)):
        hi = [min(n, a + sizes[(i + step) % 6]) if (i + step) % 3 else a for i, (a, n) in enumerate(zip(at, lens))]
        if hi != at:
            outs = iter(y.run(at, hi))
            for i in range(6):
                if hi[i] > at[i]:
                    got[i].append(next(outs))
        at, step = hi, step + 1
    y.check([torch.cat(o) for o in got], want, "portions")
    y.check_states(states)


@pytest.mark.parametrize("dtype,heads,dk,dv,rank,tau", GLA_SHAPES)
def test_gated_linear_token_by_token(cuda_device, dtype, heads, dk, dv, rank, tau):
    lens = [20, 9, 20]
    x = Gla(dtype, heads, dk, dv, rank, lens, tau, seed=1)
    want, states = x.expect()
    got = [[] for _ in lens]
    for t in range(20):
        lo = [min(t, n) for n in lens]
        hi = [min(t + 1, n) for n in lens]
        outs = iter(x.run(lo, hi, decode=True))
        for i in range(3):
            if hi[i] > lo[i]:
                got[i].append(next(outs))
    x.check([torch.cat(o) for o in got], want, "decode")
    x.check_states(states)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("bias,spread,tau", [(-6.0, 3.0, 1.0), (0.0, 12.0, 1.0), (-40.0, 30.0, 0.5), (9.0, 1.0, 16.0), (-3.0, 2.0, 2.0)])
def test_gated_linear_strong_and_weak_decay(cuda_device, dtype, bias, spread, tau):
    """Channels that forget everything within a token beside channels that keep it for the whole sequence: no factor of the
    chunked form may overflow or lose what is left."""
    lens = [200, 77]
    x = Gla(dtype, 2, 64, 64, 8, lens, tau, bias=bias, spread=spread, seed=2)
    want, states = x.expect()
    x.check(x.run([0, 0], lens), want, f"bias {bias}")
    x.check_states(states)


@pytest.mark.parametrize("dtype,heads,dk,dv", [(torch.bfloat16, 1, 128, 128), (torch.bfloat16, 2, 64, 96), (torch.float32, 1, 64, 64)])
def test_gated_linear_long_runs(cuda_device, dtype, heads, dk, dv):
    """Runs long enough to be cut into segments: the same outputs and states as uncut, and what a far token left behind is
    still there."""
    lens = [1500, 700, 3]
    x = Gla(dtype, heads, dk, dv, 16, lens, 16.0, bias=6.0, seed=3)
    want, states = x.expect()
    x.check(x.run([0] * 3, lens), want, "cut")
    x.check_states(states)
    y = Gla(dtype, heads, dk, dv, 16, lens, 16.0, bias=6.0, seed=3)
    y.check(y.run([0] * 3, lens, segments=False), want, "uncut")
    y.check_states(states)
    z = Gla(dtype, heads, dk, dv, 16, lens, 16.0, bias=6.0, seed=3)
    first = z.run([0] * 3, [410, 5, 1])
    rest = z.run([410, 5, 1], lens)
    z.check([torch.cat(p) for p in zip(first, rest)], want, "carried over")
    z.check_states(states)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_far_key_stays_in_the_state(cuda_device, dtype):
    """One key a hundred times the others', hundreds of tokens back, through channels that hardly decay: its value dominates
    every later output, so a state lost between portions or chunks shows."""
    lens = [400]
    x = Gla(dtype, 1, 64, 64, 8, lens, 16.0, bias=12.0, spread=0.5, seed=4, k_size=0.01)
    x.proj[0][30, x.at["k_at"]:x.at["v_at"]] = 3.0
    x.proj[0][:, x.at["q_at"]:x.at["k_at"]] = 0.5
    want, states = x.expect()
    value = x.proj[0][30, x.at["v_at"]:][:64].double()
    raw = want[0][399, 0] / (1.7 * x.norm.double() * oracle.silu(x.proj[0][399, x.at["g_at"]:][:64].double()))
    assert torch.nn.functional.cosine_similarity(raw, value, dim=0).item() > 0.95  # the case is what it claims to be
    a = x.run([0], [31])
    b = x.run([31], [32], decode=True)
    c = x.run([32], [395])
    d = [x.run([t], [t + 1], decode=True)[0] for t in range(395, 400)]
    x.check([torch.cat([a[0], b[0], c[0], *d])], want)
    x.check_states(states)
