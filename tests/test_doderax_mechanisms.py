"""The mechanisms of the Doderax layers alone, on the device, against float64 statements of the same: sliding-window attention
that keeps a sequence's first tokens, the rotation + append in front of it, and the gated delta rule with its convolutions."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from oracle import doderax as oracle
from tests.test_vozozen_mechanisms import LL, SHAPES, TOL, Pool, i32, stream

pytestmark = pytest.mark.gpu


def rotary_table(positions, dims, base):
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32, device="cuda")
    table = torch.empty(len(positions), dims // 2, 2, device="cuda")
    llaisys.rotary_table_dev(table, i32(positions), freq, len(positions), dims // 2, stream=stream())
    return table


# ---- attention --------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", SHAPES)
@pytest.mark.parametrize("window,keep", [(1, 1), (5, 3), (16, 16), (33, 17), (64, 40), (200, 6), (20, 100), (100000, 5)])
def test_kept_first_tokens_decode_and_portions(cuda_device, dtype, nkvh, nh, d, dv, window, keep):
    lens = [1, 15, 16, 17, 130, 300, 64, 65]
    pool = Pool(dtype, nkvh, d, dv, lens, seed=window)
    pool.append([0] * len(lens), lens)
    g = torch.Generator().manual_seed(3)
    scale = 1.3 * d ** -0.5
    for q_lens, kv_lens in (([1] * len(lens), lens), ([min(n, 3 + 40 * (i % 4)) for i, n in enumerate(lens)], lens), (lens, lens)):
        q = torch.randn(sum(q_lens), nh, d, generator=g).to(dtype)
        want = pool.expect(q, q_lens, kv_lens, scale, window, None, keep)
        for decode in ([True, False] if max(q_lens) == 1 else [False]):
            got = pool.attend(q, q_lens, kv_lens, nh, scale, window, None, decode, keep)
            assert (got.double() - want).abs().max().item() <= TOL[dtype] * max(1.0, want.abs().max().item()), (q_lens, decode)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv", [SHAPES[1], SHAPES[3], SHAPES[4]])
@pytest.mark.parametrize("window,keep", [(2, 1), (16, 15), (17, 16), (48, 17), (64, 64), (40, 65)])
def test_the_last_kept_and_the_first_dropped_token(cuda_device, dtype, nkvh, nh, d, dv, window, keep):
    """One key wins every softmax it takes part in. The last kept token is seen from everywhere; the one behind it, and a token
    in the middle, until the window has passed: queries around that edge, in a prompt and decoded alone."""
    for place in (0, keep - 1, keep, keep + 20):
        n = max(place + window, keep) + 90
        pool = Pool(dtype, nkvh, d, dv, [n], seed=place)
        pool.k[0] *= 0.05
        direction = torch.ones(d) / d ** 0.5
        pool.k[0][place] = (direction * 30).to(dtype)
        pool.append([0], [n])
        q = (direction.expand(n, nh, d) * 2.0).to(dtype).contiguous()
        got = pool.attend(q, [n], [n], nh, 1.0, window, None, False, keep)
        want = pool.expect(q, [n], [n], 1.0, window, None, keep)
        assert (got.double() - want).abs().max().item() <= TOL[dtype] * 4
        value = pool.v[0][place].double().repeat_interleave(nh // nkvh, 0)
        for at in (place + window - 1, place + window, n - 1):
            distance = (got[at].double() - value).abs().max().item()
            one = pool.attend(q[:1], [1], [at + 1], nh, 1.0, window, None, True, keep)
            assert (one[0].double() - want[at]).abs().max().item() <= TOL[dtype] * 4
            if place < keep or at < place + window:
                assert distance <= 0.02 * max(1.0, value.abs().max().item()), (place, at)
            else:
                assert distance > 0.1, (place, at)


def test_kept_tokens_on_the_fast_kernels_over_long_sequences(cuda_device):
    """Thousands of tokens, so that tiles are cut over CTAs and pairs over spans, with key blocks left out in between."""
    lens, nh = [4000, 2500, 700], 8
    for window, keep in ((700, 130), (300, 4), (65, 64)):
        pool = Pool(torch.bfloat16, 1, 128, 128, lens)
        pool.append([0, 0, 0], lens)
        q_lens = [600, 333, 700]
        q = torch.randn(sum(q_lens), nh, 128).to(torch.bfloat16)
        got = pool.attend(q, q_lens, lens, nh, 0.09, window, None, False, keep)
        assert pool.cache.last_kernel() == llaisys.Kernel.PREFILL_TC
        assert (got.double() - pool.expect(q, q_lens, lens, 0.09, window, None, keep)).abs().max().item() <= 1.2e-2
        one = pool.attend(q[:3], [1, 1, 1], lens, nh, 0.09, window, None, True, keep)
        assert pool.cache.last_kernel() == llaisys.Kernel.DECODE_TMA
        assert (one.double() - pool.expect(q[:3], [1, 1, 1], lens, 0.09, window, None, keep)).abs().max().item() <= 1.2e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d,dv,rot,base", [(64, 64, 16, 1e4), (20, 12, 20, 50.0), (128, 128, 128, 1e6), (13, 9, 6, 1e4), (24, 40, 24, 3.0),
                                           (256, 8, 2, 9.0)])
@pytest.mark.parametrize("rows", [37, 1100])
def test_rotation_and_append(cuda_device, dtype, d, dv, rot, base, rows):
    """The first dims of q and k turn with their position, far ones too; the rest, and v, pass."""
    nh, nkvh, first = 4, 2, 3000
    g = torch.Generator().manual_seed(d)
    cache = llaisys.PagedKVCache.with_layers((first + rows) // 16 + 3, [(nkvh, d, dv)], dtype=LL[dtype], max_seqs=2,
                                             max_pages_per_seq=(first + rows) // 16 + 1)
    seq = cache.add_seq()
    cache.reserve(seq, first + rows)
    cache.flush()
    width = (nh * d + nkvh * d + nkvh * dv + 15) // 8 * 8
    proj = torch.randn(rows, width, generator=g).to(dtype)
    positions = list(range(first, first + rows))
    q_out = torch.zeros(rows, nh, d, dtype=dtype, device="cuda")
    cache.norm_append_dev(0, stream(), proj=proj.cuda(), row_stride=width, q_at=0, k_at=nh * d, v_at=(nh + nkvh) * d, gate_at=-1,
                          q_norm=None, k_norm=None, eps=0.0, gate_scale=1.0, q_out=q_out, row_scale=None, seq_ids_dev=i32([seq] * rows),
                          positions_dev=i32(positions), n_rows=rows, nh=nh, rot_dims=rot, rot_table=rotary_table(positions, rot, base))
    cache.check()
    pick = [0, 1, 15, 16, rows - 1]
    for row in pick:
        x = proj[row:row + 1].double()
        want = oracle.rotate(x[:, :nh * d].view(1, nh, d), rot, base, first=first + row)[0]
        got = q_out[row].cpu().double()
        tol = 3e-4 if dtype == torch.float32 else 2 ** -7  # (f32 angles of up to 4000 radians)
        assert (got - want).abs().max().item() <= tol * max(1.0, want.abs().max().item())
        assert torch.equal(q_out[row].cpu()[:, rot:], proj[row, :nh * d].view(nh, d)[:, rot:])
        out = torch.zeros(1, nh, dv, dtype=dtype, device="cuda")
        cache.attention_dev(0, out, q_out[row:row + 1].contiguous(), i32([seq]), None, i32([first + row + 1]), n_seqs=1, total_q=1,
                            max_q_len=1, max_kv_len=first + rows, nh=nh, scale=1.0, stream=stream(), window=1)
        v = proj[row, (nh + nkvh) * d:(nh + nkvh) * d + nkvh * dv].view(nkvh, dv).repeat_interleave(2, 0)
        assert torch.equal(out[0].cpu(), v)
    if d == dv and d * proj.element_size() % 16 == 0:
        k_out, v_out = (torch.zeros(first + rows, nkvh, d, dtype=dtype, device="cuda") for _ in range(2))
        cache.gather(0, seq, first + rows, k_out, v_out)
        for row in pick:
            want = oracle.rotate(proj[row, nh * d:(nh + nkvh) * d].double().view(1, nkvh, d), rot, base, first=first + row)[0]
            assert (k_out[first + row].cpu().double() - want).abs().max().item() <= tol * max(1.0, want.abs().max().item())


# ---- gated delta rule -------------------------------------------------------------------------------------------------------


class Delta:
    """Inputs of one delta-rule layer for several sequences, and both ways to run them. rank 0: one decay per head."""

    def __init__(self, dtype, heads, kv_heads, dk, dv, taps, rank, lens, *, bias=-2.0, spread=2.0, seed=0, silu_gate=None, beta_bias=0.0):
        g = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
        self.dtype, self.heads, self.kv_heads, self.dk, self.dv, self.taps, self.rank, self.lens = dtype, heads, kv_heads, dk, dv, taps, rank, lens
        self.silu_gate = (rank == 0) if silu_gate is None else silu_gate
        nq, nv, up8 = kv_heads * dk, heads * dv, lambda n: (n + 7) // 8 * 8
        at, self.at = 8, {}
        for name, n in (("q", nq), ("k", nq), ("v", nv), ("b", heads), ("a", rank or heads), ("g", nv)):
            self.at[name], at = at, at + up8(n)
        self.width = at + 8
        self.proj = [rand(t, self.width) for t in lens]
        for p in self.proj:
            p[:, self.at["b"]:self.at["a"]] += beta_bias
        self.proj = [p.to(dtype) for p in self.proj]
        self.conv = {"q": rand(nq, taps) / taps ** 0.5, "k": rand(nq, taps) / taps ** 0.5, "v": rand(nv, taps) / taps ** 0.5}
        self.conv = {n: w.to(dtype) for n, w in self.conv.items()}
        self.decay_ld = up8(rank)
        self.decay_w = torch.nn.functional.pad(rand(heads * dk, rank) * 0.5, (0, self.decay_ld - rank)).to(dtype) if rank else None
        self.a_log = (0.5 * rand(heads)).to(dtype)
        self.dt_bias = (bias + spread * rand(heads * dk if rank else heads)).to(dtype)
        self.norm = (1 + 0.3 * rand(dv)).to(dtype)
        state, _, self.segment_floats = llaisys.gated_delta_sizes(LL[dtype], 1, heads, kv_heads, dk, dv, taps)
        self.stride = (state + 3) // 4 * 4 + 8
        self.slots = len(lens) + 3
        # slots start with garbage: a sequence's first token must not see it
        self.state = torch.full((self.slots, self.stride), float("nan"), device="cuda")
        self.slot_of = [int(s) for s in torch.randperm(self.slots, generator=g)[:len(lens)]]
        self.out_width = up8(nv) + 16
        self.dev = {n: t.cuda().contiguous() for n, t in (("conv_q", self.conv["q"]), ("conv_k", self.conv["k"]), ("conv_v", self.conv["v"]),
                                                         ("a_log", self.a_log), ("dt_bias", self.dt_bias), ("norm_w", self.norm))}
        self.dev["decay_w"] = self.decay_w.cuda().contiguous() if rank else None

    def part(self, p, name, n):
        return p[:, self.at[name]:self.at[name] + n]

    def inputs(self, p):
        """What enters the recurrence, in float64; convolutions rounded where the device rounds them."""
        T, H, G, dk = p.shape[0], self.heads, self.kv_heads, self.dk
        p = p.double()
        conv = {n: oracle.short_conv(self.part(p, n, w.shape[0]), w.double()).to(self.dtype).double() for n, w in self.conv.items()}
        q = oracle.unit(conv["q"].view(T, G, dk)).repeat_interleave(H // G, 1) * dk ** -0.5
        k = oracle.unit(conv["k"].view(T, G, dk)).repeat_interleave(H // G, 1)
        A, bias = self.a_log.double(), self.dt_bias.double()
        if self.rank:
            x = (self.part(p, "a", self.rank) @ self.decay_w[:, :self.rank].double().T + bias).view(T, H, dk)
            log = oracle.decay_log(A.unsqueeze(1), x)
        else:
            log = oracle.decay_log(A, self.part(p, "a", H) + bias).unsqueeze(2).expand(T, H, dk)
        return q, k, conv["v"].view(T, H, self.dv), log, torch.sigmoid(self.part(p, "b", H))

    def gate(self, p):
        y = self.part(p.double(), "g", self.heads * self.dv).view(p.shape[0], self.heads, self.dv)
        return oracle.silu(y) if self.silu_gate else torch.sigmoid(y)

    def expect(self):
        outs, states = [], []
        for p in self.proj:
            y, S = oracle.delta_rule(*self.inputs(p))
            outs.append(oracle.rms(y, 1e-4) * self.norm.double() * self.gate(p))
            states.append(S)
        return outs, states

    def run(self, lo, hi, decode=False, segments=True):
        """Rows [lo_i, hi_i) of every sequence with any; -> their outputs"""
        who = [i for i in range(len(self.lens)) if hi[i] > lo[i]]
        counts = [hi[i] - lo[i] for i in who]
        rows = sum(counts)
        proj = torch.cat([self.proj[i][lo[i]:hi[i]] for i in who]).cuda().contiguous()
        out = torch.full((rows, self.out_width), 5.0, dtype=self.dtype, device="cuda")
        n_scratch = llaisys.gated_delta_sizes(LL[self.dtype], rows, self.heads, self.kv_heads, self.dk, self.dv, self.taps)[1]
        scratch = torch.full((n_scratch,), float("nan"), device="cuda")
        seg = torch.full((self.segment_floats,), float("nan"), device="cuda") if self.segment_floats and segments else None
        torch.cuda.synchronize()
        llaisys.gated_delta_dev(
            LL[self.dtype], decode=decode, stream=stream(), proj=proj, row_stride=self.width, q_at=self.at["q"], k_at=self.at["k"],
            v_at=self.at["v"], b_at=self.at["b"], a_at=self.at["a"], **self.dev, decay_ld=self.decay_ld,
            gate=proj.data_ptr() + self.at["g"] * proj.element_size(), gate_stride=self.width, gate_silu=int(self.silu_gate),
            q_scale=self.dk ** -0.5, eps=1e-4, unit_eps=oracle.UNIT_EPS, taps=self.taps, heads=self.heads, kv_heads=self.kv_heads,
            dk=self.dk, dv=self.dv, rank=self.rank, state=self.state, slot_stride=self.stride,
            seq_ids_dev=i32([self.slot_of[i] for i in who]), q_starts_dev=i32([0, *np.cumsum(counts).tolist()]),
            kv_lens_dev=i32([hi[i] for i in who]), n_seqs=len(who), n_rows=rows, max_q_len=max(counts), out=out,
            out_stride=self.out_width, scratch=scratch, scratch_floats=n_scratch, scratch_segments=seg,
            scratch_segment_floats=self.segment_floats if seg is not None else 0)
        llaisys.RuntimeAPI(llaisys.DeviceType.NVIDIA).stream_synchronize(stream())
        assert torch.all(out[:, self.heads * self.dv:] == 5.0)
        return list(out[:, :self.heads * self.dv].reshape(rows, self.heads, self.dv).cpu().split(counts))

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


# dtype, heads, q/k heads, key size, value size, taps, decay rank
DELTA_SHAPES = [(torch.float32, 2, 1, 24, 20, 3, 5), (torch.float32, 4, 2, 64, 64, 4, 0), (torch.float32, 1, 1, 300, 33, 2, 4),
                (torch.bfloat16, 4, 2, 64, 64, 4, 16), (torch.bfloat16, 2, 2, 128, 128, 4, 16), (torch.bfloat16, 3, 1, 128, 128, 3, 0),
                (torch.bfloat16, 3, 3, 64, 128, 2, 0), (torch.bfloat16, 2, 1, 128, 64, 6, 40), (torch.bfloat16, 2, 2, 13, 9, 1, 3),
                (torch.bfloat16, 1, 1, 144, 256, 4, 20), (torch.bfloat16, 2, 1, 96, 200, 5, 130), (torch.bfloat16, 2, 1, 8, 8, 4, 0)]


@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_whole_and_carried(cuda_device, shape):
    lens = [1, 2, 31, 32, 33, 64, 65, 150]
    n = len(lens)
    x = Delta(*shape, lens)
    want, states = x.expect()
    x.check(x.run([0] * n, lens), want, "whole")
    x.check_states(states)
    # the same in portions that end anywhere, sequences joining and pausing, single tokens in between
    y = Delta(*shape, lens)
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


@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_token_by_token(cuda_device, shape):
    lens = [20, 9, 20]
    x = Delta(*shape, lens, seed=1)
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


@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_in_two_token_portions(cuda_device, shape):
    """Every portion shorter than the convolution: its inputs come from several portions back."""
    lens = [23]
    x = Delta(*shape, lens, seed=6)
    want, states = x.expect()
    x.check([torch.cat([x.run([t], [min(t + 2, 23)])[0] for t in range(0, 23, 2)])], want)
    x.check_states(states)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank", [0, 8])
@pytest.mark.parametrize("bias,spread", [(3.0, 3.0), (0.0, 12.0), (40.0, 60.0), (-9.0, 1.0), (-3.0, 2.0)])
def test_delta_strong_and_weak_decay(cuda_device, dtype, rank, bias, spread):
    """Channels that forget everything within a token beside channels that keep it for the whole sequence: no factor of the
    chunked form may overflow or lose what is left."""
    lens = [200, 77]
    x = Delta(dtype, 4, 2, 64, 64, 3, rank, lens, bias=bias, spread=spread, seed=2)
    want, states = x.expect()
    x.check(x.run([0, 0], lens), want, f"bias {bias}")
    x.check_states(states)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank", [0, 8])
def test_delta_repeated_keys_written_in_full(cuda_device, dtype, rank):
    """Keys that are all alike, write strength one and no decay: every token replaces what the one before it wrote, the hardest
    triangular systems. The read-out along that key is the newest value alone."""
    lens = [100]
    x = Delta(dtype, 2, 1, 64, 32, 2, rank, lens, bias=-30.0, spread=0.0, seed=5, beta_bias=20.0)
    x.proj[0][:, x.at["k"]:x.at["v"]] = x.proj[0][:1, x.at["k"]:x.at["v"]]
    want, states = x.expect()
    x.check(x.run([0], lens), want)
    x.check_states(states)
    q, k, v, _, beta = x.inputs(x.proj[0])
    assert beta.min().item() > 0.9999
    S = x.state[x.slot_of[0]][:2 * 64 * 32].view(2, 64, 32).cpu().double()
    read = torch.einsum("hdv,hd->hv", S, k[-1])
    assert (read - v[-1]).abs().max().item() <= 2e-2 * v[-1].abs().max().item()


@pytest.mark.parametrize("dtype,heads,kv_heads,dk,dv,rank", [(torch.bfloat16, 1, 1, 128, 128, 16), (torch.bfloat16, 2, 1, 64, 96, 0),
                                                             (torch.bfloat16, 1, 1, 96, 256, 0), (torch.bfloat16, 3, 3, 40, 24, 5),
                                                             (torch.float32, 1, 1, 64, 64, 8)])
def test_delta_long_runs(cuda_device, dtype, heads, kv_heads, dk, dv, rank):
    """Runs long enough to be cut into segments: the same outputs and states as uncut, from a fresh and from a carried state."""
    lens = [1500, 700, 3]
    make = lambda: Delta(dtype, heads, kv_heads, dk, dv, 4, rank, lens, bias=-6.0, seed=3)  # noqa: E731
    x = make()
    want, states = x.expect()
    x.check(x.run([0] * 3, lens), want, "cut")
    x.check_states(states)
    y = make()
    y.check(y.run([0] * 3, lens, segments=False), want, "uncut")
    y.check_states(states)
    z = make()
    first = z.run([0] * 3, [410, 5, 1])
    rest = z.run([410, 5, 1], lens)
    z.check([torch.cat(p) for p in zip(first, rest)], want, "carried over")
    z.check_states(states)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank", [0, 8])
def test_one_far_write_stays_in_the_state(cuda_device, dtype, rank):
    """Every token but one writes next to nothing, hundreds of tokens pass through channels that hardly decay: the value written
    at token 30 is what every later query along its key reads, so a state lost between portions or chunks shows."""
    lens = [400]
    x = Delta(dtype, 1, 1, 64, 64, 2, rank, lens, bias=-14.0, spread=0.5, seed=4, beta_bias=-12.0)
    x.proj[0][30, x.at["b"]] = 12.0
    x.proj[0][31:, x.at["q"]:x.at["k"]] = 1.0
    x.proj[0][29:31, x.at["k"]:x.at["v"]] = 1.0
    x.conv["k"] = x.conv["q"].clone()
    x.dev["conv_k"] = x.conv["k"].cuda()
    want, states = x.expect()
    _, _, v, _, _ = x.inputs(x.proj[0])
    raw = want[0][399, 0] / (x.norm.double() * x.gate(x.proj[0])[399, 0])
    assert torch.nn.functional.cosine_similarity(raw, v[30, 0], dim=0).item() > 0.95  # the case is what it claims to be
    a = x.run([0], [31])
    b = x.run([31], [32], decode=True)
    c = x.run([32], [395])
    d = [x.run([t], [t + 1], decode=True)[0] for t in range(395, 400)]
    x.check([torch.cat([a[0], b[0], c[0], *d])], want)
    x.check_states(states)
