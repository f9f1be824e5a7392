"""The mechanisms of the Lilovik layers alone, on the device, against float64 statements of the same: attention without a softmax and
its mixing over the heads, the row norm + query factor + append in front of it, and the minGRU."""
import numpy as np
import pytest
import torch

import llaisys_b200 as llaisys
from oracle import lilovik as oracle
from tests.test_vozozen_mechanisms import LL, Pool, i32, stream

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
TOL = {F32: 2e-5, BF16: 1.2e-2}


class Gates:
    """A filled pool and the constants of one layer's attention."""

    def __init__(self, dtype, nkvh, nh, d, dv, lens, *, softcap=5.0, talk=True, bias=True, slopes=None, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.pool, self.dtype, self.nh, self.dv, self.softcap = Pool(dtype, nkvh, d, dv, lens, seed=seed), dtype, nh, dv, softcap
        self.talk = (0.7 * torch.eye(nh) + torch.randn(nh, nh, generator=g) * 0.5 / nh ** 0.5).to(dtype) if talk else None
        self.bias = (torch.randn(nh, generator=g) - 1.5).to(dtype) if bias else None
        self.slopes = oracle.slopes(nh).float() if slopes is None else torch.tensor(slopes, dtype=F32)

    def run(self, q, q_lens, kv_lens, scale, *, decode, window=0):
        n, rows, width = len(q_lens), sum(q_lens), self.nh * self.dv + 24
        out = torch.full((rows, width), 7.0, dtype=self.dtype, device="cuda")
        keep = [None if t is None else t.cuda() for t in (self.slopes, self.bias, self.talk)]
        self.pool.cache.gates_dev(0, out, q.cuda().contiguous(), i32(self.pool.seqs[:n]),
                                  None if decode else i32([0, *np.cumsum(q_lens).tolist()]), i32(kv_lens), n_seqs=n, total_q=rows,
                                  max_q_len=max(q_lens), max_kv_len=max(kv_lens), nh=self.nh, scale=scale, stream=stream(),
                                  softcap=self.softcap, slopes=keep[0], bias=keep[1], talk=keep[2], window=window, row_stride=width)
        self.pool.cache.check()
        assert torch.all(out[:, self.nh * self.dv:] == 7.0), "columns behind the heads were written"
        return out[:, :self.nh * self.dv].reshape(rows, self.nh, self.dv).cpu()

    def expect(self, q, q_lens, kv_lens, scale, *, window=0):
        outs, at = [], 0
        for i, (n, kv) in enumerate(zip(q_lens, kv_lens)):
            k, v = self.pool.k[i][:kv].double(), self.pool.v[i][:kv].double()
            a = torch.zeros(self.nh, n, kv, dtype=torch.float64)
            ago = torch.arange(kv - n, kv).unsqueeze(1) - torch.arange(kv).unsqueeze(0)
            share = self.nh // k.shape[1]
            for h in range(self.nh):
                s = q[at:at + n, h].double() @ k[:, h // share].T * scale
                s = self.softcap * torch.tanh(s / self.softcap) if self.softcap else s
                s = s - self.slopes[h].double() * ago + (self.bias[h].double() if self.bias is not None else 0.0)
                a[h] = torch.where((ago >= 0) & ((ago < window) if window else True), torch.sigmoid(s), torch.zeros_like(s))
            if self.talk is not None:
                a = oracle.mix_heads(a, self.talk.double())
            outs.append(oracle.weigh_values(a, v))
            at += n
        return torch.cat(outs)


def test_the_statement_here_is_the_oracles():
    g = Gates.__new__(Gates)
    gen = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(n, h, 8, generator=gen, dtype=torch.float64) for n, h in ((5, 4), (9, 2), (9, 2)))
    g.nh, g.softcap, g.slopes = 4, 3.0, oracle.slopes(4)
    g.talk, g.bias = torch.randn(4, 4, generator=gen, dtype=torch.float64), torch.randn(4, generator=gen, dtype=torch.float64)
    g.pool = type("P", (), {"k": [k], "v": [v]})
    want = oracle.mixed_gate_attention(q, k, v, 0.4, 3.0, g.bias, g.talk, first=4)
    assert (g.expect(q, [5], [9], 0.4) - want).abs().max() < 1e-12


def close(got, want, dtype, factor=1.0, what=""):
    err = (got.double() - want).abs().max().item()
    assert err <= TOL[dtype] * factor * max(1.0, want.abs().max().item()), (what, err, want.abs().max().item())


# dtype, kv heads, heads, key size, value size; does the tile kernel serve it
SHAPES = [(F32, 2, 6, 20, 12, False), (F32, 3, 3, 64, 64, False), (BF16, 3, 3, 40, 72, False), (BF16, 1, 5, 13, 9, False),
          (BF16, 5, 5, 64, 64, True), (BF16, 2, 6, 64, 32, True), (BF16, 3, 3, 16, 48, True), (BF16, 1, 7, 32, 128, True),
          (BF16, 8, 32, 128, 128, True), (BF16, 2, 12, 128, 128, True), (BF16, 5, 20, 96, 112, True), (BF16, 1, 1, 128, 16, True),
          (BF16, 24, 24, 32, 32, True), (BF16, 2, 64, 48, 80, True), (BF16, 25, 25, 32, 32, False), (BF16, 1, 66, 32, 32, False),
          (BF16, 1, 5, 128, 128, True), (BF16, 4, 4, 128, 128, True), (BF16, 16, 32, 128, 128, True), (BF16, 3, 24, 128, 128, True)]
LENS = [1, 15, 16, 17, 130, 300, 64, 65]


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv,tiles", SHAPES)
@pytest.mark.parametrize("options", [{}, {"softcap": 0.0}, {"talk": False}, {"bias": False, "softcap": 1.2}])
def test_gates_decode_and_portions(cuda_device, dtype, nkvh, nh, d, dv, tiles, options):
    g = Gates(dtype, nkvh, nh, d, dv, LENS, seed=nh, **options)
    g.pool.append([0] * len(LENS), LENS)
    gen = torch.Generator().manual_seed(3)
    scale = 1.5 * d ** -0.5
    for q_lens in ([1] * len(LENS), [min(n, 3 + 40 * (i % 4)) for i, n in enumerate(LENS)], LENS, [1, 2, 1, 17, 129, 1, 2, 64]):
        q = torch.randn(sum(q_lens), nh, d, generator=gen).to(dtype)
        want = g.expect(q, q_lens, LENS, scale)
        for decode in ([True, False] if max(q_lens) == 1 else [False]):
            close(g.run(q, q_lens, LENS, scale, decode=decode), want, dtype, what=(q_lens, decode))
            on_tcgen05 = tiles and d == dv == 128 and nh <= 32 and not decode and max(q_lens) >= 8
            assert g.pool.cache.last_kernel() == (llaisys.Kernel.GATES_TC if on_tcgen05 else
                                                  llaisys.Kernel.GATES_TILES if tiles else llaisys.Kernel.GATES)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv,tiles", [SHAPES[1], SHAPES[3], SHAPES[4], SHAPES[9]])
@pytest.mark.parametrize("window", [1, 16, 17, 64, 129, 1000])
def test_gates_with_a_window(cuda_device, dtype, nkvh, nh, d, dv, tiles, window):
    g = Gates(dtype, nkvh, nh, d, dv, LENS, seed=window)
    g.pool.append([0] * len(LENS), LENS)
    for q_lens in ([1] * len(LENS), [min(n, 50) for n in LENS]):
        q = torch.randn(sum(q_lens), nh, d).to(dtype)
        close(g.run(q, q_lens, LENS, 0.2, decode=max(q_lens) == 1, window=window), g.expect(q, q_lens, LENS, 0.2, window=window), dtype)


@pytest.mark.parametrize("dtype,nkvh,nh,d,dv,tiles", [SHAPES[0], SHAPES[2], SHAPES[5], SHAPES[8]])
def test_one_key_far_away(cuda_device, dtype, nkvh, nh, d, dv, tiles):
    """Score biases silence every key but one that all queries match: outputs are that key's value times its gate and the sums over
    the talk matrix's rows, for places at page borders and tile borders, at the start and under the query itself, in prompts and
    decoded; the query just before the key sees nothing."""
    n = 400
    for place in (0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 255, n - 1):
        g = Gates(dtype, nkvh, nh, d, dv, [n], softcap=15.0, slopes=[0.01 * (h + 1) / nh for h in range(nh)], seed=place)
        g.bias = torch.full((nh,), -14.0).to(dtype)
        g.pool.k[0] *= 0.02
        direction = torch.ones(d) / d ** 0.5
        g.pool.k[0][place] = (direction * 30).to(dtype)
        g.pool.append([0], [n])
        q = (direction.expand(n, nh, d) * 1.5).to(dtype).contiguous()
        got, want = g.run(q, [n], [n], 1.0, decode=False), g.expect(q, [n], [n], 1.0)
        close(got, want, dtype, 2.0)
        assert want[place].abs().max() > 0.1 and (place == 0 or got[place - 1].abs().max() < 0.01)
        for at in {place, min(place + 1, n - 1), n - 1}:
            close(g.run(q[:1], [1], [at + 1], 1.0, decode=True)[0], want[at], dtype, 2.0, (place, at))


def test_distance_counts_from_the_query(cuda_device):
    """Under a cap, a penalty on i - j is not one on j: the steepest slope at a far position."""
    g = Gates(BF16, 2, 4, 64, 64, [2000], softcap=4.0, slopes=[1.0, 0.1, 0.01, 0.001])
    g.pool.append([0], [2000])
    q = torch.randn(40, 4, 64).to(BF16)
    close(g.run(q, [40], [2000], 0.3, decode=False), g.expect(q, [40], [2000], 0.3), BF16)


def test_small_weights_keep_their_precision(cuda_device):
    """Weights near 1e-5 over thousands of keys: the result is small, and accurate relative to itself."""
    for softcap in (0.0, 8.0):
        g = Gates(BF16, 2, 4, 64, 64, [3000], softcap=softcap, slopes=[0.0] * 4)
        g.bias = torch.full((4,), -11.5).to(BF16)
        g.pool.append([0], [3000])
        q = torch.randn(20, 4, 64).to(BF16)
        for q_lens, decode in (([20], False), ([1], True)):
            want = g.expect(q[:q_lens[0]], q_lens, [3000], 0.2)
            got = g.run(q[:q_lens[0]], q_lens, [3000], 0.2, decode=decode)
            assert (got.double() - want).abs().max() <= 0.015 * want.abs().max()


def test_blocks_cut_over_many_ctas(cuda_device):
    """Long contexts with few queries, and chunks whose blocks straddle shares; twice, so that counters are seen to be reset."""
    lens = [4000, 2500, 700, 30]
    for nkvh, nh, d in ((8, 32, 128), (2, 12, 128), (1, 16, 128), (4, 8, 64)):
        g = Gates(BF16, nkvh, nh, d, d, lens, slopes=[0.002 * (h + 1) for h in range(nh)])
        g.pool.append([0] * 4, lens)
        for q_lens in ([1, 1, 1, 1], [100, 33, 2, 30], [3, 1, 1, 7]):
            q = torch.randn(sum(q_lens), nh, d).to(BF16)
            want = g.expect(q, q_lens, lens, 0.1)
            first = g.run(q, q_lens, lens, 0.1, decode=max(q_lens) == 1)
            close(first, want, BF16)
            assert torch.equal(first, g.run(q, q_lens, lens, 0.1, decode=max(q_lens) == 1))


# ---- row norm + append ------------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("nh,nkvh,d,dv", [(4, 2, 64, 64), (3, 1, 20, 12), (5, 5, 13, 9), (32, 8, 128, 128), (1, 1, 8, 40)])
@pytest.mark.parametrize("temp", [(0.0, 1.0), (0.4, 1.0), (0.3, 100.0), (-0.2, 7.0)])
@pytest.mark.parametrize("norms", [True, False])
def test_row_norm_and_append(cuda_device, dtype, nh, nkvh, d, dv, temp, norms):
    """Biases, one root mean square over all heads of q and of k, the query factor around its steps, and k / v in their pages."""
    gen = torch.Generator().manual_seed(d)
    positions = [0, 5, 6, 7, 98, 99, 100, 198, 199, 200, 1500]
    rows, eps = len(positions), 1e-3
    cache = llaisys.PagedKVCache.with_layers(110, [(nkvh, d, dv)], dtype=LL[dtype], max_seqs=2, max_pages_per_seq=100)
    seq = cache.add_seq()
    cache.reserve(seq, 1504)
    cache.flush()
    width = (nh * d + nkvh * d + nkvh * dv + 15) // 8 * 8
    proj, bias = torch.randn(rows, width, generator=gen).to(dtype), torch.randn(width, generator=gen).to(dtype)
    qn, kn = ((1 + 0.3 * torch.randn(n, generator=gen)).to(dtype) for n in (nh * d, nkvh * d))
    q_out = torch.zeros(rows, nh, d, dtype=dtype, device="cuda")
    on = [t.cuda() for t in (proj, bias, qn, kn)]
    cache.norm_append_dev(0, stream(), proj=on[0], row_stride=width, q_at=0, k_at=nh * d, v_at=(nh + nkvh) * d, gate_at=-1,
                          q_norm=on[2] if norms else None, k_norm=on[3] if norms else None, eps=eps, gate_scale=1.0, q_out=q_out,
                          row_scale=None, seq_ids_dev=i32([seq] * rows), positions_dev=i32(positions), n_rows=rows, nh=nh, row_norm=1,
                          bias=on[1], temp_coef=temp[0], temp_every=temp[1])
    cache.check()
    x = proj.double() + bias.double()
    q, k, v = x[:, :nh * d], x[:, nh * d:(nh + nkvh) * d], x[:, (nh + nkvh) * d:(nh + nkvh) * d + nkvh * dv]
    if norms:
        q, k = oracle.rms(q, eps) * qn.double(), oracle.rms(k, eps) * kn.double()
    q = q * oracle.query_factors(positions, {"coef": temp[0], "every": temp[1]}).unsqueeze(1)
    tol = 3e-6 if dtype == F32 else 2 ** -8
    assert ((q_out.cpu().double().view(rows, -1) - q).abs() <= tol * q.abs().clamp(min=0.5)).all()
    ones = torch.ones(1, nh, d, dtype=dtype, device="cuda")
    for r, pos in enumerate(positions):  # read the row back: a window of one key; its weight is the sigmoid of its score
        out = torch.zeros(1, nh, dv, dtype=dtype, device="cuda")
        cache.gates_dev(0, out, ones, i32([seq]), None, i32([pos + 1]), n_seqs=1, total_q=1, max_q_len=1, max_kv_len=1504, nh=nh,
                        scale=0.05, stream=stream(), window=1)
        share = nh // nkvh
        gate = torch.sigmoid(k[r].view(nkvh, d).sum(-1) * 0.05).repeat_interleave(share)
        want = v[r].view(nkvh, dv).repeat_interleave(share, 0) * gate.unsqueeze(1)
        close(out[0].cpu(), want, dtype)


# ---- minGRU -----------------------------------------------------------------------------------------------------------------------


class Gru:
    def __init__(self, dtype, width, lens, *, seed=0, z_bias=-2.0, garbage=True):
        gen = torch.Generator().manual_seed(seed)
        self.dtype, self.width, self.lens = dtype, width, lens
        self.pad = (width + 7) // 8 * 8
        self.x = [torch.randn(n, 3 * self.pad, generator=gen).to(dtype) for n in lens]
        self.bz, self.bx = ((torch.randn(width, generator=gen) + b).to(dtype) for b in (z_bias, 0.0))
        self.stride = (width + 3) // 4 * 4 + 4
        self.slots = list(np.random.default_rng(seed).permutation(len(lens) + 2)[:len(lens)])
        self.state = torch.full((len(lens) + 2, self.stride), 1e3 if garbage else 0.0, device="cuda")

    def run(self, lo, hi, *, decode=False):
        """Tokens [lo[i], hi[i]) of every sequence as one batch."""
        live = [i for i in range(len(lo)) if hi[i] > lo[i]]
        proj = torch.cat([self.x[i][lo[i]:hi[i]] for i in live]).cuda()
        q_lens = [hi[i] - lo[i] for i in live]
        out = torch.full((len(proj), self.pad + 8), 7.0, dtype=self.dtype, device="cuda")
        bz, bx = self.bz.cuda(), self.bx.cuda()
        floats = llaisys.min_gru_scratch_floats(len(proj), self.width)
        scratch = torch.full((floats + 8,), 3e3, device="cuda")
        llaisys.min_gru_dev(LL[self.dtype], decode=decode, stream=stream(), proj=proj, row_stride=3 * self.pad, z_at=0, x_at=self.pad,
                            g_at=2 * self.pad, bias_z=bz, bias_x=bx, width=self.width, state=self.state, slot_stride=self.stride,
                            seq_ids_dev=i32([int(self.slots[i]) for i in live]), q_starts_dev=i32([0, *np.cumsum(q_lens).tolist()]),
                            kv_lens_dev=i32([hi[i] for i in live]), n_seqs=len(live), n_rows=len(proj), max_q_len=max(q_lens), out=out,
                            out_stride=self.pad + 8, scratch=scratch, scratch_floats=floats)
        assert torch.all(scratch[floats:] == 3e3)
        torch.cuda.synchronize()
        assert torch.all(out[:, self.width:] == 7.0)
        parts = out[:, :self.width].cpu().split(q_lens)
        return {i: p for i, p in zip(live, parts)}

    def expect(self, i):
        z, u, o = (self.x[i][:, p * self.pad:p * self.pad + self.width].double() for p in range(3))
        return oracle.min_gru(z + self.bz.double(), u + self.bx.double(), o)

    def check(self, got, what=""):
        for i in range(len(self.lens)):
            want, state = self.expect(i)
            close(got[i], want, self.dtype, what=(what, i))
            left = self.state[int(self.slots[i]), :self.width].cpu().double()
            assert (left - state).abs().max() <= 2e-5 * max(1.0, state.abs().max().item()), (what, i)


WIDTHS = [1, 7, 36, 64, 100, 2048]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", WIDTHS)
@pytest.mark.parametrize("z_bias", [-5.0, 0.0, 4.0])
def test_min_gru_whole_and_in_portions(cuda_device, dtype, width, z_bias):
    lens = [1, 2, 7, 8, 9, 255, 257, 600] if width < 2000 else [3, 300]
    for sizes in ([10 ** 6], [1], [2], [3, 2, 5], [64, 1, 17, 300]):
        g = Gru(dtype, width, lens, seed=width, z_bias=z_bias)
        if sizes == [1] and width >= 64:
            g.lens, g.x = lens[:5], g.x[:5]
        at, got, i = [0] * len(g.lens), {s: [] for s in range(len(g.lens))}, 0
        while any(a < n for a, n in zip(at, g.lens)):
            to = [min(n, a + sizes[i % len(sizes)]) for a, n in zip(at, g.lens)]
            for s, part in g.run(at, to, decode=sizes == [1]).items():
                got[s].append(part)
            at, i = to, i + 1
        g.check({s: torch.cat(p) for s, p in got.items()}, sizes)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_min_gru_long_runs_and_mixed_batches(cuda_device, dtype):
    """Thousands of tokens in many segments, beside single tokens and short runs, and a far write that lasts."""
    g = Gru(dtype, 40, [9000, 1, 2, 2049, 300, 4096], z_bias=-2.0)
    got = g.run([0] * 6, g.lens)
    g.check(got)
    for width, lens in ((10, [127, 128, 129, 255, 256, 257, 1, 385]), (3, [300, 128, 512])):
        g = Gru(dtype, width, lens, z_bias=-3.0)
        g.check(g.run([0] * len(lens), lens), lens)
    g = Gru(dtype, 12, [6000], z_bias=-14.0)  # after the first token everything is kept
    g.x[0][0, :12] = 30.0
    g.x[0][0, g.pad:g.pad + 12] = 5.0
    got = g.run([0], [6000])
    g.check(got)
    silu = oracle.silu(g.x[0][-1, 2 * g.pad:2 * g.pad + 12].double())
    assert (got[0][-1].double() / silu).abs().min() > 2.0


def test_min_gru_reused_slots(cuda_device):
    """A slot that a finished sequence left behind does not show in the next one."""
    g = Gru(F32, 24, [50, 60], garbage=False)
    g.check(g.run([0, 0], [50, 60]))
    g.slots = g.slots[::-1]
    g.check(g.run([0, 0], [50, 60]))
    h = Gru(F32, 24, [1, 1])
    h.check(h.run([0, 0], [1, 1], decode=True))


def test_min_gru_candidate_at_its_kink(cuda_device):
    """u just below, at and above zero: sigmoid(0) = 1/2 = 0 + 1/2."""
    g = Gru(F32, 5, [1])
    g.x[0][0, :5] = 40.0
    g.x[0][0, g.pad:g.pad + 5] = torch.tensor([-1e-3, 0.0, 1e-3, -90.0, 90.0])
    g.bx = torch.zeros(5)
    g.check(g.run([0], [1]))
