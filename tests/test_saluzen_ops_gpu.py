"""The mechanisms of the Saluzen layers one by one, through the C ABI, against the oracle's functions."""
import ctypes
import math

import pytest
import torch

from oracle import saluzen_oracle as O

pytestmark = pytest.mark.gpu

BF16, F32 = 0, 1
TORCH = {BF16: torch.bfloat16, F32: torch.float32}
# limits relative to the largest of the wanted values
TOL = {BF16: 2e-2, F32: 2e-5}
SSD, DELTA = 0, 1


@pytest.fixture()
def call(pkg):
    from sglang_cpp_b200 import _lib

    yield _lib.call
    st = (ctypes.c_int32 * 2)()
    torch.cuda.synchronize()
    _lib.call("b200_read_device_status", st, None)
    assert list(st) == [0, 0]


def stream():
    return torch.cuda.current_stream().cuda_stream


def gen(seed):
    return torch.Generator().manual_seed(seed)


def ints(*values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


def close(got, want, dtype, factor=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    worst = float((got - want).abs().max())
    assert worst <= factor * TOL[dtype] * max(float(want.abs().max()), 1e-6), worst


def pad_to(x, *shape):
    out = torch.zeros(shape, dtype=x.dtype)
    out[tuple(slice(0, n) for n in x.shape)] = x
    return out


def up64(n):
    return -(-n // 64) * 64


# ---- recurrences ---------------------------------------------------------------------
class Recurrence:
    """Requests of given lengths through one recurrent mixer between its projections."""

    def __init__(self, rule, exts, heads, kv_heads, d, dv, taps, dtype, groups=1, seed=0, decay=(-2.0, 1.0), bias=(-4.0, 0.0)):
        g, dt = gen(seed), TORCH[dtype]
        self.rule, self.exts, self.H, self.G, self.d, self.dv, self.taps = rule, exts, heads, kv_heads, d, dv, taps
        self.dtype, self.groups, self.eps = dtype, groups, 1e-5
        T = sum(exts)
        rand = lambda *s: torch.randn(*s, generator=g).to(dt)
        uniform = lambda n, r: r[0] + (r[1] - r[0]) * torch.rand(n, generator=g)
        self.gate, self.v, self.k, self.q = rand(T, heads, dv), rand(T, heads, dv), rand(T, kv_heads, d), rand(T, kv_heads, d)
        self.a, self.b = rand(T, heads), rand(T, heads)
        w = lambda *s: torch.randn(*s, taps, generator=g) * 1.5 / math.sqrt(taps)
        self.cv, self.ck, self.cq = w(heads, dv), w(kv_heads, d), w(kv_heads, d)
        some = 0.3 if rule == SSD else 0.0
        self.bv, self.bk, self.bq = (some * torch.randn(*s, generator=g) for s in ((heads, dv), (kv_heads, d), (kv_heads, d)))
        self.a_log, self.dt_bias = uniform(heads, decay), uniform(heads, bias)
        self.skip = torch.randn(heads, generator=g)
        self.norm = (1 + 0.3 * torch.randn(heads if rule == SSD else 1, dv, generator=g)).to(dt)
        self.dp, self.vp = up64(d), up64(dv)

    def states(self, rows):
        c = self.H * self.vp + 2 * self.G * self.dp
        return (torch.full((rows, self.H, self.dp, self.vp), 7.0, device="cuda"),
                torch.full((rows, self.taps, c), 5.0, dtype=TORCH[self.dtype], device="cuda"))

    def run(self, call, states, cached, table_idx, tokens=None, plain=0, decode=0, scale=1.0, wide=0):
        """tokens: for every request, which of its tokens to bring (a slice); the states are changed in place."""
        from sglang_cpp_b200 import _lib

        H, G, dp, vp, dt = self.H, self.G, self.dp, self.vp, TORCH[self.dtype]
        starts = [0] + torch.tensor(self.exts).cumsum(0).tolist()
        pick = [list(range(starts[i], starts[i + 1]))[tokens[i] if tokens else slice(None)] for i in range(len(self.exts))]
        rows = torch.tensor([t for p in pick for t in p])
        T, lens = len(rows), [len(p) for p in pick]
        heads = lambda x, n, to: pad_to(x[rows], T, n, to).flatten(1)
        steps = self.a[rows] if self.rule == SSD else torch.cat([self.a[rows], self.b[rows]], 1)
        joint = torch.cat([torch.full((T, 64), 9.0, dtype=dt), heads(self.gate, H, vp), heads(self.v, H, vp), heads(self.k, G, dp),
                           heads(self.q, G, dp), pad_to(steps, T, up64(steps.shape[1]))], 1).cuda()
        per_channel = lambda v, k, q: torch.cat([pad_to(v, H, vp, *v.shape[2:]).flatten(0, 1), pad_to(k, G, dp, *k.shape[2:]).flatten(0, 1),
                                                 pad_to(q, G, dp, *q.shape[2:]).flatten(0, 1)])
        conv, bias = per_channel(self.cv, self.ck, self.cq).T.contiguous().cuda(), per_channel(self.bv, self.bk, self.bq).cuda()
        f = lambda x: x.float().cuda()
        a_log, dt_bias, skip = f(self.a_log), f(self.dt_bias), f(self.skip)
        norm = pad_to(self.norm, len(self.norm), vp).flatten().cuda()
        ld = H * vp + wide
        out = torch.full((T, ld), 4.0, dtype=dt, device="cuda")
        nbytes = (ctypes.c_int64 * 4)()
        call("b200_recurrence_scratch", self.rule, T, len(lens), H, G, dp, vp, self.dtype, nbytes)
        scratch = [torch.full((max(n, 16),), 0x7f, dtype=torch.uint8, device="cuda") for n in nbytes]
        qo, idx, ca = ints(0, *torch.tensor(lens).cumsum(0).tolist()), ints(*table_idx), ints(*cached)
        esz = joint.element_size()
        a = _lib.RecurrenceArgs(
            out=out.data_ptr(), out_ld=ld, joint=joint.data_ptr() + 64 * esz, joint_ld=joint.stride(0), rule=self.rule, tokens=T,
            batch=len(lens), max_extend=max(lens), decode=decode, plain=plain, table_idx=idx.data_ptr(), cached=ca.data_ptr(),
            qo_indptr=qo.data_ptr(), state=states[0].data_ptr(), conv_state=states[1].data_ptr(), heads=H, kv_heads=G, dim=self.d,
            padded_dim=dp, value_dim=self.dv, padded_value_dim=vp, taps=self.taps, norm_groups=self.groups, conv=conv.data_ptr(),
            conv_bias=bias.data_ptr() if self.rule == SSD else None, decay_log=a_log.data_ptr(), step_bias=dt_bias.data_ptr(),
            skip=skip.data_ptr(), norm=norm.data_ptr(), eps=self.eps, out_scale=scale, mixed=scratch[0].data_ptr(),
            steps=scratch[1].data_ptr(), units=scratch[2].data_ptr(), chunks=scratch[3].data_ptr())
        call("b200_recurrence", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        if wide:
            assert float((out[:, H * vp:].float() - 4).abs().sum()) == 0
        out = out[:, :H * vp].view(T, H, vp)
        assert float(out[..., self.dv:].float().abs().sum()) == 0
        return out[..., :self.dv].cpu()

    def want(self):
        """Per request, outputs and last state."""
        H, G, d, dv = self.H, self.G, self.d, self.dv
        outs, states, at = [], [], 0
        spread = torch.arange(H) // (H // G)
        for n in self.exts:
            s = slice(at, at + n)
            at += n
            conv = lambda x, w, b: O.short_conv(x[s].double().flatten(1), w.double().flatten(0, 1), b.double().flatten()).view(n, *x.shape[1:])
            v, k, q = conv(self.v, self.cv, self.bv), conv(self.k, self.ck, self.bk)[:, spread], conv(self.q, self.cq, self.bq)[:, spread]
            step = torch.nn.functional.softplus(self.a[s].double() + self.dt_bias.double(), threshold=1e9)
            g = torch.exp(-torch.exp(self.a_log.double()) * step)
            gate = torch.nn.functional.silu(self.gate[s].double())
            if self.rule == SSD:
                y, S = O.ssd_recurrence(v, k, q, g, step)
                y = (y + self.skip.double()[:, None] * v) * gate
                y = O.rms_normalise(y.reshape(n, self.groups, -1), 1.0, self.eps).reshape(n, H, dv) * self.norm.double()
            else:
                unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
                y, S = O.delta_recurrence(unit(q) / math.sqrt(d), unit(k), v, g, torch.sigmoid(self.b[s].double()))
                y = O.rms_normalise(y, self.norm[0].double(), self.eps) * gate
            outs.append(y)
            states.append(S)
        return outs, states


# rule, heads, key heads, dim, value dim, taps, norm groups
SHAPES = [(SSD, 8, 1, 128, 64, 4, 1), (SSD, 4, 2, 64, 128, 2, 4), (SSD, 6, 3, 40, 20, 3, 5), (SSD, 3, 3, 100, 72, 7, 1),
          (DELTA, 4, 2, 128, 128, 4, 1), (DELTA, 3, 3, 64, 64, 3, 1), (DELTA, 6, 2, 24, 40, 2, 1), (DELTA, 5, 1, 100, 72, 9, 1)]
BIG = [(SSD, 2, 1, 260, 136, 3, 1), (DELTA, 2, 2, 200, 264, 4, 1), (DELTA, 1, 1, 600, 20, 1, 1), (SSD, 2, 2, 64, 600, 1, 3)]


@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 0)])
@pytest.mark.parametrize("rule, heads, kv_heads, d, dv, taps, groups", SHAPES + BIG)
def test_recurrence_of_prompts(call, dtype, plain, rule, heads, kv_heads, d, dv, taps, groups):
    x = Recurrence(rule, [1, 2, 63, 64, 65, 200, 17], heads, kv_heads, d, dv, taps, dtype, groups, d)
    states = x.states(9)
    rows = [8, 0, 3, 2, 7, 1, 5]
    got = x.run(call, states, [0] * 7, rows, plain=plain, scale=0.7, wide=64)
    outs, last = x.want()
    close(got, 0.7 * torch.cat(outs), dtype)
    for r, S in zip(rows, last):
        close(states[0][r, :, :d, :dv], S, dtype)
        assert float(states[0][r, :, d:].abs().sum()) == 0 and float(states[0][r, :, :, dv:].abs().sum()) == 0
    assert bool((states[0][4] == 7).all() and (states[0][6] == 7).all() and (states[1][4] == 5).all())   # rows of other requests


@pytest.mark.parametrize("rule", [SSD, DELTA])
@pytest.mark.parametrize("decay, bias", [((4.0, 7.0), (2.0, 9.0)), ((-9.0, -7.0), (-9.0, -6.0)), ((-9.0, 6.0), (-8.0, 5.0))])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_decays_however_steep_or_flat(call, rule, decay, bias, dtype):
    """From heads that forget at once to heads that never do, beside one another."""
    x = Recurrence(rule, [150, 70], 6, 2, 128, 64, 4, dtype, 1, 3, decay, bias)
    states = x.states(2)
    got = x.run(call, states, [0, 0], [0, 1])
    outs, last = x.want()
    close(got, torch.cat(outs), dtype, 2.0)
    for r, S in enumerate(last):
        close(states[0][r, :, :128, :64], S, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("rule, heads, kv_heads, d, dv, taps, groups", SHAPES + BIG)
@pytest.mark.parametrize("cut", [1, 2, 37, 64, 99])
def test_portions_and_decoding_carry_the_states_on(call, dtype, rule, heads, kv_heads, d, dv, taps, groups, cut):
    n = 130
    x = Recurrence(rule, [n, n], heads, kv_heads, d, dv, taps, dtype, groups, 11)
    states = x.states(3)
    parts, at = [], 0
    while at < n:
        m = min(cut, n - at)
        part = x.run(call, states, [at, at], [2, 0], [slice(at, at + m)] * 2, decode=int(m == 1 and at > 0), scale=1.5, wide=128)
        parts.append(part.view(2, m, heads, dv))
        at += m
    outs, last = x.want()
    close(torch.cat(parts, 1).reshape(2 * n, heads, dv), 1.5 * torch.cat(outs), dtype, 1.0 if dtype == BF16 else 2.0)
    for r, S in zip((2, 0), last):
        close(states[0][r, :, :d, :dv], S, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_keys_that_repeat(call, dtype):
    """The delta rule on a prompt of one key over and over, at full strength and without decay: every write replaces
    the one before it, which is where an inverse that loses digits shows."""
    n = 190
    x = Recurrence(DELTA, [n], 2, 1, 128, 64, 2, dtype, 1, 4, (-20.0, -19.0), (-9.0, -8.0))
    x.b.fill_(9.0)
    x.ck.zero_()
    x.cq.zero_()
    x.ck[..., -1] = x.cq[..., -1] = 1
    x.k[:] = x.k[0]
    x.q[:] = x.k[0]
    states = x.states(1)
    got = x.run(call, states, [0], [0])
    outs, _ = x.want()
    close(got, outs[0], dtype)


@pytest.mark.parametrize("rule", [SSD, DELTA])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_a_token_is_remembered_across_a_long_prompt(call, rule, dtype):
    """One key stands out at token 3 of a state that does not decay; it is read out 600 tokens later, from a prompt,
    from portions and from decoding."""
    n = 640
    for steps in ([n], [n - 1, 1], [100, 300, 240]):
        x = Recurrence(rule, [n], 1, 1, 64, 64, 2, dtype, 1, 4, (-20.0, -19.0), (1.0, 1.1))
        x.ck.zero_()
        x.cq.zero_()
        x.ck[..., -1] = x.cq[..., -1] = 1
        for b in (x.bk, x.bq):
            b.zero_()
        x.k[..., 5] = -30.0 if rule == SSD else 0.0     # (silu leaves nothing of it)
        x.k[3], x.q[n - 1] = -30.0, -30.0
        x.k[3, 0, 5], x.q[n - 1, 0, 5] = 8.0, 8.0
        if rule == DELTA:
            x.k[:3, 0, 5] = x.k[4:, 0, 5] = -30.0
            x.b.fill_(9.0)
        x.skip.zero_()
        states, at, got = x.states(1), 0, None
        for m in steps:
            got = x.run(call, states, [at], [0], [slice(at, at + m)], decode=int(m == 1))
            at += m
        outs, _ = x.want()
        close(got[-1], outs[0][-1], dtype)
        v = O.short_conv(x.v[:, 0].double(), x.cv[0].double(), x.bv[0].double())[3]
        gate = torch.nn.functional.silu(x.gate[-1, 0].double())
        if rule == SSD:
            want = O.rms_normalise(v * gate, x.norm[0].double(), 0.0)
        else:
            want = O.rms_normalise(v, x.norm[0].double(), 0.0) * gate
        close(got[-1, 0], want, BF16, 2.0)


# ---- attention with chunks, sinks and gates ------------------------------------------------
class Paged:
    """Requests of given lengths in paged pools whose pages are shuffled; the last `ext` positions of each are
    queries."""

    def __init__(self, lens, exts, heads, kv_heads, d, dv, page, dtype, seed=0, pad=(128, 128)):
        g = gen(seed)
        self.lens, self.exts, self.heads, self.kv_heads, self.d, self.dv = lens, exts, heads, kv_heads, d, dv
        self.page, self.dtype, (self.dp, self.vp) = page, dtype, pad
        dt = TORCH[dtype]
        self.k = [torch.randn(n, kv_heads, d, generator=g).to(dt) for n in lens]
        self.v = [torch.randn(n, kv_heads, dv, generator=g).to(dt) for n in lens]
        self.q = [(1.5 * torch.randn(n, heads, d, generator=g)).to(dt) for n in exts]
        self.gate = [torch.randn(n, heads, dv, generator=g).to(dt) for n in exts]
        self.sinks = torch.randn(heads, generator=g) * 2
        pages = sum(-(-n // page) for n in lens) + 2
        self.slots = pages * page
        perm = torch.randperm(pages, generator=g)
        self.cols = (max(lens) + page + 31) // 32 * 32
        self.table = torch.zeros(len(lens), self.cols, dtype=torch.int32)
        at = 0
        for r, n in enumerate(lens):
            m = -(-n // page)
            s = (perm[at:at + m, None] * page + torch.arange(page)).flatten()
            self.table[r, :len(s)] = s.int()
            at += m

    def attend(self, call, scale, chunk, sinks, gate, out_scale, plain=0, decode=0):
        """gate: 0 none, 1 per element, 2 per head."""
        from sglang_cpp_b200 import _lib

        H, G, dp, vp, dt = self.heads, self.kv_heads, self.dp, self.vp, TORCH[self.dtype]
        kc, vc = torch.full((self.slots, G, dp), 3.0, dtype=dt), torch.full((self.slots, G, vp), 50.0, dtype=dt)
        kc[..., self.d:], vc[..., self.dv:] = 0, 0
        for r, n in enumerate(self.lens):
            s = self.table[r, :n].long()
            kc[s, :, :self.d], vc[s, :, :self.dv] = self.k[r], self.v[r]
        T, gate_cols = sum(self.exts), H * vp if gate == 1 else 64
        rows = torch.zeros(T, H * dp + 64 + gate_cols, dtype=dt)
        rows[:, :H * dp] = pad_to(torch.cat(self.q), T, H, dp).view(T, -1)
        g = torch.cat(self.gate)
        rows[:, H * dp + 64:] = pad_to(g, T, H, vp).view(T, -1) if gate == 1 else pad_to(g[..., 0], T, 64)
        rows, kc, vc, table = rows.cuda(), kc.cuda(), vc.cuda(), self.table.cuda()
        out = torch.full((T, H * vp + 64), 9.0, dtype=dt, device="cuda")
        idx, lens, sk = ints(*range(len(self.lens))), ints(*self.lens), self.sinks.cuda()
        qo = ints(0, *torch.tensor(self.exts).cumsum(0).tolist())
        row_table = ints(*[r for r, n in enumerate(self.exts) for _ in range(n)])
        row_len = ints(*[n - e + i + 1 for n, e in zip(self.lens, self.exts) for i in range(e)])
        nbytes = max(_lib.load().b200_attention_decode_workspace_bytes(len(self.lens), H, G, 128), 16)
        ws = torch.zeros(nbytes, dtype=torch.uint8, device="cuda")
        a = _lib.WindowAttentionArgs(
            out=out.data_ptr(), q=rows.data_ptr(), q_stride=rows.stride(0), k_cache=kc.data_ptr(), v_cache=vc.data_ptr(),
            num_slots=self.slots, page_table=table.data_ptr(), page_table_stride=self.cols, table_idx=idx.data_ptr(),
            seq_lens=lens.data_ptr(), qo_indptr=qo.data_ptr(), row_table=row_table.data_ptr(), row_len=row_len.data_ptr(),
            tokens=T, batch=len(self.lens), max_extend=max(self.exts), decode=decode, plain=plain, heads=H, kv_heads=G,
            padded_dim=dp, padded_value_dim=vp, page_size=self.page, scale=scale, window=2 ** 31 - 1, keep_first=0,
            gate=rows.data_ptr() + (H * dp + 64) * rows.element_size() if gate else None, gate_stride=rows.stride(0),
            workspace=ws.data_ptr(), workspace_bytes=nbytes, chunk=chunk, sinks=sk.data_ptr() if sinks else None,
            gate_per_head=int(gate == 2), out_scale=out_scale, out_stride=out.stride(0))
        call("b200_window_attention", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        assert float((out[:, H * vp:].float() - 9).abs().sum()) == 0
        out = out[:, :H * vp].view(T, H, vp)
        assert float(out[..., self.dv:].float().abs().sum()) == 0
        return out[..., :self.dv].cpu()

    def want(self, scale, chunk, sinks, gate, out_scale):
        out = []
        for r, (n, e) in enumerate(zip(self.lens, self.exts)):
            seen = O.visible(n, chunk or None)[n - e:]
            rep = self.heads // self.kv_heads
            k, v = (x[r].double().repeat_interleave(rep, 1) for x in (self.k, self.v))
            s = (torch.einsum("ihd,jhd->hij", self.q[r].double(), k) * scale).masked_fill(~seen, float("-inf"))
            p = torch.stack([O.sink_softmax(s[h], self.sinks[h].double() if sinks else None) for h in range(self.heads)])
            o = torch.einsum("hij,jhd->ihd", p, v) * out_scale
            g = torch.sigmoid(self.gate[r].double())
            out.append(o if gate == 0 else o * g if gate == 1 else o * g[..., :1])
        return torch.cat(out)


CHUNKS = [0, 1, 5, 64, 100, 128, 129, 1000]


@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("heads, kv_heads, page, sinks, gate", [(8, 2, 64, True, 2), (4, 4, 1, True, 1), (16, 1, 16, False, 2), (8, 8, 256, True, 0)])
def test_chunked_attention_in_prompts(call, chunk, heads, kv_heads, page, sinks, gate):
    p = Paged([300, 1, 65, 700, 130, 128], [300, 1, 2, 90, 66, 127], heads, kv_heads, 128, 128, page, BF16, chunk)
    close(p.attend(call, 0.09, chunk, sinks, gate, 0.8), p.want(0.09, chunk, sinks, gate, 0.8), BF16)


@pytest.mark.parametrize("chunk", CHUNKS)
@pytest.mark.parametrize("heads, kv_heads, page, sinks, gate", [(8, 2, 64, True, 2), (5, 1, 16, True, 1), (8, 8, 1, False, 2), (12, 4, 64, True, 0)])
def test_chunked_attention_of_decoded_tokens(call, chunk, heads, kv_heads, page, sinks, gate):
    lens = [1, 2, 63, 64, 65, 128, 129, 700, 1500, 333, 201]
    p = Paged(lens, [1] * len(lens), heads, kv_heads, 128, 128, page, BF16, chunk)
    close(p.attend(call, 0.09, chunk, sinks, gate, -1.2, decode=1), p.want(0.09, chunk, sinks, gate, -1.2), BF16)


def test_decoding_one_long_request_and_many_short_ones(call):
    for lens in ([30000], [int(n) for n in torch.randint(1, 90, (300,), generator=gen(0))]):
        p = Paged(lens, [1] * len(lens), 8, 2, 128, 128, 64, BF16, 3)
        for chunk in (0, 20000, 50):
            close(p.attend(call, 0.09, chunk, True, 2, 1.0, decode=1), p.want(0.09, chunk, True, 2, 1.0), BF16)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads, kv_heads, d, dv, pad", [(6, 2, 40, 56, (128, 128)), (3, 3, 144, 200, (192, 256)), (7, 7, 8, 16, (64, 64))])
@pytest.mark.parametrize("chunk, gate", [(33, 2), (1, 1), (150, 0), (0, 2)])
def test_attention_plain_kernel(call, dtype, heads, kv_heads, d, dv, pad, chunk, gate):
    p = Paged([1, 190, 400, 7], [1, 150, 3, 2], heads, kv_heads, d, dv, 16, dtype, 5, pad)
    for sinks in (False, True):
        close(p.attend(call, 0.2, chunk, sinks, gate, 1.5, plain=1), p.want(0.2, chunk, sinks, gate, 1.5), dtype)


@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("plain", [0, 1])
@pytest.mark.parametrize("chunk", [64, 100, 128, 129, 400, 401])
def test_a_key_that_stands_out_at_a_chunks_edges(call, decode, plain, chunk):
    """Keys on both sides of the edge before the query, one at a time, carry a huge score: the output is that key's
    value, or shows nothing of it."""
    n = 401
    edge = (n - 1) // chunk * chunk
    spots = sorted({s for s in (0, edge - 1, edge, edge + 1, n - 1) if 0 <= s < n})
    p = Paged([n] * len(spots), [1] * len(spots), 4, 1, 128, 128, 64, BF16, 1)
    p.sinks.fill_(-3.0)
    for r, s in enumerate(spots):
        p.q[r].zero_()
        p.q[r][:, :, 0] = 8.0
        p.k[r][:, :, 0] = 0
        p.k[r][s, :, 0] = 8.0
    got, want = p.attend(call, 0.5, chunk, True, 0, 1.0, plain, decode), p.want(0.5, chunk, True, 0, 1.0)
    close(got, want, BF16)
    for r, s in enumerate(spots):
        same = float((got[r].float() - p.v[r][s].float()).abs().max()) < 0.05
        assert same == (s >= edge), s


@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 1)])
@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("sink", [-40.0, 0.0, 3.0, 30.0])
def test_sinks_from_nothing_to_everything(call, dtype, plain, decode, sink):
    """Scores of 0 against sinks that take none of the weight, a share that the number of keys decides, or all."""
    lens = [1, 5, 130, 700]
    p = Paged(lens, [1] * 4, 4, 2, 128, 128, 16, dtype, 2)
    p.sinks.fill_(sink)
    for r in range(4):
        p.q[r].zero_()
    got = p.attend(call, 0.3, 0, True, 0, 1.0, plain, decode)
    want = torch.stack([p.v[r].double().sum(0).repeat_interleave(2, 0) / (n + math.exp(sink)) for r, n in enumerate(lens)])
    close(got, want, dtype)


# ---- latents with a rotated part ---------------------------------------------------------
@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 1)])
@pytest.mark.parametrize("heads, width, out_width", [(16, 640, 512), (40, 384, 256), (5, 256, 128), (64, 640, 128), (3, 512, 512)])
@pytest.mark.parametrize("page", [1, 64])
def test_latent_attention_averages_a_part(call, dtype, plain, heads, width, out_width, page):
    from sglang_cpp_b200 import _lib

    g, dt = gen(width + heads), TORCH[dtype]
    lens = [1, 700, 64, 65, 130, 333]
    pages = sum(-(-n // page) for n in lens) + 1
    cache = torch.randn(pages * page, width, generator=g).to(dt)
    q = (1.5 * torch.randn(len(lens), heads, width, generator=g)).to(dt)
    perm, at, cols = torch.randperm(pages, generator=g), 0, 1024
    table = torch.zeros(len(lens), cols, dtype=torch.int32)
    for r, n in enumerate(lens):
        m = -(-n // page)
        s = (perm[at:at + m, None] * page + torch.arange(page)).flatten()
        table[r, :len(s)] = s.int()
        at += m
    scale = 0.5 / math.sqrt(width)
    want = []
    for r, n in enumerate(lens):
        c = cache[table[r, :n].long()].double()
        want.append(torch.softmax(q[r].double() @ c.T * scale, -1) @ c[:, :out_width])
    out = torch.zeros(len(lens), heads, out_width, dtype=dt, device="cuda")
    nbytes = _lib.load().b200_latent_attention_workspace_bytes(len(lens), heads, width)
    ws = torch.zeros(nbytes, dtype=torch.uint8, device="cuda")
    cc, qc, tc, rt, rl = cache.cuda(), q.cuda(), table.cuda(), ints(*range(len(lens))), ints(*lens)
    call("b200_latent_attention_part", out.data_ptr(), qc.data_ptr(), cc.data_ptr(), len(cache), tc.data_ptr(), cols, rt.data_ptr(),
         rl.data_ptr(), len(lens), heads, width, out_width, page, scale, dtype, plain, ws.data_ptr(), nbytes, stream())
    torch.cuda.synchronize()
    close(out, torch.stack(want), dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("dims", [2, 12, 30, 64, 128])
def test_rotation_in_neighbouring_pairs(call, dtype, dims):
    T, H, ld = 37, 5, 128
    x = torch.randn(T, H, ld, generator=gen(dims)).to(TORCH[dtype])
    rot = {"base": 777.0, "dims": dims, "scaling": {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 99}}
    pos = torch.randint(0, 2000, (T,), generator=gen(1))
    angle = torch.arange(2000, dtype=torch.float64)[:, None] * O.frequencies(rot)
    cos, sin, y, p = angle.cos().float().cuda(), angle.sin().float().cuda(), x.cuda(), pos.int().cuda()
    call("b200_rotate_pairs", y.data_ptr(), T, H, ld, dims, cos.data_ptr(), sin.data_ptr(), p.data_ptr(), 2000, dtype, stream())
    torch.cuda.synchronize()
    close(y, O.rotate_neighbours(x.double(), pos, rot), dtype)


# ---- residual stream ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [40, 192, 1000, 9000])
@pytest.mark.parametrize("normed, last", [(1, 1), (0, 0), (1, 0), (0, 1)])
def test_residual_pair_norm(call, dtype, width, normed, last):
    T, padded, eps = 7, up64(width), 1e-5
    g, dt = gen(width), TORCH[dtype]
    rand = lambda rows, gain=1.0: pad_to((gain * torch.randn(rows, width, generator=g)).to(dt), rows, padded)
    res = pad_to(torch.randn(T, width, generator=g), T, padded)
    a, b = rand(T, 3.0), rand(T, 0.2)
    wa, wb, add, out_w = (rand(1)[0] for _ in range(4))
    n = lambda x, w: O.rms_normalise(x[..., :width].double(), w[:width].double(), eps)
    y = 0.5 * (n(a, wa) + n(b, wb))
    want_res = res[:, :width].double() + (n(y, add) if normed else y)
    want = n(want_res, out_w) if last else want_res
    r, out = res.cuda(), torch.zeros(T, padded, dtype=dt, device="cuda")
    dev = [x.cuda() for x in (a, b, wa, wb, add, out_w)]
    p = [x.data_ptr() for x in dev]
    call("b200_residual_pair_norm", out.data_ptr(), r.data_ptr(), p[0], p[1], p[2], p[3], 0.5, p[4] if normed else None,
         p[5] if last else None, T, width, padded, eps, dtype, stream())
    torch.cuda.synchronize()
    close(r[:, :width], want_res, F32)
    close(out[:, :width], want, dtype)
    assert float(out[:, width:].float().abs().sum()) == 0 and float(r[:, width:].abs().sum()) == 0
