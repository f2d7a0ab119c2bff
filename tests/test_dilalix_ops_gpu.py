"""The mechanisms of the Dilalix layers one by one, through the C ABI, against the oracle's functions."""
import ctypes
import math

import pytest
import torch

from oracle import dilalix_oracle as O

pytestmark = pytest.mark.gpu

BF16, F32 = 0, 1
TORCH = {BF16: torch.bfloat16, F32: torch.float32}
# limits relative to the spread of the wanted values
TOL = {BF16: 2e-2, F32: 2e-5}


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


# ---- attention through a window --------------------------------------------------------
class Paged:
    """Requests of given lengths in paged pools whose pages are shuffled; the last `ext` positions of each are
    queries."""

    def __init__(self, lens, exts, heads, kv_heads, d, dv, page, dtype, seed=0, pad=(128, 128)):
        g = gen(seed)
        self.lens, self.exts, self.heads, self.kv_heads, self.d, self.dv = lens, exts, heads, kv_heads, d, dv
        self.page, self.dtype, (self.dp, self.vp) = page, dtype, pad
        self.k = [torch.randn(n, kv_heads, d, generator=g).to(TORCH[dtype]) for n in lens]
        self.v = [torch.randn(n, kv_heads, dv, generator=g).to(TORCH[dtype]) for n in lens]
        self.q = [1.5 * torch.randn(n, heads, d, generator=g) for n in exts]
        self.q = [q.to(TORCH[dtype]) for q in self.q]
        self.gate = [torch.randn(n, heads, dv, generator=g).to(TORCH[dtype]) for n in exts]
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

    def attend(self, call, scale, window, keep_first, gated=True, plain=0, decode=0):
        from sglang_cpp_b200 import _lib

        H, G, dp, vp, dt = self.heads, self.kv_heads, self.dp, self.vp, TORCH[self.dtype]
        kc, vc = torch.full((self.slots, G, dp), 3.0, dtype=dt), torch.full((self.slots, G, vp), 50.0, dtype=dt)
        kc[..., self.d:], vc[..., self.dv:] = 0, 0
        for r, n in enumerate(self.lens):
            s = self.table[r, :n].long()
            kc[s, :, :self.d], vc[s, :, :self.dv] = self.k[r], self.v[r]
        T = sum(self.exts)
        # queries and gates in rows of a wider buffer, as the joint projection leaves them
        rows = torch.zeros(T, H * dp + 64 + H * vp, dtype=dt)
        rows[:, :H * dp] = pad_to(torch.cat(self.q), T, H, dp).view(T, -1)
        rows[:, H * dp + 64:] = pad_to(torch.cat(self.gate), T, H, vp).view(T, -1)
        rows, kc, vc, table = rows.cuda(), kc.cuda(), vc.cuda(), self.table.cuda()
        out = torch.full((T, H, vp), 9.0, dtype=dt, device="cuda")
        idx, lens = ints(*range(len(self.lens))), ints(*self.lens)
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
            padded_dim=dp, padded_value_dim=vp, page_size=self.page, scale=scale, window=window, keep_first=keep_first,
            gate=rows.data_ptr() + (H * dp + 64) * rows.element_size() if gated else None, gate_stride=rows.stride(0),
            workspace=ws.data_ptr(), workspace_bytes=nbytes)
        call("b200_window_attention", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        assert float(out[..., self.dv:].float().abs().sum()) == 0
        return out[..., :self.dv].cpu()

    def want(self, scale, window, keep_first, gated=True):
        out = []
        for r, (n, e) in enumerate(zip(self.lens, self.exts)):
            seen = O.visible(n, window, keep_first)[n - e:]
            rep = self.heads // self.kv_heads
            k, v = (x[r].double().repeat_interleave(rep, 1) for x in (self.k, self.v))
            s = torch.einsum("ihd,jhd->hij", self.q[r].double(), k) * scale
            o = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), -1), v)
            out.append(o * torch.sigmoid(self.gate[r].double()) if gated else o)
        return torch.cat(out)


WINDOWS = [(1, 0), (5, 2), (64, 4), (128, 0), (129, 130), (200, 1), (1000, 3), (2 ** 31 - 1, 0), (7, 300)]


@pytest.mark.parametrize("window, keep", WINDOWS)
@pytest.mark.parametrize("heads, kv_heads, page", [(8, 2, 64), (4, 4, 1), (16, 1, 16), (8, 8, 256)])
def test_window_attention_in_prompts(call, window, keep, heads, kv_heads, page):
    p = Paged([300, 1, 65, 700, 130, 128], [300, 1, 2, 90, 66, 127], heads, kv_heads, 128, 128, page, BF16, window + keep)
    close(p.attend(call, 0.09, window, keep), p.want(0.09, window, keep), BF16)


@pytest.mark.parametrize("window, keep", WINDOWS)
@pytest.mark.parametrize("heads, kv_heads, page", [(8, 2, 64), (5, 1, 16), (8, 8, 1), (12, 4, 64)])
def test_window_attention_of_decoded_tokens(call, window, keep, heads, kv_heads, page):
    lens = [1, 2, 63, 64, 65, 128, 129, 700, 1500, 333, 201]
    p = Paged(lens, [1] * len(lens), heads, kv_heads, 128, 128, page, BF16, window + keep)
    close(p.attend(call, 0.09, window, keep, decode=1), p.want(0.09, window, keep), BF16)


def test_decoding_one_long_request_and_many_short_ones(call):
    for lens in ([30000], [int(n) for n in torch.randint(1, 90, (300,), generator=gen(0))]):
        p = Paged(lens, [1] * len(lens), 8, 2, 128, 128, 64, BF16, 3)
        for window, keep in ((20000, 4), (50, 4)):
            close(p.attend(call, 0.09, window, keep, decode=1), p.want(0.09, window, keep), BF16)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads, kv_heads, d, dv, pad", [(6, 2, 40, 56, (128, 128)), (3, 3, 144, 200, (192, 256)),
                                                         (2, 1, 64, 600, (64, 640)), (7, 7, 8, 16, (64, 64))])
@pytest.mark.parametrize("window, keep", [(33, 3), (1, 0), (130, 200), (500, 0)])
def test_window_attention_plain_kernel(call, dtype, heads, kv_heads, d, dv, pad, window, keep):
    p = Paged([1, 190, 400, 7], [1, 150, 3, 2], heads, kv_heads, d, dv, 16, dtype, 5, pad)
    close(p.attend(call, 0.2, window, keep, plain=1), p.want(0.2, window, keep), dtype)
    close(p.attend(call, 0.2, window, keep, gated=False, plain=1), p.want(0.2, window, keep, False), dtype)


@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("plain", [0, 1])
@pytest.mark.parametrize("window, keep", [(64, 4), (128, 128), (100, 0), (129, 1), (31, 5)])
def test_a_key_that_stands_out_at_every_edge(call, decode, plain, window, keep):
    """Keys just inside and outside the window and the kept ones, one at a time, carry a huge score: the output
    is that key's value, or shows nothing of it."""
    n = 401
    spots = sorted({s for s in (0, keep - 1, keep, keep + 1, n - 1 - window, n - window, n - window + 1, n - 1) if 0 <= s < n})
    p = Paged([n] * len(spots), [1] * len(spots), 4, 1, 128, 128, 64, BF16, 1)
    for r, s in enumerate(spots):
        p.q[r].zero_()
        p.q[r][:, :, 0] = 8.0
        p.k[r][:, :, 0] = 0
        p.k[r][s, :, 0] = 8.0
    got, want = p.attend(call, 0.5, window, keep, False, plain, decode), p.want(0.5, window, keep, False)
    close(got, want, BF16)
    for r, s in enumerate(spots):
        same = float((got[r].float() - p.v[r][s].float()).abs().max()) < 0.05
        assert same == (n - 1 - s < window or s < keep), s


# ---- norms, rotation, value mixing, store ------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T", [7, 900])
@pytest.mark.parametrize("heads, kv_heads, d, dv, dims, pad", [(4, 2, 128, 128, 128, (128, 128)), (3, 1, 48, 80, 20, (128, 128)),
                                                               (2, 2, 128, 100, 2, (128, 128)), (6, 2, 96, 128, 64, (128, 128)),
                                                               (2, 1, 160, 192, 160, (192, 192)), (4, 4, 120, 128, 0, (128, 128))])
@pytest.mark.parametrize("mix", [0, 1, 2])
def test_head_prepare(call, dtype, T, heads, kv_heads, d, dv, dims, pad, mix):
    from sglang_cpp_b200 import _lib

    g, dt, (dp, vp), eps, base = gen(T + d), TORCH[dtype], pad, 1e-5, 5000.0
    rand = lambda *s: torch.randn(*s, generator=g).to(dt)
    q, k, v, first = rand(T, heads, d), rand(T, kv_heads, d), rand(T, kv_heads, dv), rand(T, kv_heads, dv)
    qw, kw = (1 + 0.3 * torch.randn(d, generator=g)).to(dt), (1 + 0.3 * torch.randn(d, generator=g)).to(dt)
    tail = 64
    joint = torch.cat([pad_to(q, T, heads, dp).flatten(1), pad_to(k, T, kv_heads, dp).flatten(1),
                       pad_to(v, T, kv_heads, vp).flatten(1), torch.full((T, tail), 2.0, dtype=dt)], 1).cuda()
    pos = torch.randint(0, 3000, (T,), generator=g)
    slots = torch.randperm(T + 50, generator=g)[:T]
    half = dims // 2
    angle = pos.max() + 1
    f = base ** (-2.0 * torch.arange(half, dtype=torch.float64) / max(dims, 1))
    table = torch.arange(int(angle), dtype=torch.float64)[:, None] * f
    cos, sin = table.cos().float().cuda().contiguous(), table.sin().float().cuda().contiguous()
    kc, vc = torch.zeros(T + 50, kv_heads, dp, dtype=dt, device="cuda"), torch.zeros(T + 50, kv_heads, vp, dtype=dt, device="cuda")
    fv = pad_to(first, T, kv_heads, vp).cuda()
    lam, qn, kn = torch.tensor([0.3], device="cuda"), pad_to(qw, dp).cuda(), pad_to(kw, dp).cuda()
    p32, s32 = pos.int().cuda(), slots.int().cuda()
    any_ptr = lam.data_ptr()
    a = _lib.HeadPrepareArgs(
        joint=joint.data_ptr(), joint_ld=joint.stride(0), tokens=T, heads=heads, kv_heads=kv_heads, dim=d, padded_dim=dp,
        padded_value_dim=vp, q_norm=qn.data_ptr(), k_norm=kn.data_ptr(), eps=eps, rotary_dim=dims, max_pos=int(angle),
        cos_table=cos.data_ptr() or any_ptr, sin_table=sin.data_ptr() or any_ptr, positions=p32.data_ptr(),
        out_loc=s32.data_ptr(), k_cache=kc.data_ptr(), v_cache=vc.data_ptr(), num_slots=T + 50, mix=mix,
        lambda_=lam.data_ptr(), first_values=fv.data_ptr())
    call("b200_head_prepare", ctypes.byref(a), dtype, stream())
    torch.cuda.synchronize()

    def turned(x, w):
        x = O.rms_normalise(x.double(), w.double(), eps)
        return O.rotate_half(x, pos, base, dims) if dims else x

    close(joint[:, :heads * dp].view(T, heads, dp)[..., :d], turned(q, qw), dtype)
    close(kc[s32.long()][..., :d], turned(k, kw), dtype)
    want = v.double() if mix < 2 else 0.7 * v.double() + 0.3 * first.double()
    close(vc[s32.long()][..., :dv], want, dtype)
    close(fv[..., :dv], v if mix == 1 else first, dtype)
    assert float(joint[:, -tail:].float().min()) == 2.0 and float(kc[..., d:].float().abs().sum()) == 0


# ---- gated linear attention --------------------------------------------------------------
class Linear:
    def __init__(self, exts, heads, d, dv, rank, tau, dtype, seed=0, bias=(-6.0, 8.0)):
        g = gen(seed)
        self.exts, self.heads, self.d, self.dv, self.rank, self.tau, self.dtype = exts, heads, d, dv, rank, tau, dtype
        dt = TORCH[dtype]
        rand = lambda *s: torch.randn(*s, generator=g).to(dt)
        T = sum(exts)
        self.q, self.k, self.v, self.gate, self.low = rand(T, heads, d), rand(T, heads, d), rand(T, heads, dv), rand(T, heads, dv), rand(T, rank)
        self.up = (1.5 / math.sqrt(rank) * torch.randn(heads * d, rank, generator=g)).to(dt)
        self.bias = bias[0] + (bias[1] - bias[0]) * torch.rand(heads * d, generator=g)
        self.norm = (1 + 0.3 * torch.randn(dv, generator=g)).to(dt)
        self.eps = 1e-5

    def run(self, call, state, cached, table_idx, tokens=None, plain=0, decode=0):
        """tokens: for every request, which of its tokens to bring (a slice); the state is changed in place."""
        from sglang_cpp_b200 import _lib

        H, d, dv = self.heads, self.d, self.dv
        dp, vp, ld_up = -(-d // 64) * 64, -(-dv // 64) * 64, -(-self.rank // 16) * 16
        rp = -(-self.rank // 64) * 64
        starts = [0] + torch.tensor(self.exts).cumsum(0).tolist()
        pick = [list(range(starts[i], starts[i + 1]))[tokens[i] if tokens else slice(None)] for i in range(len(self.exts))]
        rows = torch.tensor([t for p in pick for t in p])
        T = len(rows)
        joint = torch.cat([pad_to(self.q[rows], T, H, dp).flatten(1), pad_to(self.k[rows], T, H, dp).flatten(1),
                           pad_to(self.v[rows], T, H, vp).flatten(1), pad_to(self.gate[rows], T, H, vp).flatten(1),
                           pad_to(self.low[rows], T, rp)], 1).cuda()
        up = pad_to(self.up.view(H, d, self.rank), H, dp, ld_up).cuda()
        bias, norm = pad_to(self.bias.view(H, d), H, dp).cuda(), pad_to(self.norm, vp).cuda()
        out = torch.full((T, H, vp), 9.0, dtype=TORCH[self.dtype], device="cuda")
        qo = ints(0, *torch.tensor([len(p) for p in pick]).cumsum(0).tolist())
        idx, ca = ints(*table_idx), ints(*cached)
        a = _lib.LinearAttentionArgs(
            out=out.data_ptr(), joint=joint.data_ptr(), joint_ld=joint.stride(0), tokens=T, batch=len(self.exts), decode=decode,
            plain=plain, table_idx=idx.data_ptr(), cached=ca.data_ptr(), qo_indptr=qo.data_ptr(), state=state.data_ptr(),
            heads=H, dim=d, padded_dim=dp, value_dim=dv, padded_value_dim=vp, rank=self.rank, up_ld=ld_up, up=up.data_ptr(),
            bias=bias.data_ptr(), norm=norm.data_ptr(), tau=self.tau, eps=self.eps, q_scale=d ** -0.5)
        call("b200_linear_attention", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        assert float(out[..., dv:].float().abs().sum()) == 0
        return out[..., :dv].cpu()

    def new_state(self, rows):
        return torch.full((rows, self.heads, -(-self.d // 64) * 64, -(-self.dv // 64) * 64), 7.0, device="cuda")

    def want(self):
        """Per request, outputs and last state."""
        z = (self.low.double() @ self.up.double().T + self.bias.double()).view(-1, self.heads, self.d)
        ld = torch.nn.functional.logsigmoid(z) / self.tau
        outs, states, at = [], [], 0
        for n in self.exts:
            s = slice(at, at + n)
            o, S = O.linear_recurrence(self.q[s].double() * self.d ** -0.5, self.k[s].double(), self.v[s].double(), ld[s])
            outs.append(O.rms_normalise(o, self.norm.double(), self.eps) * torch.nn.functional.silu(self.gate[s].double()))
            states.append(S)
            at += n
        return outs, states


SHAPES = [(3, 128, 128, 16), (2, 48, 32, 16), (1, 64, 192, 40), (4, 100, 72, 10), (2, 24, 64, 64)]


@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 0)])
@pytest.mark.parametrize("heads, d, dv, rank", SHAPES + [(2, 144, 136, 70), (1, 200, 264, 16)])
@pytest.mark.parametrize("tau", [16.0, 1.0])
def test_linear_attention_of_prompts(call, dtype, plain, heads, d, dv, rank, tau):
    x = Linear([1, 2, 63, 64, 65, 200, 17], heads, d, dv, rank, tau, dtype, d)
    state = x.new_state(9)
    rows = [8, 0, 3, 2, 7, 1, 5]
    got = x.run(call, state, [0] * 7, rows, plain=plain)
    outs, states = x.want()
    close(got, torch.cat(outs), dtype)
    for r, S in zip(rows, states):
        close(state[r, :, :d, :dv], S, F32 if dtype == F32 else BF16, 1.0 if dtype == F32 else 0.02)
        assert float(state[r, :, d:].abs().sum()) == 0 and float(state[r, :, :, dv:].abs().sum()) == 0
    assert bool((state[4] == 7).all() and (state[6] == 7).all())     # rows of other requests


@pytest.mark.parametrize("bias", [(-300.0, 2.0), (-60.0, -40.0), (30.0, 40.0), (-2000.0, -1000.0), (-12.0, -8.0)])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_decays_however_steep_or_flat(call, bias, dtype):
    """From channels that forget at once to channels that never do, beside one another."""
    x = Linear([150, 70], 2, 128, 64, 16, 1.0, dtype, 3, bias)
    state = x.new_state(2)
    got = x.run(call, state, [0, 0], [0, 1])
    outs, states = x.want()
    close(got, torch.cat(outs), dtype)
    for r, S in enumerate(states):
        close(state[r, :, :, :64], S, F32 if dtype == F32 else BF16, 1.0 if dtype == F32 else 0.02)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads, d, dv, rank", SHAPES + [(2, 144, 136, 70)])
@pytest.mark.parametrize("cut", [1, 2, 37, 64, 99])
def test_portions_and_decoding_carry_the_state_on(call, dtype, heads, d, dv, rank, cut):
    n = 130
    x = Linear([n, n], heads, d, dv, rank, 8.0, dtype, 11)
    state = x.new_state(3)
    parts, at = [], 0
    while at < n:
        m = min(cut, n - at)
        decode = int(m == 1 and at > 0)
        part = x.run(call, state, [at, at], [2, 0], [slice(at, at + m)] * 2, decode=decode)
        parts.append(part.view(2, m, heads, dv))
        at += m
    outs, states = x.want()
    close(torch.cat(parts, 1).reshape(2 * n, heads, dv), torch.cat(outs), dtype)
    for r, S in zip((2, 0), states):
        close(state[r, :, :d, :dv], S, F32 if dtype == F32 else BF16, 2.0 if dtype == F32 else 0.05)


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_a_token_is_remembered_across_a_long_prompt(call, dtype):
    """One key stands out at token 3 in channels that do not decay; it is read out 600 tokens later, from a prompt and
    from decoding."""
    n = 640
    for steps in ([n], [n - 1, 1], [100, 300, 240]):
        x = Linear([n], 1, 128, 64, 16, 16.0, dtype, 4, (20.0, 25.0))
        x.low.zero_()
        x.k *= 0.02
        x.k[3, 0, :] = 0
        x.k[3, 0, 5] = 60.0
        x.q[n - 1, 0, :] = 0
        x.q[n - 1, 0, 5] = 8.0
        state, at, got = x.new_state(1), 0, None
        for m in steps:
            got = x.run(call, state, [at], [0], [slice(at, at + m)], decode=int(m == 1))
            at += m
        want = O.rms_normalise(x.v[3, 0].double(), x.norm.double(), 0.0) * torch.nn.functional.silu(x.gate[-1, 0].double())
        close(got[-1, 0], want, BF16, 2.0)


# ---- residual stream ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [40, 192, 1000, 9000])
@pytest.mark.parametrize("top, shared, init, normed, last", [(0, 0, 0, 1, 0), (1, 0, 1, 0, 0), (3, 1, 0, 1, 0), (20, 1, 0, 1, 1),
                                                             (0, 0, 0, 1, 1), (4, 0, 0, 0, 1)])
def test_residual_post_norm(call, dtype, width, top, shared, init, normed, last):
    T, padded, eps = 7, -(-width // 64) * 64, 1e-5
    g, dt = gen(width + top), TORCH[dtype]
    rand = lambda rows: pad_to(torch.randn(rows, width, generator=g).to(dt), rows, padded)
    res = pad_to(torch.randn(T, width, generator=g), T, padded)
    src, src2 = rand(50 if top else T), rand(T)
    rows = torch.randint(0, 50, (T, max(top, 1)), generator=g).int()
    weights = torch.rand(T, max(top, 1), generator=g)
    aw, ow = rand(1)[0], rand(1)[0]
    add = src.double() if not top else (src.double()[rows.long()] * weights.double()[..., None]).sum(1)
    add = add + src2.double() if shared else add
    if normed:
        add[:, :width] = O.rms_normalise(add[:, :width], aw[:width].double(), eps)
    want_res = add if init else res.double() + add
    want = want_res.clone()
    if last:
        want[:, :width] = O.rms_normalise(want[:, :width], ow[:width].double(), eps)
    out, r, s, s2, wa, wo = torch.zeros(T, padded, dtype=dt).cuda(), res.cuda(), src.cuda(), src2.cuda(), aw.cuda(), ow.cuda()
    ids, ws = rows.cuda(), weights.cuda()
    call("b200_residual_post_norm", out.data_ptr(), r.data_ptr(), s.data_ptr(), ids.data_ptr() if top else None,
         ws.data_ptr() if top else None, max(top, 1), len(src), s2.data_ptr() if shared else None, init,
         wa.data_ptr() if normed else None, wo.data_ptr() if last else None, T, width, padded, eps, dtype, stream())
    torch.cuda.synchronize()
    close(r, want_res, F32)
    close(out, want, dtype)
    assert float(out[:, width:].float().abs().sum()) == 0 and float(r[:, width:].abs().sum()) == 0


# ---- routing -------------------------------------------------------------------------------
@pytest.mark.parametrize("tokens", [1, 9, 1500])
@pytest.mark.parametrize("experts, top, groups, keep", [(1, 1, 1, 1), (16, 2, 4, 3), (12, 3, 4, 1), (8, 3, 8, 3), (64, 8, 8, 4),
                                                        (300, 20, 5, 2), (7, 7, 1, 1), (2000, 4, 1000, 30)])
def test_scored_routing(call, tokens, experts, top, groups, keep):
    g = gen(experts + tokens)
    ld = -(-experts // 64) * 64
    logits = pad_to(2 * torch.randn(tokens, experts, generator=g), tokens, ld).cuda()
    x = torch.randn(tokens, 64, generator=g).bfloat16().cuda()
    i32 = dict(dtype=torch.int32, device="cuda")
    ids, rows = torch.full((tokens, top), -1, **i32), torch.full((tokens, top), -1, **i32)
    weights, counts, off = torch.zeros(tokens, top, device="cuda"), torch.zeros(2 * experts, **i32), torch.zeros(experts + 1, **i32)
    xp = torch.zeros(tokens * top, 64, dtype=torch.bfloat16, device="cuda")
    call("b200_score_route", ids.data_ptr(), weights.data_ptr(), rows.data_ptr(), counts.data_ptr(), off.data_ptr(), xp.data_ptr(),
         x.data_ptr(), 128, logits.data_ptr(), ld, tokens, experts, top, groups, keep, 1.7, 0, 0, None, stream())
    torch.cuda.synchronize()
    want_ids, want_w = O.choose_experts(torch.sigmoid(logits[:, :experts].cpu().double()), top, groups, keep, 1.7)
    order, want_order = ids.cpu().long().sort(1), want_ids.sort(1)
    assert torch.equal(order.values, want_order.values)
    torch.testing.assert_close(weights.cpu().gather(1, order.indices).double(), want_w.gather(1, want_order.indices), rtol=1e-5, atol=1e-6)
    n = torch.bincount(want_ids.flatten(), minlength=experts)
    assert torch.equal(counts[:experts].cpu().long(), n)
    assert torch.equal(off.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), n.cumsum(0)]))
    r = rows.cpu().long()
    assert torch.equal(r.flatten().sort().values, torch.arange(tokens * top))
    chosen = ids.cpu().long()
    assert bool(((r >= off.cpu().long()[chosen]) & (r < off.cpu().long()[chosen + 1])).all())
    assert torch.equal(xp.cpu()[r], x.cpu()[:, None].expand(-1, top, -1))


# ---- projections ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("M", [5, 128, 400])
@pytest.mark.parametrize("N, K", [(64, 128), (1024, 2048), (320, 64)])
def test_activations_behind_a_projection(call, dtype, M, N, K):
    dt = TORCH[dtype]
    x = torch.randn(M, K, generator=gen(M)).to(dt).cuda()
    w = (torch.randn(N, K, generator=gen(N)) * 1.5 / K ** 0.5).to(dt).cuda()
    full = x.double() @ w.double().T
    g, u = torch.clamp(full[:, :N // 2], max=0.9), torch.clamp(full[:, N // 2:], -0.9, 0.9)
    wants = {5: torch.nn.functional.gelu(full), 6: g * torch.sigmoid(1.702 * g) * (u + 1), 7: full}
    for epi, want in wants.items():
        y = torch.zeros(want.shape, device="cuda", dtype=torch.float32 if epi == 7 else dt)
        call("b200_linear_act", y.data_ptr(), x.data_ptr(), w.data_ptr(), M, N, K, 0 if epi == 7 and dtype == F32 else epi, 0.9, dtype,
             stream())
        torch.cuda.synchronize()
        close(y, want, F32 if epi == 7 else dtype)
