"""The mechanisms of the Retotar layers one by one, through the C ABI, against the oracle's functions."""
import ctypes
import math

import pytest
import torch

from oracle import retotar_oracle as O

pytestmark = pytest.mark.gpu

BF16, F32 = 0, 1
TORCH = {BF16: torch.bfloat16, F32: torch.float32}
# limits relative to the largest of the wanted values
TOL = {BF16: 2e-2, F32: 2e-5}
LIGHTNING, MEMORY = 2, 3


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


def angles(base, dims, length, factor=1.0):
    a = torch.arange(length, dtype=torch.float64)[:, None] * base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims) / factor
    return a.cos().float().cuda(), a.sin().float().cuda()


# ---- mixing heads ------------------------------------------------------------------------
class Paged:
    """Requests of given lengths in paged pools whose pages are shuffled; the last `ext` positions of each are queries.
    Queries and keys are unit vectors up to sqrt(d), as the layers make them."""

    def __init__(self, lens, exts, heads, kv_heads, d, dv, page, dtype, seed=0, pad=(128, 128)):
        g = gen(seed)
        self.lens, self.exts, self.heads, self.kv_heads, self.d, self.dv = lens, exts, heads, kv_heads, d, dv
        self.page, self.dtype, (self.dp, self.vp) = page, dtype, pad
        dt = TORCH[dtype]
        unit = lambda *s: O.unit_rms(torch.randn(*s, generator=g), 1e-6).to(dt)
        self.k = [unit(n, kv_heads, d) for n in lens]
        self.v = [torch.randn(n, kv_heads, dv, generator=g).to(dt) for n in lens]
        self.q = [unit(n, heads, d) for n in exts]
        self.gate = [torch.randn(n, heads, dv, generator=g).to(dt) for n in exts]
        self.mix = torch.eye(heads) + 0.4 * torch.randn(heads, heads, generator=g)
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

    def attend(self, call, scale, window=2 ** 31 - 1, keep=0, gate=1, turned=True, out_scale=1.0, plain=0, decode=0, bound=True):
        """gate: 0 none, 1 per element, 2 per head."""
        from sglang_cpp_b200 import _lib

        H, G, dp, vp, dt = self.heads, self.kv_heads, self.dp, self.vp, TORCH[self.dtype]
        kc, vc = torch.full((self.slots, G, dp), 3.0, dtype=dt), torch.full((self.slots, G, vp), 50.0, dtype=dt)
        kc[..., self.d:], vc[..., self.dv:] = 0, 0
        for r, n in enumerate(self.lens):
            s = self.table[r, :n].long()
            kc[s, :, :self.d], vc[s, :, :self.dv] = self.k[r], self.v[r]
        T, gate_cols = sum(self.exts), H * vp if gate == 1 else up64(H)
        rows = torch.zeros(T, H * dp + 64 + gate_cols, dtype=dt)
        rows[:, :H * dp] = pad_to(torch.cat(self.q), T, H, dp).view(T, -1)
        g = torch.cat(self.gate)
        rows[:, H * dp + 64:] = pad_to(g, T, H, vp).view(T, -1) if gate == 1 else pad_to(g[..., 0], T, gate_cols)
        rows, kc, vc, table = rows.cuda(), kc.cuda(), vc.cuda(), self.table.cuda()
        out = torch.full((T, H * vp + 64), 9.0, dtype=dt, device="cuda")
        idx, lens, mix = ints(*range(len(self.lens))), ints(*self.lens), self.mix.cuda()
        qo = ints(0, *torch.tensor(self.exts).cumsum(0).tolist())
        row_table = ints(*[r for r, n in enumerate(self.exts) for _ in range(n)])
        row_len = ints(*[n - e + i + 1 for n, e in zip(self.lens, self.exts) for i in range(e)])
        positions = row_len - 1
        cos, sin = angles(70.0, self.dv, self.cols)
        lib = _lib.load()
        nbytes = max(lib.b200_head_mix_workspace_bytes(len(self.lens), H, G), 16)
        ws = torch.full((nbytes,), 0x7f, dtype=torch.uint8, device="cuda")
        scratch = torch.full((lib.b200_head_mix_scratch_bytes(T, H, G, vp, self.dtype),), 0x7f, dtype=torch.uint8, device="cuda")
        a = _lib.WindowAttentionArgs(
            out=out.data_ptr(), q=rows.data_ptr(), q_stride=rows.stride(0), k_cache=kc.data_ptr(), v_cache=vc.data_ptr(),
            num_slots=self.slots, page_table=table.data_ptr(), page_table_stride=self.cols, table_idx=idx.data_ptr(),
            seq_lens=lens.data_ptr(), qo_indptr=qo.data_ptr(), row_table=row_table.data_ptr(), row_len=row_len.data_ptr(),
            tokens=T, batch=len(self.lens), max_extend=max(self.exts), decode=decode, plain=plain, heads=H, kv_heads=G,
            padded_dim=dp, padded_value_dim=vp, page_size=self.page, scale=scale, window=window, keep_first=keep,
            gate=rows.data_ptr() + (H * dp + 64) * rows.element_size() if gate else None, gate_stride=rows.stride(0),
            workspace=ws.data_ptr(), workspace_bytes=nbytes, gate_per_head=int(gate == 2), out_scale=out_scale,
            out_stride=out.stride(0), head_mix=mix.data_ptr(), value_rotary=self.dv if turned else 0, max_pos=self.cols,
            value_cos=cos.data_ptr(), value_sin=sin.data_ptr(), positions=positions.data_ptr(),
            score_bound=1.02 * self.d if bound else 0.0, mix_scratch=scratch.data_ptr())
        call("b200_window_attention", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        assert float((out[:, H * vp:].float() - 9).abs().sum()) == 0
        out = out[:, :H * vp].view(T, H, vp)
        assert float(out[..., self.dv:].float().abs().sum()) == 0
        return out[..., :self.dv].cpu()

    def want(self, scale, window=2 ** 31 - 1, keep=0, gate=1, turned=True, out_scale=1.0):
        out = []
        for r, (n, e) in enumerate(zip(self.lens, self.exts)):
            seen = O.visible(n, window)
            seen[:, :keep] |= O.visible(n)[:, :keep]
            q = torch.cat([torch.zeros(n - e, self.heads, self.d, dtype=torch.float64), self.q[r].double()])
            p = O.talking_heads(O.softmax_weights(q, self.k[r].double(), scale, seen)[:, n - e:], self.mix.double())
            o = O.weighted_values(p, self.v[r].double())
            if turned:
                o = O.rotate_half(o, -torch.arange(n - e, n), 70.0, self.dv)
            g = torch.sigmoid(self.gate[r].double())
            out.append(out_scale * (o if gate == 0 else o * g if gate == 1 else o * g[..., :1]))
        return torch.cat(out)


WINDOWS = [1, 5, 64, 100, 128, 129, 140, 1000, 2 ** 31 - 1]
LENS, EXTS = [300, 1, 65, 700, 130, 128, 900], [300, 1, 2, 90, 66, 127, 33]


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("heads, kv_heads, dv, page, gate", [(8, 2, 128, 64, 1), (4, 4, 64, 1, 0), (16, 1, 128, 16, 2), (32, 8, 50, 256, 1),
                                                             (3, 3, 96, 64, 1), (8, 1, 10, 64, 1), (16, 4, 128, 64, 1), (32, 4, 128, 64, 1)])
def test_mixing_heads_in_prompts(call, window, heads, kv_heads, dv, page, gate):
    p = Paged(LENS, EXTS, heads, kv_heads, 128, dv, page, BF16, window % 97)
    close(p.attend(call, 0.09, window, gate=gate, out_scale=0.8), p.want(0.09, window, gate=gate, out_scale=0.8), BF16)


@pytest.mark.parametrize("window", WINDOWS)
@pytest.mark.parametrize("heads, kv_heads, dv, page, gate", [(8, 2, 128, 64, 1), (5, 1, 64, 16, 1), (16, 4, 50, 1, 2), (32, 8, 128, 64, 1),
                                                             (12, 2, 96, 64, 0), (40, 4, 128, 32, 1), (8, 8, 10, 64, 1), (16, 1, 128, 256, 1),
                                                             (24, 2, 128, 64, 1), (60, 4, 128, 64, 1)])
def test_mixing_heads_of_decoded_tokens(call, window, heads, kv_heads, dv, page, gate):
    lens = [1, 2, 63, 64, 65, 128, 129, 700, 1500, 333, 201]
    p = Paged(lens, [1] * len(lens), heads, kv_heads, 128, dv, page, BF16, window % 97)
    close(p.attend(call, 0.09, window, gate=gate, out_scale=-1.2, decode=1), p.want(0.09, window, gate=gate, out_scale=-1.2), BF16)


def test_mixing_heads_of_one_long_request_and_many_short_ones(call):
    for lens in ([6000], [int(n) for n in torch.randint(1, 90, (300,), generator=gen(0))]):
        p = Paged(lens, [1] * len(lens), 8, 2, 128, 128, 64, BF16, 3)
        for window in (50, 4000, 2 ** 31 - 1):
            close(p.attend(call, 0.09, window, decode=1), p.want(0.09, window), BF16)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("heads, kv_heads, d, dv, pad", [(6, 2, 40, 56, (128, 128)), (3, 3, 144, 200, (192, 256)), (7, 7, 8, 16, (64, 64)),
                                                         (12, 3, 96, 34, (128, 128)), (12, 12, 64, 128, (128, 128))])
@pytest.mark.parametrize("window, gate, turned", [(33, 1, True), (1, 0, True), (150, 2, False), (2 ** 31 - 1, 1, True)])
def test_mixing_heads_plain_kernel(call, dtype, heads, kv_heads, d, dv, pad, window, gate, turned):
    p = Paged([1, 190, 400, 7], [1, 150, 3, 2], heads, kv_heads, d, dv, 16, dtype, 5, pad)
    close(p.attend(call, 0.2, window, gate=gate, turned=turned, out_scale=1.5, plain=1),
          p.want(0.2, window, gate=gate, turned=turned, out_scale=1.5), dtype)


@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("keep", [1, 4, 130])
@pytest.mark.parametrize("heads, kv_heads", [(8, 2), (12, 12), (32, 8)])
def test_mixing_heads_with_the_first_keys_kept(call, decode, keep, heads, kv_heads):
    lens = [500, 64, 333, 1]
    exts = [1] * 4 if decode else [500, 64, 40, 1]
    p = Paged(lens, exts, heads, kv_heads, 128, 128, 64, BF16, keep)
    for window in (3, 100, 129):
        close(p.attend(call, 0.09, window, keep, decode=decode), p.want(0.09, window, keep), BF16)


@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("scale, bound", [(0.3, True), (0.9, True), (0.09, False), (-0.1, True)])
def test_scores_of_any_size(call, decode, scale, bound):
    """Scores up to what the kernels without a running maximum take, beyond it, without a bound, and upside down."""
    p = Paged([200, 70, 1], [1] * 3 if decode else [200, 30, 1], 8, 2, 128, 128, 64, BF16, 7)
    close(p.attend(call, scale, 90, bound=bound, decode=decode), p.want(scale, 90), BF16, 1.5)


@pytest.mark.parametrize("decode", [0, 1])
@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 1)])
@pytest.mark.parametrize("window", [64, 100, 128, 129, 400, 401])
def test_a_key_that_stands_out_at_a_windows_edge(call, decode, dtype, plain, window):
    """Keys on both sides of the edge, one at a time, carry a huge score for every head: the output is the mixing
    matrix's row sums times that key's value, or shows nothing of it."""
    n = 401
    edge = n - window
    spots = sorted({s for s in (0, edge - 1, edge, edge + 1, n - 1) if 0 <= s < n})
    p = Paged([n] * len(spots), [1] * len(spots), 4, 1, 128, 128, 64, dtype, 1)
    for r, s in enumerate(spots):
        p.q[r].zero_()
        p.q[r][:, :, 0] = 128 ** 0.5
        p.k[r][:, :, 0] = 0
        p.k[r][s] = 0
        p.k[r][s, :, 0] = 128 ** 0.5
    got, want = p.attend(call, 0.2, window, gate=0, turned=False, plain=plain, decode=decode), p.want(0.2, window, gate=0, turned=False)
    close(got, want, dtype)
    rows = p.mix.sum(1)
    for r, s in enumerate(spots):
        same = float((got[r].float() - rows[:, None] * p.v[r][s].float()).abs().max()) < 0.05 * float(rows.abs().max() * p.v[r][s].abs().max())
        assert same == (s >= edge), s


def test_heads_mix_as_the_matrix_says(call):
    """With one key per request the softmax weights are 1: what comes out is the row sums of the matrix.  With a
    permutation, heads trade places within a key head's group."""
    p = Paged([1, 1], [1, 1], 4, 2, 128, 64, 16, BF16, 2)
    for decode in (0, 1):
        got = p.attend(call, 0.1, gate=0, turned=False, decode=decode)
        want = p.mix.sum(1)[None, :, None] * torch.stack([v[0].float().repeat_interleave(2, 0) for v in p.v])
        close(got, want, BF16)
    p = Paged([200], [60], 4, 2, 128, 64, 16, BF16, 3)
    p.mix = torch.eye(4)
    straight = p.attend(call, 0.1)
    p.mix, p.gate[0] = torch.eye(4)[[1, 0, 3, 2]], p.gate[0][:, [1, 0, 3, 2]]
    close(p.attend(call, 0.1)[:, [1, 0, 3, 2]], straight, BF16, 0.5)


# ---- heads between projection and attention --------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("tokens, heads, kv_heads, d, dv, dims", [(9, 6, 2, 40, 56, 24), (700, 6, 2, 128, 128, 64), (700, 8, 0, 128, 128, 128),
                                                                  (5, 3, 3, 144, 200, 100), (700, 6, 2, 64, 40, 16), (700, 6, 2, 100, 50, 8)])
def test_heads_turn_and_become_unit_vectors(call, dtype, tokens, heads, kv_heads, d, dv, dims):
    from sglang_cpp_b200 import _lib

    g, dt = gen(d + dv), TORCH[dtype]
    dp, vp = (128 if d <= 128 else up64(d)), (128 if dv <= 128 else up64(dv))
    q, k, v = (torch.randn(tokens, n, m, generator=g).to(dt) for n, m in ((heads, d), (kv_heads, d), (kv_heads, dv)))
    joint = torch.cat([pad_to(q, tokens, heads, dp).flatten(1), pad_to(k, tokens, kv_heads, dp).flatten(1),
                       pad_to(v, tokens, kv_heads, vp).flatten(1), torch.full((tokens, 64), 2.0, dtype=dt)], 1).cuda()
    slots = tokens + 7
    kc, vc = torch.full((slots, kv_heads, dp), 4.0, dtype=dt, device="cuda"), torch.full((slots, kv_heads, vp), 4.0, dtype=dt, device="cuda")
    loc, pos = torch.randperm(slots, generator=g)[:tokens], torch.randint(0, 900, (tokens,), generator=g)
    (cos, sin), (vcos, vsin) = angles(300.0, dims, 900, 3.0), angles(300.0, dv, 900)
    dl, dpos = loc.int().cuda(), pos.int().cuda()
    a = _lib.HeadPrepareArgs(
        joint=joint.data_ptr(), joint_ld=joint.stride(0), tokens=tokens, heads=heads, kv_heads=kv_heads, dim=d, padded_dim=dp,
        padded_value_dim=vp, eps=1e-3, rotary_dim=dims, max_pos=900, cos_table=cos.data_ptr(), sin_table=sin.data_ptr(),
        positions=dpos.data_ptr(), out_loc=dl.data_ptr(), k_cache=kc.data_ptr() or joint.data_ptr(), v_cache=vc.data_ptr() or joint.data_ptr(),
        num_slots=slots, unit_norm=1, value_rotary=dv, value_cos=vcos.data_ptr(), value_sin=vsin.data_ptr())
    call("b200_head_prepare", ctypes.byref(a), dtype, stream())
    torch.cuda.synchronize()
    want = O.unit_rms(O.rotate_half(q.double(), pos, 300.0, dims, 3.0), 1e-3)
    got = joint[:, :heads * dp].view(tokens, heads, dp)
    close(got[..., :d], want, dtype)
    assert float(got[..., d:].float().abs().sum()) == 0 and bool((joint[:, -64:] == 2).all())
    if kv_heads:
        close(kc[dl.long()][..., :d], O.unit_rms(O.rotate_half(k.double(), pos, 300.0, dims, 3.0), 1e-3), dtype)
        close(vc[dl.long()][..., :dv], O.rotate_half(v.double(), pos, 300.0, dv), dtype)
        assert float(vc[dl.long()][..., dv:].float().abs().sum()) == 0
        free = torch.ones(slots, dtype=torch.bool)
        free[loc] = False
        assert bool((kc.cpu()[free] == 4).all() and (vc.cpu()[free] == 4).all())


# ---- recurrences ---------------------------------------------------------------------
class Recurrence:
    """Requests of given lengths through one recurrent mixer between its projections."""

    def __init__(self, rule, exts, heads, d, dv, dtype, seed=0, decays=None, gates=((0.0, 3.0), (3.0, 3.0)), cap=9.0):
        g, dt = gen(seed), TORCH[dtype]
        self.rule, self.exts, self.H, self.d, self.dv, self.dtype, self.cap, self.eps = rule, exts, heads, d, dv, dtype, cap, 1e-5
        T = sum(exts)
        rand = lambda *s: torch.randn(*s, generator=g).to(dt)
        self.gate, self.v, self.k, self.q = rand(T, heads, dv), rand(T, heads, dv), rand(T, heads, d), rand(T, heads, d)
        self.i, self.f = (gain * rand(T, heads) for _, gain in gates)
        self.bias = torch.cat([centre + torch.randn(heads, generator=g) for centre, _ in gates])
        self.decay = torch.tensor(decays) if decays else 1 - 2.0 ** -(1 + 9 * torch.rand(heads, generator=g))
        self.norm = (1 + 0.3 * torch.randn(heads, dv, generator=g)).to(dt)
        self.dp, self.vp = up64(d), up64(dv)

    def states(self, rows):
        from sglang_cpp_b200 import _lib

        width = _lib.load().b200_recurrence_memory_bytes(self.dp, self.vp) // 4
        return torch.full((rows, self.H, self.dp, self.vp), 7.0, device="cuda"), torch.full((rows, self.H, width), 5.0, device="cuda")

    def run(self, call, states, cached, table_idx, tokens=None, plain=0, decode=0, wide=0):
        """tokens: for every request, which of its tokens to bring (a slice); the states are changed in place."""
        from sglang_cpp_b200 import _lib

        H, dp, vp, dt = self.H, self.dp, self.vp, TORCH[self.dtype]
        starts = [0] + torch.tensor(self.exts).cumsum(0).tolist()
        pick = [list(range(starts[i], starts[i + 1]))[tokens[i] if tokens else slice(None)] for i in range(len(self.exts))]
        rows = torch.tensor([t for p in pick for t in p])
        T, lens = len(rows), [len(p) for p in pick]
        heads = lambda x, to: pad_to(x[rows], T, H, to).flatten(1)
        parts = [torch.full((T, 64), 9.0, dtype=dt), heads(self.gate, vp), heads(self.v, vp), heads(self.k, dp), heads(self.q, dp)]
        if self.rule == MEMORY:
            parts.append(pad_to(torch.cat([self.i[rows], self.f[rows]], 1), T, up64(2 * H)))
        joint = torch.cat(parts, 1).cuda()
        decay, bias, norm = self.decay.log().cuda(), self.bias.cuda(), pad_to(self.norm, H, vp).flatten().cuda()
        ld = H * vp + wide
        out = torch.full((T, ld), 4.0, dtype=dt, device="cuda")
        nbytes = (ctypes.c_int64 * 4)()
        call("b200_recurrence_scratch", self.rule, T, len(lens), H, H, dp, vp, self.dtype, nbytes)
        scratch = [torch.full((max(n, 16),), 0x7f, dtype=torch.uint8, device="cuda") for n in nbytes]
        qo, idx, ca = ints(0, *torch.tensor(lens).cumsum(0).tolist()), ints(*table_idx), ints(*cached)
        a = _lib.RecurrenceArgs(
            out=out.data_ptr(), out_ld=ld, joint=joint.data_ptr() + 64 * joint.element_size(), joint_ld=joint.stride(0), rule=self.rule,
            tokens=T, batch=len(lens), max_extend=max(lens), decode=decode, plain=plain, table_idx=idx.data_ptr(), cached=ca.data_ptr(),
            qo_indptr=qo.data_ptr(), state=states[0].data_ptr(), heads=H, kv_heads=H, dim=self.d, padded_dim=dp, value_dim=self.dv,
            padded_value_dim=vp, taps=1, norm_groups=1 if self.rule == LIGHTNING else H,
            decay_log=decay.data_ptr() if self.rule == LIGHTNING else None, step_bias=bias.data_ptr() if self.rule == MEMORY else None,
            norm=norm.data_ptr(), eps=self.eps, out_scale=1.0, mixed=scratch[0].data_ptr(), steps=scratch[1].data_ptr(),
            units=scratch[2].data_ptr(), chunks=scratch[3].data_ptr(), gate_cap=self.cap, memory=states[1].data_ptr())
        call("b200_recurrence", ctypes.byref(a), self.dtype, stream())
        torch.cuda.synchronize()
        if wide:
            assert float((out[:, H * vp:].float() - 4).abs().sum()) == 0
        out = out[:, :H * vp].view(T, H, vp)
        assert float(out[..., self.dv:].float().abs().sum()) == 0
        return out[..., :self.dv].cpu()

    def want(self):
        """Per request, outputs and last state."""
        outs, states, at = [], [], 0
        for n in self.exts:
            s = slice(at, at + n)
            at += n
            q, k, v, gate = (x[s].double() for x in (self.q, self.k, self.v, self.gate))
            if self.rule == LIGHTNING:
                silu = torch.nn.functional.silu
                y, S = O.decayed_recurrence(silu(q), silu(k), silu(v), self.decay.double())
                y = O.unit_rms(y.reshape(n, -1), self.eps).view_as(y)
            else:
                i = O.capped(self.i[s].double() + self.bias[:self.H].double(), self.cap)
                f = torch.nn.functional.logsigmoid(O.capped(self.f[s].double() + self.bias[self.H:].double(), self.cap))
                y, S = O.matrix_memory(q / math.sqrt(self.d), k, v, i, f)
                y = O.unit_rms(y, self.eps)
            outs.append(y * self.norm.double() * torch.sigmoid(gate))
            states.append(S)
        return outs, states

    def check_state(self, states, row, S, dtype, factor=1.0):
        d, dv = self.d, self.dv
        if self.rule == LIGHTNING:
            close(states[0][row, :, :d, :dv], S, dtype, factor)
        else:
            S, z, m = S
            width = self.dp + 4
            memory = states[1][row].view(self.H, -1, width)
            for c in range(memory.shape[1]):
                close(memory[:, c, self.dp], m / math.log(2), F32, 5.0)
                close(memory[:, c, :d], z, dtype, factor)
            close(states[0][row, :, :d, :dv], S, dtype, factor)
        assert float(states[0][row, :, d:].abs().sum()) == 0 and float(states[0][row, :, :, dv:].abs().sum()) == 0


# rule, heads, dim, value dim
SHAPES = [(LIGHTNING, 4, 128, 128), (LIGHTNING, 3, 64, 192), (LIGHTNING, 5, 40, 20), (LIGHTNING, 1, 100, 72),
          (MEMORY, 4, 128, 128), (MEMORY, 3, 64, 64), (MEMORY, 5, 24, 40), (MEMORY, 2, 100, 200)]
BIG = [(LIGHTNING, 2, 260, 136), (MEMORY, 2, 200, 264), (MEMORY, 1, 600, 20), (MEMORY, 1, 1000, 130), (LIGHTNING, 1, 64, 600)]


@pytest.mark.parametrize("dtype, plain", [(BF16, 0), (BF16, 1), (F32, 0)])
@pytest.mark.parametrize("rule, heads, d, dv", SHAPES + BIG)
def test_recurrence_of_prompts(call, dtype, plain, rule, heads, d, dv):
    x = Recurrence(rule, [1, 2, 63, 64, 65, 200, 17], heads, d, dv, dtype, d)
    states = x.states(9)
    rows = [8, 0, 3, 2, 7, 1, 5]
    got = x.run(call, states, [0] * 7, rows, plain=plain, wide=64)
    outs, last = x.want()
    close(got, torch.cat(outs), dtype, 2.0)
    for r, S in zip(rows, last):
        x.check_state(states, r, S, dtype)
    assert bool((states[0][4] == 7).all() and (states[0][6] == 7).all() and (states[1][4] == 5).all())   # rows of other requests


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("rule, heads, d, dv", SHAPES + BIG)
@pytest.mark.parametrize("cut", [1, 2, 37, 64, 99])
def test_portions_and_decoding_carry_the_states_on(call, dtype, rule, heads, d, dv, cut):
    n = 130
    x = Recurrence(rule, [n, n], heads, d, dv, dtype, 11)
    states = x.states(3)
    parts, at = [], 0
    while at < n:
        m = min(cut, n - at)
        part = x.run(call, states, [at, at], [2, 0], [slice(at, at + m)] * 2, decode=int(m == 1 and at > 0), wide=128)
        parts.append(part.view(2, m, heads, dv))
        at += m
    outs, last = x.want()
    close(torch.cat(parts, 1).reshape(2 * n, heads, dv), torch.cat(outs), dtype, 2.0 if dtype == BF16 else 3.0)
    for r, S in zip((2, 0), last):
        x.check_state(states, r, S, dtype, 1.0 if dtype == BF16 else 2.0)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("decays", [(1.0, 0.5, 0.9999), (1e-6, 1e-30, 0.2)])
def test_constant_decays_however_steep_or_flat(call, decays, dtype):
    x = Recurrence(LIGHTNING, [150, 70], 3, 128, 64, dtype, 3, decays)
    states = x.states(2)
    got = x.run(call, states, [0, 0], [0, 1])
    outs, last = x.want()
    close(got, torch.cat(outs), dtype, 2.0)
    for r, S in enumerate(last):
        x.check_state(states, r, S, dtype)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("gates, cap", [(((0.0, 30.0), (0.0, 30.0)), 30.0),      # gates from shut to wide open, token by token
                                        (((-25.0, 1.0), (20.0, 1.0)), 40.0),     # hardly any input: the denominator's floor
                                        (((25.0, 5.0), (-20.0, 5.0)), 60.0),     # huge inputs, soon forgotten
                                        (((-30.0, 2.0), (-9.0, 2.0)), 35.0),     # a maximum that falls from 0
                                        (((0.0, 3.0), (0.0, 3.0)), 0.5)])        # capped hard
def test_exponential_gates_of_any_size(call, gates, cap, dtype):
    x = Recurrence(MEMORY, [150, 70], 6, 128, 64, dtype, 3, gates=gates, cap=cap)
    outs, last = x.want()
    for portions in ([slice(None)], [slice(0, 1), slice(1, 30), slice(30, None)]):
        states, at = x.states(2), 0
        for s in portions:
            got = x.run(call, states, [at, at], [0, 1], [s, s])
            at = s.stop or 0
        from_ = portions[-1].start or 0
        close(got, torch.cat([o[from_:] for o in outs]), dtype, 2.0 if dtype == BF16 else 5.0)
        for r in range(2):
            x.check_state(states, r, last[r], dtype, 1.0 if dtype == BF16 else 5.0)


@pytest.mark.parametrize("rule", [LIGHTNING, MEMORY])
@pytest.mark.parametrize("dtype", [BF16, F32])
def test_a_token_is_remembered_across_a_long_prompt(call, rule, dtype):
    """One key stands out at token 3 of a state that does not decay; it is read out 600 tokens later, from a prompt,
    from portions and from decoding."""
    n = 640
    for steps in ([n], [n - 1, 1], [100, 300, 240]):
        x = Recurrence(rule, [n], 1, 64, 64, dtype, 4, (1.0,), cap=50.0)
        low = -30.0 if rule == LIGHTNING else 0.0               # (silu leaves nothing of it)
        x.k[..., 5] = low
        x.k[3], x.q[n - 1] = low, low
        x.k[3, 0, 5], x.q[n - 1, 0, 5] = 8.0, 8.0
        x.i.zero_()
        x.bias[0], x.bias[1] = 0.0, 45.0
        x.f.zero_()
        states, at, got = x.states(1), 0, None
        for m in steps:
            got = x.run(call, states, [at], [0], [slice(at, at + m)], decode=int(m == 1))
            at += m
        outs, _ = x.want()
        close(got[-1], outs[0][-1], dtype, 2.0)
        v = x.v[3, 0].double()
        v = torch.nn.functional.silu(v) if rule == LIGHTNING else v
        want = O.unit_rms(v, 0.0) * x.norm[0].double() * torch.sigmoid(x.gate[-1, 0].double())
        close(got[-1, 0], want, BF16, 2.0)


# ---- residual stream ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [40, 192, 1000, 9000])
@pytest.mark.parametrize("top, init, normed, last", [(0, 1, 0, 1), (0, 0, 1, 1), (1, 0, 1, 0), (3, 0, 1, 1), (20, 0, 0, 1), (2, 1, 0, 0)])
def test_residual_layer_norm(call, dtype, width, top, init, normed, last):
    T, padded, eps, shift = 7, up64(width), 1e-5, 40.0
    g, dt = gen(width + top), TORCH[dtype]
    rand = lambda rows, gain=1.0, at=0.0: pad_to((at + gain * torch.randn(rows, width, generator=g)).to(dt), rows, padded)
    res = pad_to(shift + torch.randn(T, width, generator=g), T, padded)     # (a mean far from zero)
    src, self_rows = rand(11 if top else T, 2.0, 5.0), rand(T)
    rows = torch.randint(-1, 11, (T, max(top, 1)), generator=g).int()
    weights = torch.rand(T, max(top, 1), generator=g)
    aw, ab, ow, ob = rand(1, 1.0)[0], rand(1, 0.5)[0], rand(1)[0], rand(1, 0.5)[0]
    n = lambda x, w, b: O.layer_normalise(x, w[:width].double(), b[:width].double(), eps)
    add = src[:, :width].double()
    if top:
        pick = torch.where((rows >= 0)[..., None], src[rows.clamp(min=0).long()], self_rows[:, None])[..., :width].double()
        add = (weights.double()[..., None] * pick).sum(1)
    add = add * 0.7 if init else add
    add = n(add, aw, ab) if normed else add
    want_res = add if init else res[:, :width].double() + add
    want = n(want_res, ow, ob) if last else want_res
    out, r = torch.zeros(T, padded, dtype=dt, device="cuda"), res.cuda()
    dev = [x.cuda() for x in (src, self_rows, aw, ab, ow, ob, rows, weights)]
    p = [x.data_ptr() for x in dev]
    call("b200_residual_layer_norm", out.data_ptr(), r.data_ptr(), p[0], p[6] if top else None, p[7] if top else None, max(top, 1),
         len(src), p[1], 0.7, init, p[2] if normed else None, p[3], p[4] if last else None, p[5], T, width, padded, eps, dtype, stream())
    torch.cuda.synchronize()
    close(r[:, :width], want_res, F32)
    close(out[:, :width], want, dtype, 1.0 if dtype == BF16 else 3.0)
    assert float(out[:, width:].float().abs().sum()) == 0 and float(r[:, width:].abs().sum()) == 0


# ---- routing -------------------------------------------------------------------------------
@pytest.mark.parametrize("tokens", [1, 9, 1500])
@pytest.mark.parametrize("experts, identity, top, groups, keep", [(1, 0, 1, 1, 1), (12, 4, 3, 4, 3), (9, 3, 2, 4, 1), (6, 6, 4, 3, 2), (3, 61, 5, 8, 4),
                                                                  (64, 16, 8, 5, 4), (250, 50, 20, 5, 2), (7, 0, 7, 1, 1), (1500, 500, 4, 1000, 30)])
def test_softmax_routing(call, tokens, experts, identity, top, groups, keep):
    g = gen(experts + tokens)
    outputs = experts + identity
    ld = up64(outputs)
    logits = pad_to(2 * torch.randn(tokens, outputs, generator=g), tokens, ld)
    correction = -0.2 + 0.5 / outputs * torch.randn(outputs, generator=g)     # (choice scores on both sides of zero)
    x = torch.randn(tokens, 64, generator=g).bfloat16().cuda()
    i32 = dict(dtype=torch.int32, device="cuda")
    ids, rows = torch.full((tokens, top), -7, **i32), torch.full((tokens, top), -7, **i32)
    weights, counts, off = torch.zeros(tokens, top, device="cuda"), torch.zeros(2 * experts, **i32), torch.zeros(experts + 1, **i32)
    xp = torch.zeros(tokens * top, 64, dtype=torch.bfloat16, device="cuda")
    dl, dc = logits.cuda(), correction.cuda()
    call("b200_score_route", ids.data_ptr(), weights.data_ptr(), rows.data_ptr(), counts.data_ptr(), off.data_ptr(), xp.data_ptr(),
         x.data_ptr(), 128, dl.data_ptr(), ld, tokens, experts, top, groups, keep, 1.0, 1, identity, dc.data_ptr(), stream())
    torch.cuda.synchronize()
    r = {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}}
    some = range(tokens) if tokens * outputs < 100000 else range(0, tokens, 13)
    want = [O.route(logits[t, :outputs], correction, r) for t in some]       # (fp32: the kernel's own precision)
    for t, (chosen, w) in zip(some, want):
        assert ids[t].tolist() == chosen, t
        torch.testing.assert_close(weights[t].cpu(), w, rtol=1e-5, atol=1e-7)
    chosen, r = ids.cpu().long(), rows.cpu().long()
    real = chosen < experts
    assert bool((r[~real] == -1).all())
    n = torch.bincount(chosen[real], minlength=experts)
    assert torch.equal(counts[:experts].cpu().long(), n)
    assert torch.equal(off.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), n.cumsum(0)]))
    assert torch.equal(r[real].sort().values, torch.arange(int(real.sum())))
    first = off.cpu().long()[chosen.clamp(max=experts - 1)]
    behind = off.cpu().long()[chosen.clamp(max=experts - 1) + 1]
    assert bool(((r >= first) & (r < behind))[real].all())
    assert torch.equal(xp.cpu()[r[real]], x.cpu()[:, None].expand(-1, top, -1)[real])


def test_routing_of_logits_that_are_not_numbers(call):
    """A token's experts are valid and differ all the same: what follows counts on it."""
    for score in (0, 1):
        logits = torch.full((5, 64), float("nan"), device="cuda")
        i32 = dict(dtype=torch.int32, device="cuda")
        ids, rows, weights = torch.zeros(5, 3, **i32), torch.zeros(5, 3, **i32), torch.zeros(5, 3, device="cuda")
        counts, off, xp = torch.zeros(24, **i32), torch.zeros(13, **i32), torch.zeros(15, 64, dtype=torch.bfloat16, device="cuda")
        x = torch.zeros(5, 64, dtype=torch.bfloat16, device="cuda")
        call("b200_score_route", ids.data_ptr(), weights.data_ptr(), rows.data_ptr(), counts.data_ptr(), off.data_ptr(), xp.data_ptr(),
             x.data_ptr(), 128, logits.data_ptr(), 64, 5, 12, 3, 4, 2, 1.0, score, 0, None, stream())
        torch.cuda.synchronize()
        for t in ids.tolist():
            assert len(set(t)) == 3 and all(0 <= e < 12 for e in t)
        assert int(counts[:12].max()) <= 5 and int(counts[:12].sum()) == 15
