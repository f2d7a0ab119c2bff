"""The mechanisms of the layer stack one by one, through the C ABI, against plain torch."""
import ctypes

import pytest
import torch

pytestmark = pytest.mark.gpu

BF16, F32 = 0, 1
TORCH = {BF16: torch.bfloat16, F32: torch.float32}


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
    return torch.Generator(device="cuda").manual_seed(seed)


# ---- latent attention ----------------------------------------------------------------
class Pool:
    """A paged latent pool whose pages are shuffled; every row of queries has a page-table row of its own."""

    def __init__(self, lens, width, page, dtype, seed):
        g = gen(seed)
        pages = sum(-(-n // page) for n in lens) + 2
        self.lens, self.width, self.page, self.dtype, self.slots = lens, width, page, dtype, pages * page
        self.cache = torch.randn(self.slots, width, generator=g, device="cuda").to(TORCH[dtype])
        perm = torch.randperm(pages, generator=g, device="cuda")
        self.cols = (max(lens) + page + 31) // 32 * 32
        self.table = torch.zeros(len(lens), self.cols, dtype=torch.int32, device="cuda")
        k = 0
        for r, n in enumerate(lens):
            m = -(-n // page)
            s = (perm[k:k + m, None] * page + torch.arange(page, device="cuda")).flatten()
            self.table[r, :len(s)] = s.int()
            k += m

    def key(self, row, pos):
        return self.cache[int(self.table[row, pos])]

    def attend(self, call, q, scale, plain=0):
        from sglang_cpp_b200 import _lib

        rows, heads, _ = q.shape
        ids = torch.arange(rows, dtype=torch.int32, device="cuda")
        lens = torch.tensor(self.lens, dtype=torch.int32, device="cuda")
        n = _lib.load().b200_latent_attention_workspace_bytes(rows, heads, self.width)
        ws = torch.zeros(n, dtype=torch.uint8, device="cuda")
        out = torch.full_like(q, 9.0)
        call("b200_latent_attention", out.data_ptr(), q.data_ptr(), self.cache.data_ptr(), self.slots,
             self.table.data_ptr(), self.cols, ids.data_ptr(), lens.data_ptr(), rows, heads, self.width, self.page,
             scale, self.dtype, plain, ws.data_ptr(), n, stream())
        torch.cuda.synchronize()
        return out.float()

    def want(self, q, scale):
        out = torch.zeros(q.shape, device="cuda")
        for r, n in enumerate(self.lens):
            if n:
                c = self.cache[self.table[r, :n].long()].double()
                out[r] = (torch.softmax(q[r].double() @ c.T * scale, -1) @ c).float()
        return out


@pytest.mark.parametrize("heads", [1, 6, 16, 17, 33, 64, 65, 130])
@pytest.mark.parametrize("width, page", [(128, 64), (256, 16), (384, 1), (512, 64), (512, 256)])
def test_latent_attention_on_the_tensor_cores(call, heads, width, page):
    lens = [1, 2, 63, 64, 65, 127, 128, 129, 0, 700, 255]
    pool = Pool(lens, width, page, BF16, heads + width)
    q = (2 * torch.randn(len(lens), heads, width, generator=gen(1), device="cuda")).bfloat16()
    torch.testing.assert_close(pool.attend(call, q, width ** -0.5), pool.want(q, width ** -0.5), rtol=2e-2, atol=2e-2)


def test_latent_attention_when_rows_outnumber_ctas_and_when_one_row_spans_them_all(call):
    for lens in ([int(n) for n in torch.randint(1, 400, (333,), generator=torch.Generator().manual_seed(0))], [40000]):
        pool = Pool(lens, 256, 64, BF16, 5)
        q = torch.randn(len(lens), 12, 256, generator=gen(2), device="cuda").bfloat16()
        torch.testing.assert_close(pool.attend(call, q, 0.125), pool.want(q, 0.125), rtol=2e-2, atol=1e-2)


@pytest.mark.parametrize("dtype, width", [(F32, 128), (F32, 640), (BF16, 640)])
def test_latent_attention_plain_kernel(call, dtype, width):
    lens = [1, 3, 64, 200]
    pool = Pool(lens, width, 16, dtype, 3)
    q = torch.randn(4, 5, width, generator=gen(4), device="cuda").to(TORCH[dtype])
    tol = 1e-5 if dtype == F32 else 1e-2
    torch.testing.assert_close(pool.attend(call, q, 0.1), pool.want(q, 0.1), rtol=tol, atol=tol)


@pytest.mark.parametrize("plain", [0, 1])
@pytest.mark.parametrize("width", [128, 512])
def test_one_key_that_stands_out_is_found_wherever_it_is(call, plain, width):
    """The query points at one key: the output must be that key, at the first and last position, at page and
    tile borders - and the key just past the row's length must not be seen however well it matches."""
    n, page = 1000, 64
    spots = [0, 1, 63, 64, 127, 128, 129, 511, 512, 640, 998, 999]
    pool = Pool([n] * len(spots), width, page, BF16, 7)
    q = torch.zeros(len(spots), 6, width, device="cuda", dtype=torch.bfloat16)
    for r, at in enumerate(spots):
        q[r] = pool.key(r, at)
        pool.cache[int(pool.table[r, n])] = 50 * pool.key(r, at)     # position n: in the page, not in the row
    got = pool.attend(call, q, 0.5, plain)
    for r, at in enumerate(spots):
        torch.testing.assert_close(got[r], pool.key(r, at).float().expand(6, -1), rtol=2e-2, atol=2e-2)


def test_scores_that_grow_along_the_row_keep_their_weights(call):
    """Every tile's maximum is far above the one before (the reference maximum moves each time), and the
    other way round."""
    for flip in (False, True):
        pool = Pool([1500], 256, 64, BF16, 8)
        ramp = torch.linspace(-3, 3, 1500, device="cuda")
        u = torch.randn(256, generator=gen(9), device="cuda")
        slots = pool.table[0, :1500].long()
        pool.cache[slots] = ((ramp.flip(0) if flip else ramp)[:, None] * u + 0.3 * torch.randn(1500, 256, generator=gen(10), device="cuda")).bfloat16()
        q = (u * torch.linspace(0.1, 2, 20, device="cuda")[:, None]).bfloat16()[None].contiguous()
        torch.testing.assert_close(pool.attend(call, q, 0.2), pool.want(q, 0.2), rtol=2e-2, atol=3e-2)


# ---- residual stream ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("width", [40, 192, 1000, 9000])
@pytest.mark.parametrize("src_top, out_top, init", [(0, 0, 0), (1, 0, 1), (3, 2, 0), (20, 18, 0)])
def test_residual_norm(call, dtype, width, src_top, out_top, init):
    T, padded, eps = 7, -(-width // 64) * 64, 1e-5
    g = gen(width + src_top)

    def padded_rand(rows):
        x = torch.zeros(rows, padded, device="cuda", dtype=TORCH[dtype])
        x[:, :width] = torch.randn(rows, width, generator=g, device="cuda").to(TORCH[dtype])
        return x

    res = torch.zeros(T, padded, device="cuda")
    res[:, :width] = torch.randn(T, width, generator=g, device="cuda")
    src = padded_rand(T if src_top == 0 else 50)
    rows = torch.randint(0, 50, (T, max(src_top, 1)), generator=g, device="cuda").int()
    weight = padded_rand(1)[0] * 0.3
    out_rows = torch.randperm(T * max(out_top, 1), generator=g, device="cuda").int().view(T, -1)
    out = torch.zeros(T * max(out_top, 1), padded, device="cuda", dtype=TORCH[dtype])
    add = 0.25 * (src.float() if src_top == 0 else src.float()[rows.long()].sum(1))
    want_res = add if init else res + add
    n = want_res * torch.rsqrt(want_res[:, :width].pow(2).mean(-1, keepdim=True) + eps)
    want = 0.5 * n * (weight.float() + 1.0)
    call("b200_residual_norm", out.data_ptr(), out_rows.data_ptr() if out_top else None, max(out_top, 1), res.data_ptr(),
         src.data_ptr(), rows.data_ptr() if src_top else None, max(src_top, 1), len(src), 0.25, init, weight.data_ptr(),
         1.0, 0.5, T, width, padded, eps, dtype, stream())
    torch.cuda.synchronize()
    torch.testing.assert_close(res, want_res, rtol=1e-6, atol=1e-5)
    got = out[out_rows.long()] if out_top else out[:, None]
    tol = 1e-2 if dtype == BF16 else 1e-5
    torch.testing.assert_close(got.float(), want[:, None].expand_as(got), rtol=tol, atol=tol)
    assert float(out[:, width:].float().abs().sum()) == 0 and float(res[:, width:].abs().sum()) == 0


def test_residual_norm_without_a_source_leaves_the_stream_alone(call):
    res = torch.randn(3, 128, device="cuda")
    before, out, w = res.clone(), torch.zeros(3, 128, device="cuda"), torch.ones(128, device="cuda")
    call("b200_residual_norm", out.data_ptr(), None, 1, res.data_ptr(), None, None, 1, 0, 1.0, 0, w.data_ptr(), 0.0, 1.0,
         3, 128, 128, 1e-6, F32, stream())
    torch.cuda.synchronize()
    assert torch.equal(res, before)
    torch.testing.assert_close(out, before * torch.rsqrt(before.pow(2).mean(-1, keepdim=True) + 1e-6))


# ---- projections ---------------------------------------------------------------------------
@pytest.mark.parametrize("M", [1, 33, 64, 200, 256, 300])
@pytest.mark.parametrize("heads, N, K", [(1, 128, 512), (6, 256, 128), (16, 512, 128), (40, 128, 384), (3, 192, 64)])
def test_projection_per_head(call, M, heads, N, K):
    x = torch.randn(M, heads * K, generator=gen(M), device="cuda").bfloat16()
    w = (torch.randn(heads, N, K, generator=gen(K), device="cuda") / K ** 0.5).bfloat16()
    y = torch.zeros(M, heads, N, device="cuda", dtype=torch.bfloat16)
    call("b200_linear_heads", y.data_ptr(), x.data_ptr(), w.data_ptr(), M, heads, N, K, stream())
    torch.cuda.synchronize()
    want = torch.einsum("mhk,hnk->mhn", x.view(M, heads, K).float(), w.float())
    torch.testing.assert_close(y.float(), want, rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("M", [5, 128, 400])
@pytest.mark.parametrize("N, K", [(64, 128), (1024, 2048), (320, 64)])
def test_squared_relu_epilogue(call, M, N, K):
    x = torch.randn(M, K, generator=gen(M), device="cuda").bfloat16()
    w = (torch.randn(N, K, generator=gen(N), device="cuda") / K ** 0.5).bfloat16()
    y = torch.zeros(M, N, device="cuda", dtype=torch.bfloat16)
    call("b200_linear", y.data_ptr(), x.data_ptr(), w.data_ptr(), None, M, N, K, K, 4, stream())
    torch.cuda.synchronize()
    torch.testing.assert_close(y.float(), torch.relu(x.float() @ w.float().T) ** 2, rtol=2e-2, atol=2e-2)


def test_fp32_projections_in_all_their_forms(call):
    g = gen(0)
    x, w = torch.randn(70, 192, generator=g, device="cuda"), torch.randn(200, 192, generator=g, device="cuda") / 14
    full = (x.double() @ w.double().T)
    acts = {0: full, 2: torch.nn.functional.gelu(full[:, :100], approximate="tanh") * full[:, 100:],
            1: torch.nn.functional.silu(full[:, :100]) * full[:, 100:], 4: torch.relu(full) ** 2}
    for epi, want in acts.items():
        y = torch.zeros(want.shape, device="cuda")
        call("b200_linear_f32", y.data_ptr(), x.data_ptr(), w.data_ptr(), 70, 200, 192, 1, None, None, epi, stream())
        torch.cuda.synchronize()
        torch.testing.assert_close(y.double(), want, rtol=1e-5, atol=1e-5)
    # per head
    xh, wh = torch.randn(9, 3 * 64, generator=g, device="cuda"), torch.randn(3, 96, 64, generator=g, device="cuda")
    y = torch.zeros(9, 3, 96, device="cuda")
    call("b200_linear_f32", y.data_ptr(), xh.data_ptr(), wh.data_ptr(), 9, 96, 64, 3, None, None, 0, stream())
    torch.cuda.synchronize()
    torch.testing.assert_close(y, torch.einsum("mhk,hnk->mhn", xh.view(9, 3, 64), wh), rtol=1e-4, atol=1e-4)
    # grouped, with an empty group
    counts, off = torch.tensor([4, 0, 5], device="cuda").int(), torch.tensor([0, 4, 4, 9], device="cuda").int()
    xg = torch.randn(9, 64, generator=g, device="cuda")
    y = torch.zeros(9, 96, device="cuda")
    call("b200_linear_f32", y.data_ptr(), xg.data_ptr(), wh.data_ptr(), 9, 96, 64, 3, counts.data_ptr(), off.data_ptr(), 0, stream())
    torch.cuda.synchronize()
    torch.testing.assert_close(y, torch.cat([xg[:4] @ wh[0].T, xg[4:] @ wh[2].T]), rtol=1e-4, atol=1e-4)


# ---- table routing --------------------------------------------------------------------------
@pytest.mark.parametrize("tokens, experts, top", [(1, 1, 1), (9, 5, 5), (3000, 64, 4), (500, 3000, 2)])
def test_table_route_places_every_choice_once(call, tokens, experts, top):
    vocab = 77
    g = torch.Generator().manual_seed(tokens)
    table = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(vocab)]).int()
    ids = torch.randint(0, vocab, (tokens,), generator=g).int()
    rows = torch.full((tokens, top), -1, dtype=torch.int32, device="cuda")
    counts = torch.zeros(experts, dtype=torch.int32, device="cuda")
    off = torch.zeros(experts + 1, dtype=torch.int32, device="cuda")
    t, i = table.cuda(), ids.cuda()
    call("b200_table_route", rows.data_ptr(), counts.data_ptr(), off.data_ptr(), t.data_ptr(), i.data_ptr(), tokens, vocab,
         top, experts, stream())
    torch.cuda.synchronize()
    chosen = table[ids.long()].long()
    assert torch.equal(counts.cpu().long(), torch.bincount(chosen.flatten(), minlength=experts))
    assert torch.equal(off.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), counts.cpu().long().cumsum(0)]))
    r = rows.cpu().long()
    assert torch.equal(r.flatten().sort().values, torch.arange(tokens * top))
    assert bool(((r >= off.cpu().long()[chosen]) & (r < off.cpu().long()[chosen + 1])).all())
