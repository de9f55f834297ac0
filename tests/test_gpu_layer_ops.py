"""The kernels of libktk_layers.so, one mechanism at a time, against the plain restatement (oracle/gifetar.py)."""
import pytest
import torch

from layer_helpers import PagedCase, pad_q, plain_attention, rms, standout_inputs
from oracle import gifetar as plain

pytestmark = pytest.mark.gpu
SIMT, MMA, UMMA = 1, 2, 3


# ---------------------------------------------------------------- residual + norms

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cols", [8, 30, 72, 256, 1000, 2048, 5120])
def test_residual_norm(cuda_device, dtype, cols):
    from kinetics_b200 import layer_ops as lo
    g = torch.Generator().manual_seed(cols)
    rows, parts, S, eps, mult = 5, 3, lo.pad8(cols), 1e-4, 0.3
    pad = lambda t: torch.nn.functional.pad(t, (0, S - cols))
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y = rnd(rows, cols) + 2.0, (rnd(rows, parts, cols) - 1.0).to(dtype).float()
    w1, b1, w2, b2 = (rnd(cols) for _ in range(4))
    embed = rnd(11, cols).to(dtype).float()
    dev = lambda t, d=torch.float32: pad(t).to(d).to(cuda_device).contiguous()
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=1e-2, atol=1e-2)
    h = torch.empty(rows, S, dtype=dtype, device=cuda_device)
    xd = dev(x)
    zero = torch.ones(70, dtype=torch.int32, device=cuda_device)
    lo.residual_norm(xd, h, cols, eps, pre=(dev(w2), dev(b2)), y=dev(y, dtype), parts=parts, post=(dev(w1), dev(b1)),
                     mult=mult, zero=zero)
    want = x.double() + mult * plain.layer_norm(y.double().sum(1), w1.double(), b1.double(), eps)
    torch.testing.assert_close(xd[:, :cols].cpu().double(), want, rtol=1e-5, atol=1e-5)     # fp32 in either dtype
    torch.testing.assert_close(h[:, :cols].cpu().double(), plain.layer_norm(want, w2.double(), b2.double(), eps), **tol)
    assert xd[:, cols:].abs().sum() == 0 and h[:, cols:].float().abs().sum() == 0 and int(zero.sum()) == 0
    # the start of a model; no post-norm; no centring and no bias
    tokens = torch.tensor([3, 0, 10, 7, 3], device=cuda_device)
    lo.residual_norm(xd, h, cols, eps, pre=(dev(w2), None), tokens=tokens, embed=dev(embed, dtype), center=False)
    torch.testing.assert_close(xd[:, :cols].cpu(), embed[tokens.cpu()], rtol=0, atol=0)
    want = plain.rms_unit(embed[tokens.cpu()].double(), eps) * w2.double()
    torch.testing.assert_close(h[:, :cols].cpu().double(), want, **tol)
    lo.residual_norm(xd, None, cols, eps, y=dev(y, dtype), parts=parts, mult=mult)
    torch.testing.assert_close(xd[:, :cols].cpu(), embed[tokens.cpu()] + mult * y.sum(1), rtol=1e-5, atol=1e-5)


def test_residual_norm_reports_a_token_outside_the_vocabulary(cuda_device):
    from kinetics_b200 import layer_ops as lo, ops
    x = torch.empty(1, 8, device=cuda_device)
    status = ops.new_status(cuda_device)
    lo.residual_norm(x, None, 8, 1e-5, tokens=torch.tensor([4], device=cuda_device),
                     embed=torch.zeros(4, 8, device=cuda_device), status=status)
    assert int(status.item()) == 2


# ---------------------------------------------------------------- append

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("page", [16, 32, 64])
def test_append_writes_rows_into_their_pages(cuda_device, dtype, page):
    from kinetics_b200 import layer_ops as lo, ops
    spec = lo.AttentionSpec(heads=4, kv_heads=2, dim=20, vdim=12, scale=1.0, maps=2)
    lens, new = [70, 64, 3, 17], [66, 1, 3, 2]
    zk = lambda n: torch.zeros(n, 2, 2, 20)
    case = PagedCase([zk(n) for n in lens], [torch.zeros(n, 2, 12) for n in lens], dtype, page, cuda_device)
    rows = sum(new)
    proj = torch.randn(rows, spec.q_cols + spec.k_cols + spec.v_cols).to(dtype).to(cuda_device)
    indptr = torch.tensor([0, 66, 67, 70, 72], dtype=torch.int32, device=cuda_device)
    before_k, before_v = case.k.clone(), case.v.clone()
    status = ops.new_status(cuda_device)
    lo.kv_append(proj, spec.q_cols, spec.q_cols + spec.k_cols, case.k, case.v, case.table, spec, indptr, status=status)
    idx, ptr, _ = (t.cpu() for t in case.table.tensors)
    tokens = lambda t: t.cpu().transpose(1, 2).reshape(t.shape[0] * page, -1)       # token slot by token slot
    want_k, want_v = tokens(before_k), tokens(before_v)
    r = 0
    for b, n in enumerate(new):
        for t in range(lens[b] - n, lens[b]):
            slot = int(idx[ptr[b] + t // page]) * page + t % page
            want_k[slot] = proj[r, spec.q_cols:spec.q_cols + spec.k_cols].cpu()
            want_v[slot] = proj[r, spec.q_cols + spec.k_cols:].cpu()
            r += 1
    same = lambda a, b: torch.equal(torch.nan_to_num(a.float(), nan=7.0), torch.nan_to_num(b.float(), nan=7.0))
    assert same(tokens(case.k), want_k) and same(tokens(case.v), want_v)
    # one row per sequence: the newest token of each
    one = torch.randn(4, proj.shape[1]).to(dtype).to(cuda_device)
    lo.kv_append(one, spec.q_cols, spec.q_cols + spec.k_cols, case.k, case.v, case.table, spec, status=status)
    for b in range(4):
        t = lens[b] - 1
        slot = int(idx[ptr[b] + t // page]) * page + t % page
        assert torch.equal(tokens(case.k)[slot], one[b, spec.q_cols:spec.q_cols + spec.k_cols].cpu())
    assert int(status.item()) == 0


# ---------------------------------------------------------------- attention

def _spec(heads, kv_heads, dim, vdim, cap=30.0, every=16.0, lam=0.37, maps=2):
    from kinetics_b200.layer_ops import AttentionSpec
    return AttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=0.6, maps=maps, softcap=cap,
                         temp_coef=0.15, temp_every=every, lam=lam, eps=1e-5, out_scale=0.75)


def _run(device, spec, lens, new, page, variant, dtype, splits=1, seed=0, strength=5.0, edges=None):
    """Attention of the newest `new` tokens of sequences of `lens` tokens (new None: one each, decode)."""
    from kinetics_b200 import layer_ops as lo, ops
    qs, ks, vs = [], [], []
    for i, n in enumerate(lens):
        first = n - (1 if new is None else new[i])
        at = edges or [0, 1, 2, 15, 16, 17, 31, 32, 47, 48, 63, 64, 65, 127, 128, 129, 191, 192, 255, 256, 257, first - 1,
                       first, first + 1, n - 2, n - 1, n // 2, n // 3]
        q, k, v = standout_inputs(n, first, spec.heads, spec.kv_heads, spec.dim, spec.vdim, at, seed + i, strength,
                                  spec.maps)
        qs.append(q.to(dtype).float())
        ks.append(k.to(dtype).float())
        vs.append(v.to(dtype).float())
    case = PagedCase(ks, vs, dtype, page, device, seed)
    proj = pad_q(torch.cat(qs), device, dtype)
    proj = torch.cat((proj, torch.full((proj.shape[0], 16), float("nan"), dtype=dtype, device=device)), dim=1)  # k, v side
    indptr = None
    if new is not None:
        indptr = torch.tensor([0] + list(torch.tensor(new).cumsum(0)), dtype=torch.int32, device=device)
    status = ops.new_status(device)
    out = lo.paged_attention(proj, case.k, case.v, case.table, spec, indptr, max(new) if new else 1, splits,
                             variant=variant, status=status)
    torch.cuda.synchronize()
    assert int(status.item()) == 0
    got = out.view(-1, spec.heads, spec.vdim_stride).cpu().double()
    assert got[:, :, spec.vdim:].abs().sum() == 0
    want = torch.cat([plain_attention(q, k, v, spec, k.shape[0] - q.shape[0]) for q, k, v in zip(qs, ks, vs)])
    return got[:, :, :spec.vdim], want


def _close(got, want, dtype):
    err = (got - want).abs()
    if dtype == torch.float32:
        assert err.max() < 2e-4, float(err.max())
    else:
        # bf16 probabilities and outputs of size one; the unit norm may enlarge a row whose two maps nearly cancel
        assert rms(got - want) < 8e-3 * max(1.0, rms(want)) and err.max() < 0.12, (rms(got - want), float(err.max()))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 2, 24, 40), (3, 1, 9, 13), (2, 2, 64, 128), (5, 5, 160, 200)])
def test_attention_fma_kernel(cuda_device, dtype, sizes):
    spec = _spec(*sizes)
    _close(*_run(cuda_device, spec, [150, 40, 1], [150, 2, 1], 16, SIMT, dtype), dtype)
    _close(*_run(cuda_device, spec, [150, 40, 1], None, 64, SIMT, dtype, seed=9), dtype)


def test_attention_with_one_map_is_ordinary_softmax_attention(cuda_device):
    from kinetics_b200 import layer_ops as lo
    spec = _spec(4, 2, 32, 24, maps=1)
    q, k, v = standout_inputs(70, 60, 4, 2, 32, 24, [0, 5, 60, 69], 3, maps=1)
    case = PagedCase([k], [v], torch.float32, 16, cuda_device)
    indptr = torch.tensor([0, 10], dtype=torch.int32, device=cuda_device)
    got = lo.paged_attention(pad_q(q, cuda_device, torch.float32), case.k, case.v, case.table, spec, indptr, 10)
    temp = plain.query_temperature(torch.arange(60, 70), spec.temp_coef, spec.temp_every)
    for h in range(4):
        s = plain.soft_cap((q[:, h, 0].double() * temp[:, None]) @ k[:, h // 2, 0].double().t() * spec.scale, 30.0)
        want = plain.causal_softmax(s, 60) @ v[:, h // 2].double()
        torch.testing.assert_close(got.view(10, 4, 24)[:, h].cpu().double(), want, rtol=1e-4, atol=1e-4)


# sizes: groups of 1, 3, 4, 8, 12; head sizes under, at and over a tile; caps inside and beyond the fixed reference, none
ATTN = [((4, 1, 32, 80), 28.0), ((6, 2, 24, 40), 12.0), ((8, 1, 64, 128), 50.0), ((12, 1, 48, 80), 90.0),
        ((2, 2, 128, 128), 0.0), ((3, 3, 72, 16), 25.0), ((4, 2, 16, 96), 0.0), ((8, 2, 96, 64), 7.5)]


@pytest.mark.parametrize("sizes, cap", ATTN)
@pytest.mark.parametrize("page", [16, 64])
def test_attention_of_prompts_on_tcgen05(cuda_device, sizes, cap, page):
    spec = _spec(*sizes, cap=cap)
    # whole prompts of unequal lengths in one launch, then portions behind a history (two tokens among them)
    _close(*_run(cuda_device, spec, [300, 64, 65, 1, 130], [300, 64, 65, 1, 130], page, UMMA, torch.bfloat16), torch.bfloat16)
    _close(*_run(cuda_device, spec, [300, 257, 66, 128], [2, 100, 3, 63], page, UMMA, torch.bfloat16, seed=4), torch.bfloat16)


@pytest.mark.parametrize("sizes, cap", ATTN)
@pytest.mark.parametrize("page, splits", [(16, 1), (64, 1), (32, 3), (64, 7)])
def test_attention_of_decode_steps_on_tensor_cores(cuda_device, sizes, cap, page, splits):
    spec = _spec(*sizes, cap=cap)
    lens = [1, 2, 15, 16, 17, 63, 64, 65, 300, 129]
    _close(*_run(cuda_device, spec, lens, None, page, MMA, torch.bfloat16, splits), torch.bfloat16)


def test_far_keys_among_many(cuda_device):
    # 4000 keys, a handful of them decisive: the first ones, ones at block borders far back, the newest
    spec = _spec(4, 2, 64, 128, every=500.0)
    at = [0, 1, 63, 64, 1023, 1024, 2047, 3000, 3998, 3999]
    got, want = _run(cuda_device, spec, [4000], [200], 64, UMMA, torch.bfloat16, strength=6.0, edges=at)
    _close(got, want, torch.bfloat16)
    got, want = _run(cuda_device, spec, [4000, 3999, 2048], None, 64, MMA, torch.bfloat16, splits=5, strength=6.0, edges=at)
    _close(got, want, torch.bfloat16)


def test_scores_beyond_the_polynomial_range(cuda_device):
    # |score / cap| runs from small to well beyond one: both branches of the softcap, in both kernels
    spec = _spec(2, 1, 64, 64, cap=5.0, lam=0.2)
    for strength in (1.0, 3.0, 8.0):
        _close(*_run(cuda_device, spec, [200], [200], 64, UMMA, torch.bfloat16, strength=strength), torch.bfloat16)
        _close(*_run(cuda_device, spec, [200, 90], None, 64, MMA, torch.bfloat16, strength=strength), torch.bfloat16)


def test_a_sequence_alone_and_in_a_batch_and_cut_differently(cuda_device):
    # the same rows, computed in other company, other portions and other pages
    from kinetics_b200 import layer_ops as lo
    spec = _spec(4, 2, 32, 64)
    dtype = torch.bfloat16
    q, k, v = standout_inputs(200, 0, 4, 2, 32, 64, [0, 63, 64, 100, 199], 1)
    k2, v2 = torch.randn(77, 2, 2, 32), torch.randn(77, 2, 64)
    proj = pad_q(q, cuda_device, dtype)
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=cuda_device)
    alone = PagedCase([k], [v], dtype, 64, cuda_device, 1)
    whole = lo.paged_attention(proj, alone.k, alone.v, alone.table, spec, i32(0, 200), 200)
    both = PagedCase([k2, k], [v2, v], dtype, 16, cuda_device, 2)
    mixed = lo.paged_attention(torch.cat((proj[:5], proj)), both.k, both.v, both.table, spec, i32(0, 5, 205), 200)
    assert rms(mixed[5:].float() - whole.float()) < 4e-3
    for first in (1, 63, 64, 150, 198):                    # the tail as a portion of its own
        part = lo.paged_attention(proj[first:].contiguous(), alone.k, alone.v, alone.table, spec, i32(0, 200 - first),
                                  200 - first)
        assert rms(part.float() - whole[first:].float()) < 4e-3
    last = lo.paged_attention(proj[199:].contiguous(), alone.k, alone.v, alone.table, spec)
    assert rms(last.float() - whole[199:].float()) < 6e-3


def test_attention_refuses_and_reports(cuda_device):
    from kinetics_b200 import _lib, layer_ops as lo, ops
    spec = _spec(2, 2, 160, 64)
    case = PagedCase([torch.zeros(20, 2, 2, 160)], [torch.zeros(20, 2, 64)], torch.bfloat16, 16, cuda_device)
    q = torch.zeros(1, spec.q_cols, dtype=torch.bfloat16, device=cuda_device)
    with pytest.raises(_lib.KtkError):                     # head size without a tensor-core kernel
        lo.paged_attention(q, case.k, case.v, case.table, spec, variant=MMA)
    lo.paged_attention(q, case.k, case.v, case.table, spec)            # auto: the FMA kernel
    with pytest.raises(RuntimeError):
        lo.paged_attention(q.cpu(), case.k, case.v, case.table, spec)
    # a page id outside the cache is reported, not followed
    spec = _spec(2, 2, 32, 64)
    case = PagedCase([torch.zeros(20, 2, 2, 32)], [torch.zeros(20, 2, 64)], torch.bfloat16, 16, cuda_device)
    case.table.tensors[0][1] = 1000
    q = torch.zeros(2, spec.q_cols, dtype=torch.bfloat16, device=cuda_device)
    for indptr, rows, variant in ((None, 1, MMA), (torch.tensor([0, 2], dtype=torch.int32, device=cuda_device), 2, UMMA),
                                  (None, 1, SIMT)):
        status = ops.new_status(cuda_device)
        lo.paged_attention(q[:rows], case.k, case.v, case.table, spec, indptr, rows, variant=variant, status=status)
        assert int(status.item()) == 1


# ---------------------------------------------------------------- experts

def _moe_case(rows, experts, top, width, ff, dtype, seed=0, skew=0.0):
    from kinetics_b200.layer_ops import pad8
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, scale=1.0: (torch.randn(*s, generator=g) * scale).to(dtype).float()
    c = dict(h=r(rows, width), router=r(experts, width, scale=width ** -0.5), b=torch.randn(experts, generator=g) * 0.3,
             gate=r(experts, ff, width, scale=width ** -0.5), up=r(experts, ff, width, scale=width ** -0.5),
             down=r(experts, width, ff, scale=ff ** -0.5))
    c["b"][0] += skew
    ws, fs = pad8(width), pad8(ff)
    p = torch.nn.functional.pad
    c["dev"] = lambda d: dict(
        h=p(c["h"], (0, ws - width)).to(dtype).to(d).contiguous(),
        router=p(c["router"], (0, ws - width)).to(dtype).to(d).contiguous(), b=c["b"].to(d),
        gate_up=p(torch.stack((c["gate"], c["up"]), 2), (0, ws - width, 0, 0, 0, fs - ff)).to(dtype).to(d).contiguous(),
        down=p(c["down"], (0, fs - ff, 0, ws - width)).to(dtype).to(d).contiguous())
    return c


MOE = [(1, 4, 2, 32, 24), (3, 5, 5, 72, 56), (40, 11, 3, 100, 88), (300, 7, 1, 256, 130), (513, 64, 8, 136, 64),
       (200, 1, 1, 48, 300), (130, 3, 2, 520, 200), (77, 130, 4, 64, 32),
       (700, 3, 2, 200, 176), (520, 1, 1, 72, 40), (900, 2, 2, 264, 520), (257, 1, 1, 64, 128)]


@pytest.mark.parametrize("dtype, variant", [(torch.float32, SIMT), (torch.bfloat16, SIMT), (torch.bfloat16, MMA)])
@pytest.mark.parametrize("rows, experts, top, width, ff", MOE)
def test_router(cuda_device, dtype, variant, rows, experts, top, width, ff):
    from kinetics_b200 import layer_ops as lo
    c = _moe_case(rows, experts, top, width, ff, dtype)
    d = c["dev"](cuda_device)
    r = lo.moe_route(d["h"], d["router"], d["b"], lo.MoeSpec(experts, top, width, ff), variant=variant)
    z = c["h"].double() @ c["router"].double().t() + c["b"].double()
    ids = r.ids.cpu().long()
    got = z.gather(1, ids)
    best = torch.topk(z, top, dim=1).values
    torch.testing.assert_close(got, best, rtol=1e-4, atol=1e-4)        # the same experts, up to equal logits
    assert all(len(set(row.tolist())) == top for row in ids)
    torch.testing.assert_close(r.weights.cpu().double(), torch.softmax(got, dim=1), rtol=1e-4, atol=1e-4)
    counts = torch.bincount(ids.reshape(-1), minlength=experts)
    assert torch.equal(r.counts.cpu().long(), counts)
    bucket = r.bucket.cpu()
    for e in range(experts):
        assert sorted(bucket[e, :counts[e]].tolist()) == (ids.reshape(-1) == e).nonzero().reshape(-1).tolist()


@pytest.mark.parametrize("dtype, variant", [(torch.float32, SIMT), (torch.bfloat16, SIMT), (torch.bfloat16, UMMA)])
@pytest.mark.parametrize("rows, experts, top, width, ff", MOE)
@pytest.mark.parametrize("skew", [0.0, 50.0])
def test_expert_products(cuda_device, dtype, variant, rows, experts, top, width, ff, skew):
    # skew: one expert gets every row (tiles of one expert only), others share what is left
    from kinetics_b200 import layer_ops as lo, ops
    c = _moe_case(rows, experts, top, width, ff, dtype, seed=1, skew=skew)
    d = c["dev"](cuda_device)
    spec = lo.MoeSpec(experts, top, width, ff)
    r = lo.moe_route(d["h"], d["router"], d["b"], spec)
    status = ops.new_status(cuda_device)
    y = lo.moe_experts(d["h"], d["gate_up"], d["down"], r, spec, variant=variant, status=status)
    torch.cuda.synchronize()
    assert int(status.item()) == 0
    ids, weights = r.ids.cpu().long(), r.weights.cpu().double()
    h = c["h"].double()
    want = torch.empty(rows, top, width, dtype=torch.float64)
    for e in range(experts):
        at, place = (ids == e).nonzero(as_tuple=True)
        if at.numel():
            want[at, place] = weights[at, place].unsqueeze(1) * plain.expert(
                h[at], c["gate"][e].double(), c["up"][e].double(), c["down"][e].double())
    tol = 1e-4 if dtype == torch.float32 else 2e-2
    scale = max(rms(want), 1e-3)
    assert (y[:, :, :width].cpu().double() - want).abs().max() < tol * scale * 4
    assert rms(y[:, :, :width].cpu().double() - want) < tol * scale * 0.5
    assert y[:, :, width:].float().abs().sum() == 0


def test_a_row_gets_the_same_experts_output_in_any_batch(cuda_device):
    from kinetics_b200 import layer_ops as lo
    c = _moe_case(400, 6, 2, 128, 96, torch.bfloat16, seed=2)
    d = c["dev"](cuda_device)
    spec = lo.MoeSpec(6, 2, 128, 96)

    def run(rows):
        h = d["h"][rows].contiguous()
        r = lo.moe_route(h, d["router"], d["b"], spec)
        return r.ids.cpu(), lo.moe_experts(h, d["gate_up"], d["down"], r, spec).cpu()

    ids, y = run(slice(0, 400))
    for rows in (slice(0, 1), slice(17, 20), slice(100, 300), slice(399, 400)):
        ids2, y2 = run(rows)
        assert torch.equal(ids2, ids[rows])
        assert rms(y2.float() - y[rows].float()) < 2e-3
