"""Attention over rows that all heads share (value = first columns of the key), its append step and the linear
recurrence on the GPU, each against its plain formula: sizes, page sizes, far keys, edges, portions, splits."""
import pytest
import torch

from latent_helpers import RowPages, plain_rows, pointed_rows, rms
from oracle import munadra as plain

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def _spec(heads, cols, vdim, scale):
    from kinetics_b200.layer_ops import AttentionSpec
    return AttentionSpec(heads=heads, kv_heads=1, dim=cols, vdim=vdim, scale=scale, values_in_keys=True)


def _attend(dev, spec, q, pages, dtype, sink, gate, indptr, max_new, variant=0, splits=1):
    from kinetics_b200 import layer_ops as lo, ops
    status = ops.new_status(dev)
    out = lo.paged_attention(q.flatten(1).to(dtype).to(dev).contiguous(), pages.pages, pages.pages, pages.table, spec,
                             None if indptr is None else torch.tensor(indptr, dtype=torch.int32, device=dev), max_new,
                             splits, variant=variant, status=status, sink=sink.float().to(dev),
                             gate=gate.to(dtype).to(dev).contiguous())
    ops.raise_on_status(status)
    return out.view(q.shape[0], spec.heads, -1)[:, :, :spec.vdim].double().cpu()


# heads, columns, columns of the value
SIZES = [(16, 576, 512), (6, 160, 128), (3, 72, 56), (64, 320, 256), (128, 576, 512), (40, 264, 200), (1, 64, 64), (70, 96, 8)]


@pytest.mark.parametrize("heads,cols,vdim", SIZES)
def test_decode_rows(cuda_device, heads, cols, vdim):
    lens = [1, 63, 64, 65, 200, 777, 2000]
    for seed, (ps, splits, dtype, variant) in enumerate([(64, 1, BF, 0), (64, 5, BF, 0), (16, 3, BF, 0), (32, 40, BF, 0),
                                                         (16, 1, F32, 0), (64, 1, BF, 1)]):
        if dtype == F32 and heads > 16:
            continue
        spec = _spec(heads, cols, vdim, 1.1 / cols ** 0.5)
        parts = [pointed_rows(n, n - 1, heads, cols, [0, 1, n // 2, 63, 64, n - 1], seed + i, strength=8.0) for i, n in enumerate(lens)]
        pages = RowPages([k for _, k in parts], dtype, ps, cuda_device, seed)
        g = torch.Generator().manual_seed(seed)
        sink, gate = 2.0 * torch.randn(heads, generator=g), torch.randn(len(lens), heads, generator=g)
        q = torch.cat([x for x, _ in parts])
        got = _attend(cuda_device, spec, q, pages, dtype, sink, gate, None, 1, variant, splits)
        r = lambda t: t.to(dtype).double()
        for i, (qi, k) in enumerate(parts):
            want = plain_rows(r(qi), r(k), vdim, spec.scale, sink.double(), r(gate[i:i + 1]), lens[i] - 1)
            err = rms(got[i:i + 1] - want) / rms(want)
            assert err < (1e-5 if dtype == F32 else 1.2e-2), (ps, splits, lens[i], err)


@pytest.mark.parametrize("heads,cols,vdim", SIZES)
def test_portions(cuda_device, heads, cols, vdim):
    for seed, (ps, total, new, dtype) in enumerate([(64, 300, 300, BF), (16, 130, 2, BF), (64, 65, 3, BF), (32, 513, 70, BF),
                                                    (64, 1100, 7, BF), (16, 80, 40, F32)]):
        spec, first = _spec(heads, cols, vdim, 1.1 / cols ** 0.5), total - new
        q, k = pointed_rows(total, first, heads, cols, [0, 1, 15, 16, 63, 64, 65, first - 1, first, first + 1, total - 1],
                            seed, strength=8.0)
        pages = RowPages([k], dtype, ps, cuda_device, seed)
        g = torch.Generator().manual_seed(seed)
        sink, gate = 2.0 * torch.randn(heads, generator=g), torch.randn(new, heads, generator=g)
        r = lambda t: t.to(dtype).double()
        want = plain_rows(r(q), r(k), vdim, spec.scale, sink.double(), r(gate), first)
        for splits in (1, 4):
            got = _attend(cuda_device, spec, q, pages, dtype, sink, gate, [0, new], new, 0, splits)
            err = (got - want).pow(2).mean(-1).sqrt() / rms(want)
            assert err.max() < (1e-5 if dtype == F32 else 3e-2), (ps, total, new, splits, float(err.max()))


def test_sinks_of_every_size(cuda_device):
    # a sink far above, near and far below the scores; and scores that keep growing along the sequence
    heads, cols, vdim, n = 8, 128, 96, 700
    g = torch.Generator().manual_seed(3)
    k = torch.randn(n, cols, generator=g)
    q = torch.randn(1, heads, cols, generator=g)
    ramp = torch.linspace(0, 60, n).unsqueeze(1) * torch.nn.functional.normalize(q[0, 0], dim=0)
    spec = _spec(heads, cols, vdim, 0.2)
    for rows in (k, k + ramp, (k + ramp).flip(0)):
        pages = RowPages([rows], BF, 64, cuda_device)
        for sink in (torch.full((heads,), 40.0), torch.linspace(-30, 30, heads), torch.full((heads,), -1e4)):
            for splits in (1, 3):
                got = _attend(cuda_device, spec, q, pages, BF, sink, torch.zeros(1, heads), None, 1, 0, splits)
                want = plain_rows(q.to(BF).double(), rows.to(BF).double(), vdim, spec.scale, sink.double(),
                                  torch.zeros(1, heads).double(), n - 1)
                assert (got - want).abs().max() < 2e-2 * max(rms(want), 1e-3), (splits, sink[0])


# heads, dim, rot_dim, vdim
EXPANDED = [(4, 128, 64, 128), (3, 32, 32, 32), (2, 40, 8, 72), (1, 192, 64, 128), (5, 64, 128, 16), (2, 24, 16, 100)]


@pytest.mark.parametrize("heads,dim,rot_dim,vdim", EXPANDED)
def test_expanded_attention(cuda_device, heads, dim, rot_dim, vdim):
    from kinetics_b200 import layer_ops as lo, ops
    from kinetics_b200.layer_ops import LatentSpec, Rotation, pad8
    dev, rank = cuda_device, 48
    spec = LatentSpec(heads, dim, rot_dim, vdim, rank, 1.2 / (dim + rot_dim) ** 0.5, Rotation(rot_dim, 1e4))
    d, r, v, R = pad8(dim), pad8(rot_dim), pad8(vdim), pad8(rank)
    for seed, (total, n) in enumerate([(1, 1), (64, 64), (65, 2), (128, 128), (129, 129), (300, 257), (700, 130), (513, 513)]):
        g = torch.Generator().manual_seed(seed)
        first = total - n
        edges = [0, 1, 63, 64, 65, 127, 128, first - 1, first, first + 1, total // 2, total - 2, total - 1]
        q, k = pointed_rows(total, first, heads, dim + rot_dim, edges, seed, strength=6.0)
        keys = k[:, None, :dim] + 0.1 * torch.randn(total, heads, dim, generator=g)
        values = torch.randn(total, heads, vdim, generator=g)
        sink, gate = torch.linspace(-4, 6, heads), torch.randn(n, heads, generator=g)
        proj = torch.zeros(n, spec.proj_cols)
        qp = proj[:, :spec.q_cols].view(n, heads, d + r)
        qp[:, :, :dim], qp[:, :, d:d + rot_dim] = q[..., :dim], q[..., dim:]
        proj[:, spec.gate_col:spec.gate_col + heads] = gate
        kv = torch.zeros(total, heads * (d + v))
        kv[:, :heads * d].view(total, heads, d)[:, :, :dim] = keys
        kv[:, heads * d:].view(total, heads, v)[:, :, :vdim] = values
        lat = torch.full((total, R + r), float("nan"))
        lat[:, R:] = 0.0
        lat[:, R:R + rot_dim] = k[:, dim:]
        put = lambda t: t.to(BF).to(dev)
        proj, status = put(proj), ops.new_status(dev)
        got = lo.expanded_attention(proj, put(kv), put(lat), spec, sink.to(dev), proj[:, spec.gate_col:], status)
        ops.raise_on_status(status)
        got = got.view(n, heads, v).double().cpu()
        r64 = lambda t: t.to(BF).double()
        for h in range(heads):
            s = (r64(q[:, h, :dim]) @ r64(keys[:, h]).t() + r64(q[:, h, dim:]) @ r64(k[:, dim:]).t()) * spec.scale
            want = plain.sigmoid(r64(gate[:, h:h + 1])) * (plain.sink_softmax(s, sink[h].double(), first) @ r64(values[:, h]))
            err = (got[:, h, :vdim] - want).pow(2).mean(-1).sqrt() / rms(want)
            assert err.max() < 3e-2, (total, n, h, float(err.max()))
        assert (got[:, :, vdim:] == 0).all()


@pytest.mark.parametrize("dtype", [F32, BF])
def test_append_rotates_and_normalises(cuda_device, dtype):
    from kinetics_b200 import layer_ops as lo, ops
    from kinetics_b200.layer_ops import LatentSpec, Rotation, pad8
    dev = cuda_device
    for seed, (heads, dim, rot_dim, rank, ps, lens, new, scaling) in enumerate([
            (3, 24, 16, 40, 16, [200], 37, dict(factor=4.0, original=32, fast=6.0, slow=0.5, scaled=True)),
            (2, 20, 10, 36, 64, [1, 70, 64], None, {}), (1, 8, 2, 130, 32, [9], 9, {}),
            (5, 128, 64, 512, 64, [120000, 3], None, dict(factor=8.0, original=512, fast=32.0, slow=1.0, scaled=True))]):
        g = torch.Generator().manual_seed(seed)
        rotation = Rotation(rot_dim, 3000.0, **scaling)
        raw = {"dims": rot_dim, "base": 3000.0}
        if scaling:
            raw["scaling"] = {k: v for k, v in scaling.items() if k != "scaled"}
        spec = LatentSpec(heads, dim, rot_dim, 8, rank, 1.0, rotation, eps=1e-3)
        d, r, R, rows = pad8(dim), pad8(rot_dim), pad8(rank), new or len(lens)
        q, kv = torch.randn(rows, heads, dim + rot_dim, generator=g), 3 * torch.randn(rows, rank + rot_dim, generator=g)
        w = torch.randn(rank, generator=g)
        proj = torch.zeros(rows, spec.proj_cols)
        qp = proj[:, :spec.q_cols].view(rows, heads, d + r)
        qp[..., :dim], qp[..., d:d + rot_dim] = q[..., :dim], q[..., dim:]
        proj[:, spec.q_cols:spec.q_cols + rank] = kv[:, :rank]
        proj[:, spec.q_cols + R:spec.q_cols + R + rot_dim] = kv[:, rank:]
        at = torch.arange(lens[0] - new, lens[0]) if new else torch.tensor(lens) - 1
        r64 = lambda t: t.to(dtype).double()
        want_q = plain.rotate(r64(q[..., dim:]), at, raw)
        want_c = plain.rms_norm(r64(kv[:, :rank]), w.double(), 1e-3)
        want_k = plain.rotate(r64(kv[:, rank:]), at, raw)
        tol = dict(atol=2e-5, rtol=1e-5) if dtype == F32 else dict(atol=3e-2, rtol=1e-2)
        norm = torch.zeros(R)
        norm[:rank] = w
        indptr = torch.tensor([0, new], dtype=torch.int32, device=dev) if new else None
        for in_place in (False, True):
            pages = RowPages([torch.zeros(n, spec.row_cols) for n in lens], dtype, ps, dev, seed)
            p, status = proj.to(dtype).to(dev), ops.new_status(dev)
            q_out = None if in_place else torch.zeros(rows, heads, spec.row_cols, dtype=dtype, device=dev)
            lo.latent_append(p, spec, pages.table, pages.pages, norm.to(dev), rotation.turns().to(dev), indptr, q_out,
                             status=status)
            ops.raise_on_status(status)
            turned = p[:, :spec.q_cols].view(rows, heads, -1)[:, :, d:] if in_place else q_out[:, :, R:]
            torch.testing.assert_close(turned[..., :rot_dim].double().cpu(), want_q, **tol)
            for b in range(len(lens)):
                row = pages.row(b)[-(new or 1):].double().cpu()
                mine = slice(0, rows) if new else slice(b, b + 1)
                torch.testing.assert_close(row[:, :rank], want_c[mine], **tol)
                torch.testing.assert_close(row[:, R:R + rot_dim], want_k[mine], **tol)
                assert (pages.row(b)[:-(new or 1)] == 0).all()


# ---- the recurrence
def _lru_case(spec, tokens, seed):
    """Inputs of a sequence in true sizes, and the same padded block by block."""
    from kinetics_b200.layer_ops import pad8
    g = torch.Generator().manual_seed(seed)
    B, n, bs = spec.blocks, spec.block, pad8(spec.block)
    c = dict(x=torch.randn(tokens, B * n, generator=g), y=2 * torch.randn(tokens, B * n, generator=g),
             w=torch.randn(B * n, spec.taps, generator=g), b=torch.randn(B * n, generator=g),
             ra=torch.randn(B, n, n, generator=g) / n ** 0.5, ri=torch.randn(B, n, n, generator=g) / n ** 0.5,
             rab=torch.randn(B, n, generator=g), rib=torch.randn(B, n, generator=g),
             lam=3 * torch.randn(B * n, generator=g) - 3)

    def spread(t, fill=0.0):                                  # [..., B * n] -> [..., B * bs]
        out = torch.full((*t.shape[:-1], B, bs), fill)
        out[..., :n] = t.view(*t.shape[:-1], B, n)
        return out.flatten(-2)
    return c, spread


def _lru_plain(c, dtype):
    r = lambda t: t.to(dtype).double()
    x, y = r(c["x"]), r(c["y"])
    u, _ = plain.causal_conv(x, x.new_zeros(c["w"].shape[1] - 1, x.shape[1]), c["w"].double(), c["b"].double())
    u = r(u)
    gate = lambda w, b: plain.block_gate(u, r(w), b.double())
    s, _ = plain.linear_recurrence(gate(c["ra"], c["rab"]), gate(c["ri"], c["rib"]), u, c["lam"].double(), torch.zeros(x.shape[1]).double())
    return s * plain.gelu_tanh(y)


class _Lru:
    """Drives conv, gate products and scan over one manager-like set of slots."""

    def __init__(self, spec, cases, spread, dtype, dev, slots):
        from kinetics_b200.layer_ops import pad8
        c, n, bs = cases[0], spec.block, pad8(spec.block)
        self.spec, self.dtype, self.dev = spec, dtype, dev
        put = lambda t: t.float().to(dev).contiguous()
        self.w, self.b = put(spread(c["w"].t())), put(spread(c["b"]))
        gates = torch.zeros(spec.blocks, 2, bs, bs)
        gates[:, 0, :n, :n], gates[:, 1, :n, :n] = c["ra"], c["ri"]
        self.gates = gates.view(spec.blocks, 2 * bs, bs).to(dtype).to(dev)
        self.rb, self.ib = put(spread(c["rab"].flatten())), put(spread(c["rib"].flatten()))
        self.decay = put(spread(8 * torch.log1p(torch.exp(c["lam"].double()))))
        self.state = torch.full((slots, spec.cols), float("nan"), device=dev)       # a new sequence reads none of it
        self.ring = torch.full((slots, spec.taps, spec.cols), float("nan"), device=dev, dtype=dtype)

    def run(self, y, x, table, slots, new=None, fused=False):
        from kinetics_b200 import layer_ops as lo, ops
        proj = torch.cat((y, x), dim=1).to(self.dtype).to(self.dev)
        status, slots = ops.new_status(self.dev), torch.tensor(slots, dtype=torch.int32, device=self.dev)
        kw = dict(new_indptr=None if new is None else torch.tensor([0, new], dtype=torch.int32, device=self.dev),
                  max_new=new or 1, status=status)
        if fused and new is None and lo.lru_decode_supported(self.spec, self.dtype):
            out = lo.lru_decode(proj, self.spec, table, slots, self.w, self.b, self.gates, self.rb, self.ib, self.decay,
                                self.ring, self.state, status)
            ops.raise_on_status(status)
            return out.double().cpu()
        u = lo.lru_conv(proj, self.spec, table, slots, self.w, self.b, self.ring, **kw)
        z = lo.lru_gate_products(u, self.gates, self.spec)
        out = lo.lru_scan(z, u, proj, self.spec, table, slots, self.rb, self.ib, self.decay, self.state, **kw)
        ops.raise_on_status(status)
        return out.double().cpu()


def _length_table(lens, dev, ps=16):
    from kinetics_b200.layer_ops import PageTable
    pages = [(n + ps - 1) // ps for n in lens]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    indptr = [sum(pages[:i]) for i in range(len(lens) + 1)]
    return PageTable(i32(list(range(sum(pages)))), i32(indptr), i32([n - (c - 1) * ps for n, c in zip(lens, pages)]), ps, sum(pages))


@pytest.mark.parametrize("fused", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("blocks,block,taps", [(1, 264, 4), (3, 20, 4), (1, 48, 2), (2, 17, 1), (4, 8, 7), (2, 80, 4), (1, 16, 30)])
def test_recurrence_in_portions(cuda_device, dtype, blocks, block, taps, fused):
    from kinetics_b200.layer_ops import LruSpec
    spec = LruSpec(blocks, block, taps)
    total = 300
    c, spread = _lru_case(spec, total, blocks + taps)
    want = spread(_lru_plain(c, dtype).float()).double()
    y, x = spread(c["y"]), spread(c["x"])
    lru = _Lru(spec, [c], spread, dtype, cuda_device, 4)
    for slot, sizes in enumerate([[300], [2] * 150, [127, 1, 2, 129, 1, 1, 1, 16, 22], [1] * 300]):
        got, at = [], 0
        for n in sizes:
            got.append(lru.run(y[at:at + n], x[at:at + n], _length_table([at + n], cuda_device), [slot], n if n > 1 else None, fused))
            at += n
        err = (torch.cat(got) - want).pow(2).mean(-1).sqrt() / rms(want)
        assert err.max() < (2e-5 if dtype == F32 else 2e-2), (sizes, float(err.max()))


@pytest.mark.parametrize("dtype,fused", [(F32, False), (BF, False), (BF, True)])
def test_recurrence_of_unequal_sequences(cuda_device, dtype, fused):
    # prompts of different lengths, then steps of all of them together in changing order; then a slot is used again
    from kinetics_b200.layer_ops import LruSpec
    spec, lens, steps = LruSpec(2, 24, 4), [1, 2, 5, 70], 40
    cases = []
    for i, n in enumerate(lens + [30]):
        c, spread = _lru_case(spec, 1, 50)                    # the same weights, other inputs
        g = torch.Generator().manual_seed(i)
        c["x"], c["y"] = torch.randn(n + steps, spec.blocks * spec.block, generator=g), torch.randn(n + steps, spec.blocks * spec.block, generator=g)
        cases.append(c)
    lru = _Lru(spec, cases, spread, dtype, cuda_device, 6)
    slot_of, got = [4, 0, 5, 2], [[] for _ in cases]

    def prompt(i, n, slot):
        c = cases[i]
        got[i].append(lru.run(spread(c["y"][:n]), spread(c["x"][:n]), _length_table([n], cuda_device), [slot], n if n > 1 else None))
    for i, n in enumerate(lens):
        prompt(i, n, slot_of[i])
    for t in range(steps):
        order = [(k + t) % 4 for k in range(4)]
        rows = lambda key: torch.cat([spread(cases[i][key][lens[i] + t:lens[i] + t + 1]) for i in order])
        out = lru.run(rows("y"), rows("x"), _length_table([lens[i] + t + 1 for i in order], cuda_device), [slot_of[i] for i in order],
                      None, fused)
        for k, i in enumerate(order):
            got[i].append(out[k:k + 1])
    prompt(4, 30, slot_of[3])
    for i, n in enumerate(lens + [30]):
        want = spread(_lru_plain(cases[i], dtype).float()).double()
        mine = torch.cat(got[i])
        err = (mine - want[:mine.shape[0]]).pow(2).mean(-1).sqrt() / rms(want)
        assert err.max() < (2e-5 if dtype == F32 else 2e-2), (i, float(err.max()))


def test_fused_steps_of_many_sequences_equal_the_separate_ones(cuda_device):
    # more rows than a CTA takes, in permuted slots; some start now
    from kinetics_b200.layer_ops import LruSpec
    dev, g = cuda_device, torch.Generator().manual_seed(0)
    for spec in (LruSpec(2, 40, 4), LruSpec(1, 512, 3), LruSpec(3, 33, 2)):
        rows = 150
        c, spread = _lru_case(spec, rows, 4)
        a, b = (_Lru(spec, [c], spread, BF, dev, rows + 7) for _ in range(2))
        slots = torch.randperm(rows + 7, generator=g)[:rows].tolist()
        for lru in (a, b):
            h = torch.Generator().manual_seed(1)
            lru.state.copy_(torch.randn(lru.state.shape, generator=h))
            lru.ring.copy_(torch.randn(lru.ring.shape, generator=h))
        lens = torch.randint(1, 60, (rows,), generator=g).tolist()
        lens[:5] = [1, 2, 3, 4, 5]
        for step in range(3):
            table = _length_table([n + step for n in lens], dev)
            one, two = (m.run(spread(c["y"]), spread(c["x"]), table, slots, None, f) for m, f in ((a, False), (b, True)))
            torch.testing.assert_close(one, two, rtol=2e-2, atol=2e-3)
        torch.testing.assert_close(a.state, b.state, rtol=1e-3, atol=1e-4)
        assert torch.equal(a.ring, b.ring)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_long_memory_and_short_memory(cuda_device, dtype):
    # decays from "forgets at once" to "keeps for the whole sequence": the series and the difference in sqrt(1 - a^2)
    from kinetics_b200.layer_ops import LruSpec
    spec, total = LruSpec(1, 64, 4), 2000
    c, spread = _lru_case(spec, total, 9)
    c["lam"] = torch.linspace(-14, 4, 64)
    want = _lru_plain(c, dtype)
    got = _Lru(spec, [c], spread, dtype, cuda_device, 1).run(c["y"], c["x"], _length_table([total], cuda_device), [0], total)
    err = (got - want).pow(2).mean(0).sqrt() / want.pow(2).mean(0).sqrt()
    assert err.max() < (1e-4 if dtype == F32 else 3e-2), err


# ---- feed-forward pieces
@pytest.mark.parametrize("dtype", [F32, BF])
def test_gated_rows_and_scale_cap(cuda_device, dtype):
    from kinetics_b200 import layer_ops as lo
    g = torch.Generator().manual_seed(0)
    x = (4 * torch.randn(37, 2 * 88, generator=g)).to(dtype)
    a, b = x[:, :88].double(), x[:, 88:].double()
    tol = dict(rtol=1e-5, atol=1e-5) if dtype == F32 else dict(rtol=1e-2, atol=1e-3)
    got = lo.gated_rows(x.to(cuda_device)).double().cpu()
    torch.testing.assert_close(got, a * plain.sigmoid(a) * b, **tol)
    got = lo.gated_rows(x.to(cuda_device), lo.GateSpec(1.5, 1.702, 1.0)).double().cpu()
    a, b = a.clamp(max=1.5), b.clamp(-1.5, 1.5)
    torch.testing.assert_close(got, a * plain.sigmoid(1.702 * a) * (b + 1), **tol)
    z = 50 * torch.randn(5, 33, generator=g)
    torch.testing.assert_close(lo.scale_cap(z.clone().to(cuda_device), 0.3, 9.0).cpu(), 9 * torch.tanh(z * 0.3 / 9), rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(lo.scale_cap(z.clone().to(cuda_device), 0.3, 0.0).cpu(), z * 0.3)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_experts_with_clamped_gates_and_shares_of_the_whole_softmax(cuda_device, dtype):
    from kinetics_b200 import layer_ops as lo
    from kinetics_b200.layer_ops import GateSpec, MoeSpec
    for rows, E, top, C, F, limit in [(5, 6, 2, 72, 40, 0.8), (300, 16, 3, 256, 64, 2.0), (700, 1, 1, 64, 32, 0.5), (64, 9, 9, 40, 24, 5.0)]:
        g = torch.Generator().manual_seed(rows)
        h = torch.randn(rows, C, generator=g).to(dtype)
        # rows of one direction each: their experts stand far apart, so that rounding decides nothing
        router = (torch.randn(E, C, generator=g) * (3.0 / C ** 0.5)).to(dtype)
        gate, up, down = (torch.randn(E, *s, generator=g).div(s[1] ** 0.5).to(dtype) for s in ((F, C), (F, C), (C, F)))
        spec = MoeSpec(E, top, C, F, score_all=True, gate=GateSpec(limit, 1.702, 1.0))
        d = lambda t: t.to(cuda_device)
        for variant in (0, 1):
            r = lo.moe_route(d(h), d(router), None, spec, variant=variant)
            y = lo.moe_experts(d(h), d(torch.stack((gate, up), dim=2).contiguous()), d(down), r, spec, variant=variant)
            ids, weights = plain.route(h.double(), router.double(), top)
            got_ids, got_w = r.ids.long().cpu(), r.weights.double().cpu()
            same = (got_ids == ids).all(dim=1)
            assert same.double().mean() > (0.999 if dtype == F32 else 0.97)
            torch.testing.assert_close(got_w[same], weights[same], rtol=1e-4, atol=1e-5)
            want = torch.zeros(rows, C).double()
            for e in range(E):
                at, place = (got_ids == e).nonzero(as_tuple=True)
                if at.numel():
                    part = plain.expert(h[at].double(), gate[e].double(), up[e].double(), down[e].double(), limit)
                    want[at] += got_w[at, place].unsqueeze(1) * part
            err = (y.double().cpu().sum(dim=1) - want).pow(2).mean(-1).sqrt() / rms(want)
            assert err.max() < (1e-5 if dtype == F32 else 2e-2), float(err.max())


def test_stream_without_norms_in_front(cuda_device):
    from kinetics_b200 import layer_ops as lo, ops
    g = torch.Generator().manual_seed(1)
    rows, C, eps = 9, 72, 1e-3
    table, tokens = torch.randn(50, C, generator=g), torch.randint(0, 50, (rows,), generator=g)
    w, y = torch.randn(C, generator=g), torch.randn(rows, 3, C, generator=g)
    dev = cuda_device
    for dtype in (F32, BF):
        x, h, status = torch.empty(rows, C, device=dev), torch.empty(rows, C, dtype=dtype, device=dev), ops.new_status(dev)
        lo.residual_norm(x, h, C, eps, tokens=tokens.to(dev), embed=table.to(dtype).to(dev), embed_scale=2.5, center=False, status=status)
        want = table.to(dtype)[tokens].double() * 2.5
        torch.testing.assert_close(x.double().cpu(), want, rtol=1e-6, atol=1e-6)
        assert torch.equal(h, x.to(dtype))
        lo.residual_norm(x, h, C, eps, y=y.to(dtype).to(dev), parts=3, post=(w.to(dev), None), center=False, status=status)
        want = want + plain.rms_norm(y.to(dtype).double().sum(1), w.double(), eps)
        torch.testing.assert_close(x.double().cpu(), want, rtol=1e-5, atol=1e-5)
        assert torch.equal(h, x.to(dtype))
        ops.raise_on_status(status)
