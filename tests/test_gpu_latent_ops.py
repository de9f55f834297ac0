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
