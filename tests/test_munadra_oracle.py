"""The plain Munadra restatement itself, the configuration reader, the packed weights and the cache manager's host side.
No GPU."""
import math

import pytest
import torch

from latent_helpers import as_dtype, dense, latent, moe, random_model, rglru, rot, small_config
from oracle import munadra as plain


def _model(seed=3):
    raw = small_config()
    return raw, as_dtype(random_model(raw, seed), torch.float64)


def _tokens(n, vocab, seed=1):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))


def test_portions_and_single_tokens_equal_the_whole_prompt():
    raw, W = _model()
    tokens = _tokens(70, raw["vocab"])
    whole = plain.forward(tokens, W, raw)
    for sizes in ([1] * 70, [2] * 35, [33, 1, 16, 20]):
        hist, out, at = plain.History(len(raw["layers"])), [], 0
        for n in sizes:
            out.append(plain.forward(tokens[at:at + n], W, raw, hist))
            at += n
        torch.testing.assert_close(torch.cat(out), whole, rtol=1e-9, atol=1e-9)


def test_later_tokens_do_not_change_earlier_logits():
    raw, W = _model()
    a = _tokens(40, raw["vocab"])
    b = a.clone()
    b[25:] = (b[25:] + 1) % raw["vocab"]
    x, y = plain.forward(a, W, raw), plain.forward(b, W, raw)
    torch.testing.assert_close(x[:25], y[:25])
    assert (x[25:] - y[25:]).abs().amin(dim=1).max() > 0 and (x[39] - y[39]).abs().max() > 1e-3


@pytest.mark.parametrize("change", ["sink", "gate", "conv", "ramp", "source"])
def test_every_mechanism_shows_in_the_logits(change):
    raw, W = _model()
    tokens = _tokens(50, raw["vocab"])
    whole, W2 = plain.forward(tokens, W, raw), dict(W)
    if change == "sink":
        W2["l0.mix.sink"] = W["l0.mix.sink"] - 50
    elif change == "gate":
        W2["l2.mix.g"] = -W["l2.mix.g"]
    elif change == "conv":
        W2["l1.mix.conv"] = W["l1.mix.conv"].flip(1)
    elif change == "ramp":
        raw = small_config()
        for l in (0, 3):
            del raw["layers"][l]["mixer"]["rot"]["scaling"]
    else:
        raw = small_config()
        raw["layers"][3]["mixer"]["rot"] = rot(16, base=77.0)      # its queries only: the keys lie in layer 0's rows
    assert (plain.forward(tokens, W2, raw)[10:] - whole[10:]).pow(2).mean().sqrt() > 1e-2


def test_rotation_keeps_relative_positions_and_the_stretch_changes_slow_pairs_only():
    g = torch.Generator().manual_seed(0)
    for r in (rot(16, base=100.0), rot(16, base=1000.0, factor=4.0, original=100, fast=10.0, slow=1.0)):
        q, k = torch.randn(1, 16, generator=g).double(), torch.randn(1, 16, generator=g).double()
        at = lambda x, p: plain.rotate(x, torch.tensor([p]), r)
        assert float((at(q, 7) * at(k, 3)).sum()) == pytest.approx(float((at(q, 104) * at(k, 100)).sum()))
    from kinetics_b200.layer_ops import Rotation
    slow, _ = plain.rotary_frequencies(rot(16, base=1000.0, factor=4.0, original=100, fast=10.0, slow=1.0))
    flat, one = plain.rotary_frequencies(rot(16, base=1000.0))
    assert one == 1.0 and slow[0] == flat[0] and slow[-1] == pytest.approx(flat[-1] / 4)
    for args in (dict(), dict(factor=4.0, original=100, fast=10.0, slow=1.0), dict(factor=1.5, original=9, fast=64.0, slow=0.1),
                 dict(factor=32.0, original=4096, fast=32.0, slow=1.0)):
        spec = Rotation(16, 1000.0, scaled=bool(args), **args)
        want, factor = plain.rotary_frequencies(rot(16, base=1000.0, **args))
        torch.testing.assert_close(spec.frequencies().double(), torch.tensor(want).double(), rtol=1e-6, atol=0)
        assert spec.amplitude == pytest.approx(factor)


def test_sink_takes_its_share_once():
    s = torch.tensor([[0.0, 1.0, 5.0]])
    p = plain.sink_softmax(s, torch.tensor(2.0), 1)                # the third key is not seen
    total = 1 + math.e + math.e ** 2
    torch.testing.assert_close(p, torch.tensor([[1 / total, math.e / total, 0.0]]))


def test_configuration():
    from kinetics_b200 import Munadra, model_class
    from kinetics_b200.layer_ops import LatentSpec, LruSpec
    raw = small_config()
    assert model_class(raw) is Munadra
    c = Munadra.from_config(raw)
    assert (c.vocab, c.width, c.norm_eps, c.embed_scale, c.logit_scale, c.logit_softcap) == (93, 72, 1e-5, 1.7, 0.3, 9.0)
    a, r, b, shared, last = c.layers
    assert a.mixer == LatentSpec(3, 24, 16, 40, 56, 40 ** -0.5, a.mixer.rotation, 1e-5, None) and a.mixer.rotation.factor == 4.0
    assert r.mixer == LruSpec(3, 20, 4) and (r.ff, r.experts) == (88, 0) and r.moe(72) is None
    assert b.ff == 0 and not b.mixer.rotation.scaled and b.mixer.rotation.base == 500.0
    assert shared.mixer.kv_from == 0 and shared.moe(72).score_all and shared.moe(72).gate == (type(a.moe(72).gate))(0.7, 1.702, 1.0)
    assert last.mixer == LruSpec(1, 48, 2) and last.top == 1

    def broken(i, path, value):
        bad = small_config()
        at = bad["layers"][i]
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ValueError):
            Munadra.from_config(bad)
    broken(0, ["type"], "attention")
    broken(1, ["mixer", "blocks"], 7)
    broken(3, ["mixer", "kv_from"], 2)                             # other sizes
    broken(3, ["mixer", "kv_from"], 1)                             # a recurrence
    broken(3, ["mixer", "kv_from"], 4)                             # a later layer
    broken(0, ["mlp", "router", "top"], 6)
    broken(0, ["mlp", "kind"], "wide")
    broken(0, ["mixer", "rot", "dims"], 8)
    chain = small_config()
    chain["layers"].append(latent(2, 8, 16, 8, 56, None, kv_from=3, factor=4.0))
    with pytest.raises(ValueError):                                # layer 3 has no cache of its own
        Munadra.from_config(chain)


def test_packed_weights():
    from kinetics_b200 import Munadra
    raw = small_config([latent(2, 12, 6, 20, 30, dense(18)), rglru(22, 2, 3, moe(3, 2, 10)),
                        latent(1, 5, 6, 9, 30, None, kv_from=0)], width=30, vocab=41)
    W = random_model(raw)
    m = Munadra(Munadra.from_config(raw), W, "cpu", torch.float32)
    a, r, s = m.layers
    f = lambda n: W[n].float()
    assert tuple(a["proj"].shape) == (2 * (16 + 8) + (32 + 8) + 8, 32) and tuple(s["proj"].shape) == (8 + 8 + 8, 32)
    q = a["proj"][:48].view(2, 24, 32)
    assert torch.equal(q[:, :12, :30].reshape(24, 30), f("l0.mix.q").view(2, 18, 30)[:, :12].reshape(24, 30))
    assert torch.equal(q[:, 16:22, :30], f("l0.mix.q").view(2, 18, 30)[:, 12:]) and q[:, 22:].abs().max() == 0
    assert torch.equal(a["proj"][48:78, :30], f("l0.mix.dkv")[:30]) and torch.equal(a["proj"][80:86, :30], f("l0.mix.dkv")[30:])
    assert torch.equal(a["proj"][88:90, :30], f("l0.mix.g")) and torch.equal(s["proj"][16:17, :30], f("l2.mix.g"))
    assert torch.equal(a["mix"].uk[:, :12, :30].reshape(24, 30), f("l0.mix.uk"))
    assert torch.equal(a["mix"].uv[:, :20, :30].reshape(40, 30), f("l0.mix.uv")) and s["mix"].norm is None
    assert torch.equal(a["norm1"][0][:30], 1 + f("l0.norm1")) and a["norm1"][0][30:].abs().max() == 0
    assert torch.equal(a["dense"][24:42, :30], f("l0.mlp.up")) and torch.equal(a["dense_down"][:30, :18], f("l0.mlp.down"))
    gates = r["mix"].gates.view(2, 2, 16, 16)
    assert torch.equal(gates[:, 1, :11, :11], f("l1.mix.ri")) and gates[:, :, 11:].abs().max() == 0
    assert torch.equal(r["mix"].conv_w.view(3, 2, 16)[:, :, :11].reshape(3, 22).t(), f("l1.mix.conv"))
    decay = r["mix"].decay.view(2, 16)[:, :11].reshape(22)
    torch.testing.assert_close(decay, 8 * torch.nn.functional.softplus(f("l1.mix.lam")), rtol=1e-5, atol=1e-7)
    assert torch.equal(r["proj"].view(2, 2, 16, 32)[1, :, :11, :30].reshape(22, 30), f("l1.mix.x"))
    assert torch.equal(r["out"].view(32, 2, 16)[:30, :, :11].reshape(30, 22), f("l1.mix.o"))
    for name in ("l0.mix.q", "l0.mix.dkv", "l0.mix.uk", "l0.mix.sink", "l1.mix.ra", "l1.mix.conv", "l1.mix.lam", "l1.mlp.router",
                 "l0.mlp.up", "embed", "final.norm"):
        bad = dict(W)
        bad[name] = torch.zeros(5, 7, dtype=torch.bfloat16)
        with pytest.raises((ValueError, RuntimeError)):
            Munadra(Munadra.from_config(raw), bad, "cpu", torch.float32)


def test_caches_and_states_of_the_manager():
    from kinetics_b200 import LayeredKVManager, Munadra
    c = Munadra.from_config(small_config())
    kv = LayeredKVManager([l.mixer for l in c.layers], 3, 100, "cpu", torch.bfloat16, num_pages=9, page_size=16)
    assert tuple(kv.k_pages[0].shape) == (9, 1, 16, 56 + 16) and kv.k_pages[3] is kv.k_pages[0] and kv.k_pages[2] is not kv.k_pages[0]
    assert kv.k_pages[1] is None and tuple(kv.states[1].shape) == (3, 72) and kv.states[1].dtype == torch.float32
    assert tuple(kv.rings[1].shape) == (3, 4, 72) and kv.rings[4].dtype == torch.bfloat16 and kv.states[0] is None
    kv.admit(1, 0, 40)
    assert kv.pool.free_pages == 6
    kv.clear_cache(1)
    assert kv.pool.free_pages == 9
