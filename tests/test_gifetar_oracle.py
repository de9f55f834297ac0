"""The plain Gifetar restatement itself, the configuration and weight reader, and the command line's host side.  No
GPU."""
import json
import math

import pytest
import torch

from layer_helpers import as_dtype, layer_entry, random_model, small_config, standout_inputs
from oracle import gifetar as plain


def _model(seed=3):
    raw = small_config()
    return raw, as_dtype(random_model(raw, seed), torch.float64)


def test_portions_and_single_tokens_equal_the_whole_prompt():
    raw, W = _model()
    tokens = torch.randint(0, raw["vocab"], (70,), generator=torch.Generator().manual_seed(1))
    whole = plain.forward(tokens, W, raw)
    for sizes in ([1] * 70, [2] * 35, [33, 1, 16, 20]):
        hist, out, at = plain.History(len(raw["layers"])), [], 0
        for n in sizes:
            out.append(plain.forward(tokens[at:at + n], W, raw, hist))
            at += n
        torch.testing.assert_close(torch.cat(out), whole, rtol=1e-9, atol=1e-9)


def test_later_tokens_do_not_change_earlier_logits():
    raw, W = _model()
    tokens = torch.randint(0, raw["vocab"], (40,), generator=torch.Generator().manual_seed(2))
    other = tokens.clone()
    other[25:] = (other[25:] + 7) % raw["vocab"]
    a, b = plain.forward(tokens, W, raw), plain.forward(other, W, raw)
    torch.testing.assert_close(a[:25], b[:25], rtol=1e-10, atol=1e-10)
    assert (a[25:] - b[25:]).abs().max() > 1e-3


def test_temperature_steps_where_position_plus_one_reaches_a_multiple():
    t = plain.query_temperature(torch.arange(0, 33), 0.5, 16)
    assert torch.equal(t[:15], torch.ones(15, dtype=torch.float64))
    assert t[15] == pytest.approx(1 + 0.5 * math.log(2)) and t[30] == t[15]
    assert t[31] == pytest.approx(1 + 0.5 * math.log(3))


def test_one_standing_out_key_decides_the_output():
    # with one visible key far above the others, each map returns that key's value: the inputs of the kernel tests do
    # show a missing or a superfluous key
    q, k, v = standout_inputs(90, 0, 2, 1, 32, 24, [0, 1, 15, 16, 63, 64, 88, 89], seed=5, strength=7.0)
    mixer = {"q_temp": {"coef": 0.0, "every": 1.0}, "scale": 0.4, "softcap": 30.0, "diff": 0.2}
    base = plain.difference_attention(q, k, v, mixer, 0.4, 1e-6)
    for gone in (0, 64, 89):
        k2 = k.clone()
        k2[gone] = 0
        changed = (plain.difference_attention(q, k2, v, mixer, 0.4, 1e-6) - base).abs().amax(dim=(1, 2))
        assert (changed[gone:] > 0.5).any(), gone
        assert gone == 0 or changed[:gone].max() < 1e-6


def test_routing_weights_are_the_softmax_over_the_chosen():
    h = torch.randn(9, 12, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    w = torch.randn(6, 12, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    b = torch.tensor([0.0, 30.0, 0.0, 0.0, -30.0, 0.0], dtype=torch.float64)
    ids, weights = plain.route(h, w, b, 3)
    z = h @ w.t() + b
    assert (ids[:, 0] == 1).all() and not (ids == 4).any()          # the bias takes part in the choice
    for r in range(9):
        e = torch.exp(z[r, ids[r]])
        torch.testing.assert_close(weights[r], e / e.sum())


def test_config_reader_takes_every_size_and_refuses_what_it_does_not_know():
    from kinetics_b200 import Gifetar, model_class
    raw = small_config()
    assert model_class(raw) is Gifetar
    c = Gifetar.from_config(raw)
    assert (c.vocab, c.width, c.norm_eps, c.residual_mult) == (101, 72, 1e-5, 0.4)
    assert [l.heads for l in c.layers] == [4, 3, 2, 8] and [l.experts for l in c.layers] == [5, 0, 3, 7]
    assert c.layers[0].temp_every == 16 and c.layers[1].softcap == 80.0
    with pytest.raises(KeyError):
        model_class({"architecture": "other"})
    for bad in ({"type": "recurrent"}, {"mlp": {"kind": "dense"}},
                {"mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 2, "top": 3}}}):
        e = {**layer_entry(2, 1, 8, 8, experts=0), **bad}
        with pytest.raises(ValueError):
            Gifetar.from_config({**raw, "layers": [e]})
    with pytest.raises(ValueError):
        Gifetar.from_config({**raw, "layers": [layer_entry(3, 2, 8, 8, experts=0)]})


def test_model_weights_are_padded_with_zeros_and_shapes_are_checked():
    # the loader only moves tensors: it runs on the CPU (no kernel does)
    from kinetics_b200 import Gifetar
    raw = small_config([layer_entry(2, 1, 12, 20, experts=3, top=2, ff=18)], width=30)
    W = random_model(raw)
    m = Gifetar(Gifetar.from_config(raw), W, "cpu", torch.float32)
    L = m.layers[0]
    assert tuple(L["wqkv"].shape) == (2 * 2 * 16 + 2 * 16 + 24, 32)
    q = L["wqkv"][:64].view(4, 16, 32)
    assert torch.equal(q[:, :12, :30].reshape(48, 30), W["l0.mix.q"].float())
    assert q[:, 12:].abs().max() == 0 and q[:, :, 30:].abs().max() == 0
    wo = L["wo"].view(32, 2, 24)
    assert torch.equal(wo[:30, :, :20].reshape(30, 40), W["l0.mix.o"].float()) and wo[30:].abs().max() == 0
    assert torch.equal(L["gate_up"][1, :18, 1, :30], W["l0.mlp.e1.up"].float())
    assert torch.equal(L["down"][2, :30, :18], W["l0.mlp.e2.down"].float())
    lam = plain.difference_weight(*(W["l0.mix." + n].double() for n in ("lq1", "lk1", "lq2", "lk2")), 0.3)
    assert L["spec"].lam == pytest.approx(float(lam)) and L["spec"].out_scale == pytest.approx(0.7)
    for name in ("l0.mix.k", "embed", "l0.norm1.b", "l0.mlp.router", "l0.mlp.e1.down", "l0.mix.o"):
        broken = dict(W)
        broken[name] = torch.zeros(5, 7, dtype=torch.bfloat16)
        with pytest.raises((ValueError, RuntimeError)):
            Gifetar(Gifetar.from_config(raw), broken, "cpu", torch.float32)
    with pytest.raises(TypeError):
        Gifetar(Gifetar.from_config(raw), W, "cpu", torch.float16)


def test_safetensors_round_trip(tmp_path):
    from kinetics_b200.checkpoint import Checkpoint, save
    tensors = {"a": torch.randn(3, 5).to(torch.bfloat16), "n": torch.arange(7, dtype=torch.int32),
               "empty": torch.zeros(0, 4), "f": torch.randn(2, 2, 2)}
    save(tmp_path / "x.safetensors", tensors)
    c = Checkpoint(tmp_path / "x.safetensors")
    assert sorted(c.names()) == sorted(tensors) and "a" in c and "b" not in c
    for k, v in tensors.items():
        assert torch.equal(c[k], v) and c[k].dtype == v.dtype
    assert c.unread() == []
    with pytest.raises(KeyError):
        c["b"]
    raw = bytearray((tmp_path / "x.safetensors").read_bytes())
    (tmp_path / "cut.safetensors").write_bytes(raw[:-4])
    with pytest.raises(ValueError):
        Checkpoint(tmp_path / "cut.safetensors")


def test_load_model_reads_the_folder_and_refuses_unknown_tensors(tmp_path):
    from kinetics_b200 import load_model
    from kinetics_b200.checkpoint import save
    raw = small_config([layer_entry(2, 2, 8, 16, experts=0)], width=24)
    W = random_model(raw)
    (tmp_path / "config.json").write_text(json.dumps(raw))
    save(tmp_path / "model.safetensors", W)
    m = load_model(tmp_path, "cpu", torch.bfloat16)
    assert m.config.width == 24 and torch.equal(m.embed, W["embed"])
    save(tmp_path / "model.safetensors", {**W, "l9.norm1": torch.zeros(3)})
    with pytest.raises(ValueError):
        load_model(tmp_path, "cpu", torch.bfloat16)


def test_layered_manager_bookkeeping_on_the_host():
    # pages, lengths and page tables without a kernel: sequences grow, retire, and their pages serve others
    from kinetics_b200 import LayeredKVManager, PoolExhausted
    from kinetics_b200.layer_ops import AttentionSpec
    specs = [AttentionSpec(4, 2, 24, 40, 0.1, maps=2), AttentionSpec(2, 1, 8, 8, 0.1, maps=2)]
    kv = LayeredKVManager(specs, 3, 200, "cpu", torch.float32, num_pages=8, page_size=16)
    assert tuple(kv.k_pages[0].shape) == (8, 4, 16, 24) and tuple(kv.v_pages[1].shape) == (8, 1, 16, 8)
    assert kv.can_admit(128) and not kv.can_admit(129)
    kv.admit(0, 0, 40)
    kv.admit(1, 0, 0)
    assert kv.pool.free_pages == 5
    kv.promise(1, 17)
    assert kv.pool.free_pages == 3
    kv.promise(1, 5)                                       # a smaller promise changes nothing
    assert kv.pool.free_pages == 3
    with pytest.raises(PoolExhausted):
        kv.promise(1, 17 + 4 * 16)
    kv.pool.extend([1], 17)
    assert kv.pool.pages(1) == 2
    kv.clear_cache(1)
    assert kv.pool.free_pages == 5
    kv.clear_cache(2)                                      # a free slot: nothing to do
    with pytest.raises(ValueError):
        kv.promise(0, 201)


def test_engine_extends_a_slot_in_portions_with_a_stand_in_model():
    from kinetics_b200 import Engine

    class KV:
        max_batch_size = 2

        def __init__(self):
            self.log = []

        def clear_cache(self, slot):
            self.log.append(("clear", slot))

        def promise(self, slot, total):
            self.log.append(("promise", slot, total))

    class Model:
        def __init__(self):
            self.calls = []

        def inference(self, ids, pos, batch_idx, kv, rows=None):
            self.calls.append((ids[0].tolist(), pos[0].tolist(), rows))
            return torch.zeros(1, len(rows), 4)

    kv, model = KV(), Model()
    eng = Engine(model, kv, 16, "cpu")
    eng.open_slot(1)
    with pytest.raises(ValueError):
        eng.open_slot(1)
    with pytest.raises(ValueError):
        eng.extend(0, [1])
    assert eng.extend(1, [4, 5, 6], []) is None
    assert tuple(eng.extend(1, [7, 8], [0, 1]).shape) == (2, 4)
    assert model.calls == [([4, 5, 6], [0, 1, 2], []), ([7, 8], [3, 4], [0, 1])]
    assert eng.slots_tokens[1, :5].tolist() == [4, 5, 6, 7, 8] and int(eng.slots_offsets[1]) == 5
    with pytest.raises(ValueError):
        eng.extend(1, [0] * 12)
    eng.clear_request(1)
    assert kv.log == [("promise", 1, 3), ("promise", 1, 5), ("clear", 1)]


def test_header_and_binding_of_the_layer_library_agree():
    import ctypes
    import re
    from pathlib import Path

    from kinetics_b200 import _lib
    text = (Path(__file__).resolve().parent.parent / "include" / "ktk_layers.h").read_text()
    declared = sorted(set(re.findall(r"KTK_API\s+[\w\s\*]+?\b(ktk_\w+)\s*\(", text)))
    assert declared == sorted(_lib.LAYERS_EXPORTED)
    lib = _lib.load_layers()
    for name in declared:
        assert hasattr(lib, name)
    # argument errors come back from the host before anything is launched
    one, null = ctypes.c_void_p(16), ctypes.c_void_p(0)
    a = _lib.Attn(4, 3, 2, 8, 8, 8, 8, 1, 1.0, 0.0, 0.0, 1.0, 0.0, 0.0, 1.0)
    t = _lib.Paged(16, 16, 16, 1, 16, 4)
    call = lambda: lib.ktk_paged_attention(one, 64, null, 1, 1, one, one, ctypes.byref(t), null, null, 0, one,
                                           null, 0, 1, 0, ctypes.byref(a), null, null)
    assert call() == -1                                    # 4 heads over 3 kv heads
    a.kv_heads = 2
    t.page_size = 24
    assert call() == -2 and b"page_size" in lib.ktk_last_error()
    m = _lib.Moe(4, 5, 8, 8, 8, 8, 1, 0)
    assert lib.ktk_moe_route(one, one, one, one, one, one, one, 1, ctypes.byref(m), 0, null) == -1
    assert lib.ktk_residual_norm(null, null, 0, 1.0, one, null, 1, null, null, 1.0, null, null, null, 1e-6, 1, 1, 12, 12, null,
                                 0, 1, null, null) == -1   # a stride of 12


def test_command_line_without_a_device_says_so(capsys):
    if torch.cuda.is_available():
        pytest.skip("a device is here")
    from kinetics_b200 import cli
    assert cli.main(["generate", "--model", "x", "--prompt", "1,2"]) == 1
    assert "CUDA" in capsys.readouterr().err
    assert cli._ids("5, 17 3") == [5, 17, 3]
    with pytest.raises(SystemExit):
        cli.main(["trace", "--model", "x"])
