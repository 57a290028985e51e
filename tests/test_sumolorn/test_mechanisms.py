"""Every mechanism of the Sumolorn family alone: the framework's module on the framework's step runtime (sm_100a kernels on
the `gpu` tier, their PyTorch paths on the plumbing tier) against the float64 oracle's function of the same mechanism.
Inputs and weights are made so that a fault shows: a key that one query singles out among hundreds, keys just inside and just
outside the window and on a page's border, scores far beyond the soft cap, sink scores that outweigh the keys, decays of
almost one and almost zero, portions shorter than the convolution, widths that take the scalar paths."""
import math

import pytest
import torch

from colossalai_b200.inference.modeling.kv_runtime import PagedKVRuntime
from colossalai_b200.models.config import LayerSpec, MixerSpec, ModelConfig
from colossalai_b200.models.mixers import build_mixer
from colossalai_b200.models.sumolorn import SumolornForCausalLM, convert_sumolorn_state_dict, sumolorn_config
from colossalai_b200.ops import mixers as M

from . import oracle as O

TIERS = ["plumbing", pytest.param("gpu", marks=pytest.mark.gpu)]
F64 = torch.float64
BS = 8           # page size of the scratch runtime
WIDTH = 40
EPS = 1e-5


def _dev(tier):
    if tier == "gpu" and not torch.cuda.is_available():
        pytest.skip("needs a CUDA device")
    return "cuda" if tier == "gpu" else "cpu"


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def _close(got, want, tol):
    err = (got.double().cpu() - want).abs().max().item() / max(want.abs().max().item(), 1e-30)
    assert err < tol, f"relative error {err:.3e}"


def _layer(layer, dev, width=WIDTH, seed=0, edit=None, dtype=torch.float32):
    """One-layer model of `layer`: (framework layer module, its config, oracle weights, mixer section of the config)."""
    hf = O.make_config([layer], width=width)
    W = O.random_weights(hf, seed=seed)
    if edit:
        edit(W)
        W = {k: v.to(torch.bfloat16).float() for k, v in W.items()}
    model = SumolornForCausalLM(sumolorn_config(hf, {k: tuple(v.shape) for k, v in W.items()}))
    missing, unexpected = model.load_state_dict(convert_sumolorn_state_dict(W, model), strict=False)
    assert not missing and not unexpected
    return model.to(dtype).to(dev).eval().model.layers[0], model.cfg, O.to64(W), layer["mixer"]


def _steps(mixer, cfg, h, cuts, dev, dtype=torch.float32, batch_with=None):
    """Run h [L, width] through the mixer in portions of the given sizes on a scratch runtime (pages of BS tokens, two
    slots; the sequence under test sits in slot 1 and its pages are handed out back to front).  `batch_with`: another
    sequence's input that shares every step (a fresh one-step prompt each time)."""
    L = h.shape[0]
    rt = PagedKVRuntime.scratch(cfg, 2, L + 64, dev, dtype, block_size=BS)
    for st in rt.states:                                   # recycled slots are never cleared: leave rubbish in them
        for t in (st or {}).values():
            t.fill_(3.0)
    per = (L + 64 + BS - 1) // BS
    tables = torch.stack([torch.arange(per, dtype=torch.int32), torch.arange(2 * per - 1, per - 1, -1, dtype=torch.int32)])
    out, at = [], 0
    with torch.inference_mode():
        for n in cuts:
            if batch_with is not None:
                rt.set_ragged_step(tables, [batch_with.shape[0], n], [0, at], [0, 1], dev)
                x = torch.cat([batch_with, h[at:at + n]]).to(dev).to(dtype)
                out.append(mixer(x, None, None, rt)[batch_with.shape[0]:])
            else:
                rt.set_ragged_step(tables[1:], [n], [at], [1], dev)
                out.append(mixer(h[at:at + n].to(dev).to(dtype), None, None, rt))
            at += n
    assert at == L
    return torch.cat(out)


def _cuts(L, sizes):
    out, at = [], 0
    for n in sizes:
        n = min(n, L - at)
        if n > 0:
            out.append(n)
            at += n
    return out + [1] * (L - at)


CUTS = lambda L: ([L], [1] * L, _cuts(L, [2, 3, 2, 9, 1, 1, 17, 2, 40]), _cuts(L, [L - 3]))


# ------------------------------------------------------------------------------------------------ capped windowed attention
def _tie(W, p, conv=False):
    """Query heads read what their key head reads: a query stands out against the key made from the same input."""
    d = W[p + "q"].shape[0]
    for n in ("", ".conv") if conv else ("",):
        k = W[p + "k" + n]
        W[p + "q" + n] = k.repeat(-(-d // k.shape[0]), 1)[:d].clone()


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("window,probe", [(20, 41), (20, 40), (BS + 1, 52), (BS, 52), (1, 60), (2, 59), (100, 0), (61, 0), (60, 0)])
def test_capped_attention_at_the_window_edges(tier, window, probe):
    """The last query (position 60) repeats the input of position `probe`, whose key outscores all others IF the window lets
    the query see it.  Raw scores go far beyond the cap; one head's sink outweighs every key, one has none to speak of."""
    dev = _dev(tier)
    L = 61
    layer = O.attention_layer(heads=4, kv_heads=1, dim=16, vdim=24, scale=1.0, cap=6.0, window=window, rot_dims=4)

    def edit(W):
        _tie(W, "l0.mix.")
        W["l0.mix.sink"] = torch.tensor([-8.0, 0.5, 7.0, 3.0])
    mod, cfg, W, mx = _layer(layer, dev, seed=1, edit=edit)
    h = _rand(L, WIDTH, seed=2)
    h[L - 1] = h[probe]
    h[L - 1] *= 1.5
    ref = lambda z: O.attention(z.to(F64), W, "l0.mix.", mx, range(L))
    want = ref(h)
    for cuts in CUTS(L):
        _close(_steps(mod.self_attn, cfg, h, cuts, dev), want, 3e-5)
    _close(_steps(mod.self_attn, cfg, h, _cuts(L, [5, 30]), dev, batch_with=_rand(19, WIDTH, seed=3)), want, 3e-5)
    if probe < L - 1:                                   # the probe decides the last row exactly when it is visible
        z = h.clone()
        z[probe] = -z[probe]
        moved = (ref(z)[-1] - want[-1]).abs().max()
        assert (moved > 1e-2) if L - 1 - probe < window else (moved == 0)


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("kw", [dict(heads=1, kv_heads=1, dim=8, vdim=40, rot_dims=8), dict(heads=3, kv_heads=3, dim=24, vdim=8, rot_dims=2),
                                dict(heads=6, kv_heads=2, dim=10, vdim=7, rot_dims=6), dict(scaling=None, cap=0.5),
                                dict(scaling=(8.0, 1.0, 2.0, 16), cap=40.0)])
def test_capped_attention_sizes(tier, kw):
    dev = _dev(tier)
    L = 45
    mod, cfg, W, mx = _layer(O.attention_layer(window=11, **kw), dev, seed=3)
    h = _rand(L, WIDTH, seed=4)
    want = O.attention(h.to(F64), W, "l0.mix.", mx, range(L))
    for cuts in CUTS(L):
        got = _steps(mod.self_attn, cfg, h, cuts, dev)
        _close(got[:5], want[:5], 3e-5)
        _close(got, want, 3e-5)


@pytest.mark.parametrize("tier", TIERS)
def test_rotary_frequencies_by_wavelength(tier):
    """Waves that stay, waves that are slowed down and waves between; both pair layouts, vector and scalar widths."""
    dev = _dev(tier)
    regimes = set()
    for dims, base, sc in [(16, 1e4, (4.0, 1.0, 4.0, 64)), (32, 5e4, (2.0, 2.0, 8.0, 512)), (8, 100.0, None), (4, 1e3, (8.0, 1.0, 1.5, 32))]:
        rot = O._rot(dims, base, sc)
        for i in range(dims // 2 if sc else 0):
            turns = sc[3] * base ** (-2.0 * i / dims) / (2 * math.pi)
            regimes.add("stay" if turns > sc[2] else "slow" if turns < sc[1] else "between")
        pos = torch.tensor([0, 1, 2, 300, 1023, 4000])
        table = M.rotary_table(4001, dims, base, dev, ["wavelength", *sc] if sc else None)
        for width, off in ((dims + 3, 1), (dims + 8, 8)):
            x = _rand(6, 2, off + width, seed=dims).to(F64)
            src = x.float().reshape(6, -1).to(dev)
            for pairs in (False, True):
                dst = torch.zeros(6, 2 * width, device=dev)
                M.rotary_half(src, dst, 2, off + width, off, width, 0, width, dims, table, pos.to(torch.int32).to(dev),
                              interleaved=pairs)
                _close(dst.view(6, 2, width), O.rotate(x[:, :, off:], pos, rot, pairs), 2e-5)
    assert regimes == {"stay", "slow", "between"}


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("probe", [3, 3 * BS, 4 * BS - 1, 348])
def test_latent_attention_finds_a_far_key(tier, probe):
    """350 positions; queries read the input with its halves swapped, and the last input is that of position `probe` with its
    halves swapped: its query's unrotated part equals that position's key, which outscores the other 349 (its own included)."""
    dev = _dev(tier)
    L = 350
    layer = O.latent_layer(heads=3, dim=16, rot_dim=8, vdim=12, kv_rank=16, q_rank=16, scale=0.5)

    def edit(W):
        p = "l0.mix."
        W[p + "dq"], W[p + "dq.norm"] = W[p + "dkv"][:16].roll(WIDTH // 2, 1), W[p + "dkv.norm"].clone()
        uq = W[p + "uq"].view(3, 24, 16)
        uq[:, :16] = W[p + "uk"].view(3, 16, 16)
        uq[:, 16:] *= 0.3
        W[p + "sink"] = torch.tensor([-2.0, 0.5, 9.0])
    mod, cfg, W, mx = _layer(layer, dev, seed=5, edit=edit)
    h = _rand(L, WIDTH, seed=6)
    h[L - 1] = h[probe].roll(WIDTH // 2)
    ref = lambda z: O.latent_attention(z.to(F64), W, "l0.mix.", mx, EPS, range(L))
    want = ref(h)
    for cuts in ([L], _cuts(L, [L - 30]), _cuts(L, [2, 130, 2, 180, 7])):
        _close(_steps(mod.self_attn, cfg, h, cuts, dev), want, 3e-5)
    _close(_steps(mod.self_attn, cfg, h, _cuts(L, [1, 2, 300]), dev, batch_with=_rand(9, WIDTH, seed=3)), want, 3e-5)
    z = h.clone()
    z[probe] = -z[probe]
    assert (ref(z)[-1] - want[-1]).abs().max() > 1e-2


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("kw", [dict(heads=1, dim=8, rot_dim=4, vdim=40, kv_rank=40, q_rank=8), dict(heads=5, dim=12, rot_dim=6, vdim=7, kv_rank=19, q_rank=21),
                                dict(heads=2, dim=24, rot_dim=16, vdim=8, kv_rank=8, q_rank=64), dict(heads=2, dim=16, rot_dim=2, vdim=16, kv_rank=264)])
def test_latent_attention_sizes(tier, kw):
    dev = _dev(tier)
    L = 37
    mod, cfg, W, mx = _layer(O.latent_layer(**kw), dev, seed=7)
    h = _rand(L, WIDTH, seed=8)
    want = O.latent_attention(h.to(F64), W, "l0.mix.", mx, EPS, range(L))
    for cuts in CUTS(L):
        got = _steps(mod.self_attn, cfg, h, cuts, dev)
        _close(got[:5], want[:5], 3e-5)
        _close(got, want, 3e-5)


# ------------------------------------------------------------------------------------------------ convolved attention
@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("window,probe,conv", [(20, 41, 3), (20, 40, 3), (BS, 53, 2), (BS, 52, 2), (1, 60, 4), (100, 4, 4), (13, 48, 1)])
def test_convolved_attention_at_the_window_edges(tier, window, probe, conv):
    """The inputs in front of the last query repeat those in front of position `probe`, so that the convolved query equals
    that position's convolved key up to the rotation of a few channels."""
    dev = _dev(tier)
    L = 61
    layer = O.parallel_layer(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.8, window=window, rot_dims=2, conv=conv)
    mod, cfg, W, mx = _layer(layer, dev, seed=9, edit=lambda W: _tie(W, "l0.mix.left.", conv=True))
    h = _rand(L, WIDTH, seed=10)
    for j in range(conv):
        if probe - j != L - 1 - j:
            h[L - 1 - j] = h[probe - j].clone()
    ref = lambda z: O.convolved_attention(z.to(F64), W, "l0.mix.left.", mx["left"], EPS, range(L))
    want = ref(h)
    att = mod.self_attn.parts[0]
    for cuts in CUTS(L):
        _close(_steps(att, cfg, h, cuts, dev), want, 3e-5)
    _close(_steps(att, cfg, h, _cuts(L, [5, 30]), dev, batch_with=_rand(19, WIDTH, seed=3)), want, 3e-5)
    if probe < L - 1 - conv:
        z = h.clone()
        z[probe - conv + 1] += 2.0                      # oldest input of the probe's key: matters only to a query that sees it
        moved = (ref(z)[-1] - want[-1]).abs().max()
        assert (moved > 1e-3) if L - 1 - probe < window else (moved == 0)


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("kw", [dict(heads=1, kv_heads=1, dim=8, vdim=40, rot_dims=8, conv=4), dict(heads=4, kv_heads=1, dim=10, vdim=6, rot_dims=6, conv=3),
                                dict(heads=3, kv_heads=3, dim=24, vdim=8, rot_dims=4, conv=6), dict(heads=2, kv_heads=1, dim=160, vdim=136, rot_dims=96, conv=2),
                                dict(heads=2, kv_heads=2, dim=130, vdim=5, rot_dims=130, conv=3), dict(heads=2, kv_heads=1, dim=64, vdim=64, rot_dims=20, conv=1)])
def test_convolved_attention_sizes_and_first_tokens(tier, kw):
    """Four and fewer taps on vector and scalar widths, more taps, wide heads, a convolution of one tap."""
    dev = _dev(tier)
    L = 43
    mod, cfg, W, mx = _layer(O.parallel_layer(window=17, **kw), dev, seed=11)
    h = _rand(L, WIDTH, seed=12)
    want = O.convolved_attention(h.to(F64), W, "l0.mix.left.", mx["left"], EPS, range(L))
    for cuts in CUTS(L):
        got = _steps(mod.self_attn.parts[0], cfg, h, cuts, dev)
        _close(got[:5], want[:5], 3e-5)
        _close(got, want, 3e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("pairs", [False, True])
@pytest.mark.parametrize("dim,vdim,rot,taps", [(64, 64, 32, 3), (128, 40, 64, 4), (192, 128, 20, 2), (20, 12, 6, 3), (18, 9, 10, 4)])
def test_convolved_rows_in_one_pass(pairs, dim, vdim, rot, taps):
    """The fused kernel against its unfused chain (convolution, rotation + unit norm, page write) in fp32: queries, pages and
    the carried window, on a batch of a long portion, a short one and a single token."""
    dev = _dev("gpu")
    H, G, bs = 3, 1, 8
    q_lens, ctx = [41, 2, 1], [0, 30, 7]
    meta = M.RaggedMeta.build(q_lens, ctx, [2, 0, 1], dev)
    T, C = sum(q_lens), (H + G) * dim + G * vdim
    tables = torch.randperm(24, generator=torch.Generator().manual_seed(1)).to(torch.int32).view(3, 8).to(dev)
    x, w, st = _rand(T, C + 4, seed=2).to(dev), _rand(C, taps, seed=3).to(dev), _rand(3, taps - 1, C, seed=4).to(dev)
    table = M.rotary_table(64, rot, 500.0, dev)
    kc, vc = torch.zeros(24, bs, G, dim, device=dev), torch.zeros(24, bs, G, vdim, device=dev)
    st1, kc1, vc1 = st.clone(), kc.clone(), vc.clone()
    q = M.conv_rotary_kv_write(x[:, :C], w, st1, H, G, dim, vdim, rot, pairs, table, EPS, kc1, vc1, tables, meta)
    y = M.short_conv_silu(x[:, :C], w, st, meta, activation=False)
    M.rotary_unit_norm(y, H + G, dim, rot, pairs, table, meta.token_pos, EPS)
    M.paged_kv_write_mix(y[:, H * dim:(H + G) * dim], y[:, (H + G) * dim:], kc, vc, tables, meta)
    _close(q, y[:, : H * dim].double().cpu(), 1e-6)
    _close(kc1, kc.double().cpu(), 1e-6)
    _close(vc1, vc.double().cpu(), 1e-6)
    assert torch.equal(st1, st)


# ------------------------------------------------------------------------------------------------ gated linear attention
@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("heads,dim,vdim,tau,rank", [(4, 16, 8, 16.0, 8), (1, 40, 24, 1.0, 1), (3, 8, 40, 4.0, 13), (2, 72, 5, 2.5, 16)])
def test_gated_linear_attention_with_slow_and_fast_channels(tier, heads, dim, vdim, tau, rank):
    """Decay pre-activations from -9 (a channel forgets at once for tau = 1) to +9 (it remembers the whole sequence)."""
    dev = _dev(tier)
    L = 80

    def edit(W):
        W["l0.mix.right.a2.b"] = torch.linspace(-9, 9, heads * dim)[torch.randperm(heads * dim, generator=torch.Generator().manual_seed(1))]
    layer = O.parallel_layer(g_heads=heads, g_dim=dim, g_vdim=vdim, tau=tau, rank=rank)
    mod, cfg, W, mx = _layer(layer, dev, seed=13, edit=edit)
    h = _rand(L, WIDTH, seed=14)
    want = O.gated_linear_attention(h.to(F64), W, "l0.mix.right.", mx["right"], EPS)
    for cuts in CUTS(L):
        _close(_steps(mod.self_attn.parts[1], cfg, h, cuts, dev), want, 5e-5)
    _close(_steps(mod.self_attn.parts[1], cfg, h, _cuts(L, [1, 1, 2, 30]), dev, batch_with=_rand(3, WIDTH, seed=3)), want, 5e-5)


@pytest.mark.parametrize("tier", TIERS)
def test_the_state_remembers_the_first_token(tier):
    """A first token far larger than the rest, decays of almost one: its share in the read-out 200 tokens later is what a
    lost or restarted state would miss."""
    dev = _dev(tier)
    L = 200
    q, k, v = _rand(L, 16, seed=1), _rand(L, 16, seed=2) * 0.01, _rand(L, 12, seed=3)
    k[0] *= 1e4
    z, bias = torch.zeros(L, 16), torch.full((16,), 6.0)
    meta = lambda n, c: M.RaggedMeta.build([n], [c], [1], dev)
    S = torch.full((2, 2, 8, 6), 7.0, device=dev)
    out, at = [], 0
    for n in (1, 2, 50, 1, 1, 145):
        s = slice(at, at + n)
        out.append(M.state_scan_gla(q[s].to(dev), k[s].to(dev), v[s].to(dev), z[s].to(dev), bias.to(dev), 4.0, S, meta(n, at), 2, 8, 6))
        at += n
    r = 1.0 / (1.0 + math.exp(-6.0))
    want = torch.zeros(L, 2, 6, dtype=F64)
    state = torch.zeros(2, 8, 6, dtype=F64)
    for t in range(L):
        state = r ** 0.25 * state + k[t].to(F64).view(2, 8, 1) * v[t].to(F64).view(2, 1, 6)
        want[t] = (state * q[t].to(F64).view(2, 8, 1)).sum(1) * 8 ** -0.5
    _close(torch.cat(out), want.reshape(L, 12), 1e-5)
    _close(S[1], state, 1e-5)
    assert (S[0] == 7.0).all()


# ------------------------------------------------------------------------------------------------ pairs
@pytest.mark.parametrize("tier", TIERS)
def test_pair_averages_its_normed_outputs(tier):
    dev = _dev(tier)
    L = 50
    mod, cfg, W, mx = _layer(O.parallel_layer(), dev, seed=15)
    h = _rand(L, WIDTH, seed=16)
    want = O.pair(h.to(F64), W, "l0.mix.", mx, EPS, range(L))
    for cuts in CUTS(L):
        got = _steps(mod.self_attn, cfg, h, cuts, dev)
        assert got.dtype == torch.float32
        _close(got, want, 5e-5)
    _close(_steps(mod.self_attn, cfg, h, _cuts(L, [4, 30]), dev, batch_with=_rand(21, WIDTH, seed=3)), want, 5e-5)


@pytest.mark.parametrize("tier", TIERS)
def test_pair_whose_parts_carry_states_of_the_same_name(tier):
    """Convolved attention beside a delta rule behind a convolution: both keep a convolution window in the layer's slot.  The
    pair equals its parts run alone."""
    dev = _dev(tier)
    L = 40
    left = MixerSpec(kind="attention", heads=2, dim=8, conv=3, conv_values=True, window=9, head_unit_norm=True, rot_dims=4)
    right = MixerSpec(kind="delta", heads=2, dim=8, vdim=12, conv=4)
    cfg_of = lambda spec: ModelConfig(model_type="sumolorn", vocab_size=8, hidden_size=WIDTH, layer_specs=[LayerSpec(mixer=spec)],
                                      norm_eps=EPS, norm_type="rms", pos_type="none", fp32_residual=True)
    torch.manual_seed(0)
    cfg = cfg_of(MixerSpec(kind="pair", parts=[left, right]))
    pair = build_mixer(cfg, 0)
    with torch.no_grad():
        for p in pair.parameters():
            p.copy_(torch.randn_like(p) * 0.3)
    pair = pair.to(dev)
    assert pair.parts[0].state_tag != pair.parts[1].state_tag
    h = _rand(L, WIDTH, seed=17)
    for cuts in ([L], [1] * L, _cuts(L, [2, 3, 20])):
        parts = []
        for m, spec in zip(pair.parts, (left, right)):
            tag, m.state_tag = m.state_tag, ""
            parts.append(_steps(m, cfg_of(spec), h, cuts, dev).double().cpu())
            m.state_tag = tag
        w = [p.detach().double().cpu() for p in pair.out_norm_weights]
        want = 0.5 * (O.rms(parts[0], EPS) * w[0] + O.rms(parts[1], EPS) * w[1])
        _close(_steps(pair, cfg, h, cuts, dev), want, 2e-5)


# ------------------------------------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("ff,limit", [(48, 1.0), (50, 0.25), (7, 4.0)])
def test_clamped_feed_forward(tier, ff, limit):
    """Pre-activations of both signs on both sides of the clamp."""
    dev = _dev(tier)
    mod, cfg, W, _ = _layer(O.attention_layer(mlp=O.dense(ff, limit)), dev, seed=18)
    h = _rand(21, WIDTH, seed=19, scale=2.0)
    g, u = h.to(F64) @ W["l0.mlp.gate"].T, h.to(F64) @ W["l0.mlp.up"].T
    assert (g > limit).any() and (g < -limit).any() and (u > limit).any() and (u < -limit).any() and (u.abs() < limit).any()
    with torch.inference_mode():
        got = mod.mlp(h.to(dev))
    _close(got, O.clamped_ff(h.to(F64), W, "l0.mlp.", limit), 2e-5)


# ------------------------------------------------------------------------------------------------ 16-bit attention kernels
@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 64, 64), (4, 1, 128, 40), (6, 6, 16, 32), (2, 1, 200, 200), (8, 1, 24, 24), (3, 1, 20, 12)])
@pytest.mark.parametrize("q_lens,ctx,window", [([1, 1], [700, 3], 0), ([1], [900], 130), ([5, 1, 2], [0, 64, 333], 40),
                                              ([210, 3], [50, 0], 0), ([150], [0], 64)])
def test_capped_gated_attention_in_16_bits(heads, kv, dim, vdim, q_lens, ctx, window):
    """All forms of the tensor-core kernel (decode rows shared by the warps, split keys, wide row tiles, 256-wide rows) and
    the exact kernel on 16-bit rows: soft cap, learned sinks and head gates against float64 on the same rounded inputs.
    Raw scores reach several times the cap."""
    dev = _dev("gpu")
    T, bs, n, cap, scale = sum(q_lens), 16, len(q_lens), 5.0, 1.2 / math.sqrt(dim)
    per = (max(a + b for a, b in zip(q_lens, ctx)) + bs - 1) // bs
    tables = torch.randperm(n * per, generator=torch.Generator().manual_seed(0)).to(torch.int32).view(n, per)
    bf = lambda *s, seed, f=1.0: _rand(*s, seed=seed, scale=f).to(torch.bfloat16)
    q, kc, vc = bf(T, heads * dim, seed=1, f=3.0), bf(n * per, bs, kv, dim, seed=2, f=3.0), bf(n * per, bs, kv, vdim, seed=3)
    gate, sink = bf(T, heads + 3, seed=4, f=2.0)[:, 1:1 + heads], torch.linspace(-3.0, 6.0, heads)
    meta = M.RaggedMeta.build(q_lens, ctx, list(range(n)), dev)
    got = M.paged_bias_attention(q.to(dev), kc.to(dev), vc.to(dev), tables.to(dev), meta, scale, sink=True,
                                 sink_values=sink.to(dev), window=window, softcap=cap, head_gate=gate.to(dev), wide_weights=True)
    want, t = torch.zeros(T, heads, vdim, dtype=F64), 0
    for i, (m, c) in enumerate(zip(q_lens, ctx)):
        rows = kc[tables[i].long()].reshape(-1, kv, dim)[: c + m].to(F64), vc[tables[i].long()].reshape(-1, kv, vdim)[: c + m].to(F64)
        for hd in range(heads):
            s = O.softcap(q[t:t + m].to(F64).view(m, heads, dim)[:, hd] @ rows[0][:, hd // (heads // kv)].T * scale, cap)
            full = torch.zeros(c + m, c + m, dtype=F64)
            full[c:] = s
            w = O.weigh(full, range(c + m), window, sink[hd].to(F64))[c:]
            want[t:t + m, hd] = w @ rows[1][:, hd // (heads // kv)] * O.sigmoid(gate[t:t + m, hd:hd + 1].to(F64))
        t += m
    _close(got.view(T, heads, vdim), want, 6e-3)
