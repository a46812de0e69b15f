"""Architecture description of the owned decoder family.

One config class covers Qwen3 dense, Qwen3-MoE and Llama/Qwen2-style decoders
(q/k-norm optional, attention bias optional).  ``from_hf`` reads a Hugging Face
``config.json`` dict; ``to_hf`` writes one back, so checkpoints stay loadable by
``transformers``.  Presets are the benchmark architectures with random init.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional, Sequence, Tuple, Union


# config.json ``model_type`` values whose layer maths is what ``models/decoder.py`` computes (each checked against transformers)
SUPPORTED_MODEL_TYPES = frozenset({'llama', 'mistral', 'mixtral', 'qwen2', 'qwen2_moe', 'qwen3', 'qwen3_moe', 'seed_oss', 'qwen2_vl', 'qwen2_vl_text',
                                   'qwen2_5_vl', 'qwen2_5_vl_text', 'qwen3_vl', 'qwen3_vl_text', 'qwen3_vl_moe', 'qwen3_vl_moe_text',
                                   'qwen3_5', 'qwen3_5_text', 'qwen3_5_moe', 'qwen3_5_moe_text', 'qwen3_next', 'glm', 'glm4',
                                   'phi3', 'internlm2', 'internlm3', 'gemma', 'deepseek_v2', 'deepseek_v3', 'kimi_k2', 'glm4_moe', 'gemma2', 'gemma3_text', 'gemma3', 'gpt_oss', 'granite', 'olmo2', 'olmo3', 'ernie4_5', 'smollm3'})


def _rope_scaling_of(cfg: Dict[str, Any]) -> Optional[Dict[str, Any]]:
    """``rope_scaling`` (or the newer ``rope_parameters``) of a HF config when it describes a long-context variant."""
    rs = cfg.get('rope_scaling') or cfg.get('rope_parameters')
    if not isinstance(rs, dict):
        return None
    kind = rs.get('rope_type', rs.get('type', 'default'))
    if kind in (None, 'default', 'mrope'):  # mrope is a position layout (see DecoderConfig.mrope_section), not a frequency change
        return None
    out = {k: v for k, v in rs.items() if k != 'rope_theta'}
    out.setdefault('rope_type', kind)
    if kind in ('llama3', 'yarn', 'longrope') and not out.get('original_max_position_embeddings'):
        out['original_max_position_embeddings'] = cfg.get('original_max_position_embeddings') or cfg.get('max_position_embeddings', 4096)
    if kind in ('dynamic', 'longrope'):      # these two compare the sequence length with the model's window
        out.setdefault('max_position_embeddings', cfg.get('max_position_embeddings', 4096))
    out.pop('partial_rotary_factor', None)
    return out


def _pomelix_fields(cfg: Dict[str, Any]) -> Dict[str, Any]:
    """``config.json`` of a Pomelix checkpoint → keyword arguments of :class:`DecoderConfig`."""
    specs = []
    for i, layer in enumerate(cfg['layers']):
        if layer['type'] != 'attention':
            raise NotImplementedError(f"layer {i}: mixer type {layer['type']!r} is not implemented (attention is)")
        m, mlp, qt = layer['mixer'], layer.get('mlp'), layer['mixer'].get('q_temp')
        if mlp is not None and mlp.get('kind', 'dense') != 'dense':
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented (dense is)")
        if qt is not None and (qt['every'] != int(qt['every']) or qt['every'] < 1):
            raise ValueError(f"layer {i}: q_temp.every must be a positive whole number of positions, not {qt['every']!r}")
        specs.append(LayerSpec(heads=int(m['heads']), kv_heads=int(m['kv_heads']), dim=int(m['dim']), vdim=int(m['vdim']), scale=float(m['scale']),
                               conv=int(m.get('conv') or 0), temp_coef=float(qt['coef']) if qt else 0.0, temp_every=int(qt['every']) if qt else 0,
                               v_mix=bool(m.get('v_mix')), ff=int(mlp['ff']) if mlp else 0))
    return dict(model_type='pomelix', vocab_size=int(cfg['vocab']), hidden_size=int(cfg['width']), rms_norm_eps=float(cfg['norm']['eps']),
                residual_multiplier=float(cfg.get('residual_mult', 1.0)), tie_word_embeddings=True, qk_norm=False, layer_specs=specs,
                eos_token_id=cfg.get('eos_token_id'), pad_token_id=cfg.get('pad_token_id'), torch_dtype=str(cfg.get('torch_dtype', 'bfloat16')))


def _pomelix_mapping(c: 'DecoderConfig') -> Dict[str, Any]:
    """The inverse of :func:`_pomelix_fields`."""
    layers = []
    for sp in c.layer_specs:
        m = {'heads': sp.heads, 'kv_heads': sp.kv_heads, 'dim': sp.dim, 'vdim': sp.vdim, 'scale': sp.scale, 'conv': sp.conv, 'v_mix': sp.v_mix}
        if sp.temp_every:
            m['q_temp'] = {'coef': sp.temp_coef, 'every': sp.temp_every}
        layers.append({'type': 'attention', 'mixer': m, 'mlp': {'kind': 'dense', 'ff': sp.ff} if sp.ff else None})
    d = {'architecture': 'Pomelix', 'vocab': c.vocab_size, 'width': c.hidden_size, 'norm': {'eps': c.rms_norm_eps},
         'residual_mult': c.residual_multiplier, 'layers': layers}
    d.update({k: v for k, v in (('eos_token_id', c.eos_token_id), ('pad_token_id', c.pad_token_id)) if v is not None})
    return d


def _moronex_fields(cfg: Dict[str, Any]) -> Dict[str, Any]:
    """``config.json`` of a Moronex checkpoint → keyword arguments of :class:`DecoderConfig`."""
    specs = []
    for i, layer in enumerate(cfg['layers']):
        m, mlp = layer['mixer'], layer.get('mlp')
        sizes = {k: int(m[k]) for k in ('heads', 'dim', 'vdim')}
        if layer['type'] == 'latent_attention':
            source = m.get('kv_from')
            mixer = LatentSpec(**sizes, q_rank=int(m['q_rank']), kv_rank=int(m['kv_rank']), scale=float(m['scale']), kv_from=None if source is None else int(source))
        elif layer['type'] == 'hgrn2':
            mixer = HGRN2Spec(**sizes)
        else:
            raise NotImplementedError(f"layer {i}: mixer type {layer['type']!r} is not implemented (latent_attention and hgrn2 are)")
        if mlp is None:
            ff = None
        elif mlp['kind'] == 'dense':
            ff = FeedForwardSpec(ff=int(mlp['ff']))
        elif mlp['kind'] == 'moe':
            ff = FeedForwardSpec(ff=int(mlp['expert']['ff']), experts=int(mlp['router']['experts']), top=int(mlp['router']['top']))
        else:
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented (dense and moe are)")
        specs.append(SandwichSpec(mixer, ff))
    return dict(model_type='moronex', vocab_size=int(cfg['vocab']), hidden_size=int(cfg['width']), rms_norm_eps=float(cfg['norm']['eps']), rms_norm_offset=1.0,
                tie_word_embeddings=False, qk_norm=False, layer_specs=specs, eos_token_id=cfg.get('eos_token_id'), pad_token_id=cfg.get('pad_token_id'),
                torch_dtype=str(cfg.get('torch_dtype', 'bfloat16')))


def _moronex_mapping(c: 'DecoderConfig') -> Dict[str, Any]:
    """The inverse of :func:`_moronex_fields`."""
    layers = []
    for sp in c.layer_specs:
        m = {k: getattr(sp.mixer, k) for k in ('heads', 'dim', 'vdim', 'q_rank', 'kv_rank', 'scale', 'kv_from') if getattr(sp.mixer, k, None) is not None}
        f = sp.mlp
        mlp = None if f is None else ({'kind': 'moe', 'expert': {'ff': f.ff}, 'router': {'experts': f.experts, 'top': f.top}} if f.experts
                                      else {'kind': 'dense', 'ff': f.ff})
        layers.append({'type': sp.mixer.kind, 'mixer': m, 'mlp': mlp})
    d = {'architecture': 'Moronex', 'vocab': c.vocab_size, 'width': c.hidden_size, 'norm': {'eps': c.rms_norm_eps}, 'layers': layers}
    d.update({k: v for k, v in (('eos_token_id', c.eos_token_id), ('pad_token_id', c.pad_token_id)) if v is not None})
    return d


def _nilepel_rotary(rot: Dict[str, Any], interleaved: bool) -> 'RotarySpec':
    return RotarySpec(dims=int(rot['dims']), base=float(rot['base']), interleaved=interleaved, scaling=dict(rot['scaling']) if rot.get('scaling') else None)


def _nilepel_fields(cfg: Dict[str, Any]) -> Dict[str, Any]:
    """``config.json`` of a Nilepel checkpoint → keyword arguments of :class:`DecoderConfig`."""
    specs = []
    for i, layer in enumerate(cfg['layers']):
        kind, m, mlp = layer['type'], layer['mixer'], layer.get('mlp')
        sizes = {k: int(m[k]) for k in ('heads', 'dim', 'vdim')}
        size, scale, source = int(m['mask']['size']), float(m['scale']), None if m.get('kv_from') is None else int(m['kv_from'])
        if kind == 'attention':
            mixer = AttentionSpec(**sizes, kv_heads=int(m['kv_heads']), scale=scale, rotary=_nilepel_rotary(m['rot'], True), chunk=size, sinks=True, kv_from=source)
        elif kind == 'attention_2':
            mixer = AttentionSpec(**sizes, kv_heads=int(m['kv_heads']), scale=scale, rotary=_nilepel_rotary(m['rot'], False), window=size, bias=True, qk_norm=True,
                                  sinks=True, head_gate=True, kv_from=source)
        elif kind == 'latent_attention':
            mixer = LatentSpec(**sizes, q_rank=0, kv_rank=int(m['kv_rank']), scale=scale, kv_from=source, rot_dim=int(m['rot_dim']),
                               rotary=_nilepel_rotary(m['rot'], True), window=size, sinks=False, head_gate=False)
        else:
            raise NotImplementedError(f"layer {i}: mixer type {kind!r} is not implemented (attention, attention_2 and latent_attention are)")
        if mlp is None:
            ff = None
        elif mlp['kind'] == 'dense':
            ff = FeedForwardSpec(ff=int(mlp['ff']), limit=float(mlp['limit']))
        elif mlp['kind'] == 'moe':
            r, groups = mlp['router'], mlp['router'].get('groups') or {}
            ff = FeedForwardSpec(ff=int(mlp['expert']['ff']), experts=int(r['experts']), top=int(r['top']), gated=True, scoring='softmax_grouped',
                                 groups=int(groups.get('count', 1)), keep=int(groups.get('keep', 1)), scale=float(r.get('scale', 1.0)),
                                 shared=int(mlp['shared']['ff']) if mlp.get('shared') else 0)
        else:
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented (dense and moe are)")
        specs.append(PreNormSpec(mixer, ff))
    return dict(model_type='nilepel', vocab_size=int(cfg['vocab']), hidden_size=int(cfg['width']), rms_norm_eps=float(cfg['norm']['eps']),
                embed_scale=float((cfg.get('embedding') or {}).get('scale', 1.0)), tie_word_embeddings=False, qk_norm=False, layer_specs=specs, eos_token_id=cfg.get('eos_token_id'),
                pad_token_id=cfg.get('pad_token_id'), torch_dtype=str(cfg.get('torch_dtype', 'bfloat16')))


def _nilepel_mapping(c: 'DecoderConfig') -> Dict[str, Any]:
    """The inverse of :func:`_nilepel_fields`."""
    layers = []
    for sp in c.layer_specs:
        m, f = sp.mixer, sp.mlp
        rot = {'base': m.rotary.base, 'dims': m.rotary.dims}
        if m.rotary.scaling:
            rot['scaling'] = dict(m.rotary.scaling)
        mixer = {'heads': m.heads, 'dim': m.dim, 'vdim': m.vdim, 'scale': m.scale, 'rot': rot, 'mask': {'size': m.window or m.chunk}}
        if m.kind == 'latent_attention':
            kind = m.kind
            mixer.update(kv_rank=m.kv_rank, rot_dim=m.rot_dim)
        else:
            kind = 'attention' if m.chunk else 'attention_2'
            mixer['kv_heads'] = m.kv_heads
        if m.kv_from is not None:
            mixer['kv_from'] = m.kv_from
        mlp = None
        if f is not None and f.experts:
            mlp = {'kind': 'moe', 'expert': {'ff': f.ff}, 'router': {'experts': f.experts, 'top': f.top, 'scale': f.scale, 'groups': {'count': f.groups, 'keep': f.keep}}}
            if f.shared:
                mlp['shared'] = {'ff': f.shared}
        elif f is not None:
            mlp = {'kind': 'dense', 'ff': f.ff, 'limit': f.limit}
        layers.append({'type': kind, 'mixer': mixer, 'mlp': mlp})
    d = {'architecture': 'Nilepel', 'vocab': c.vocab_size, 'width': c.hidden_size, 'norm': {'eps': c.rms_norm_eps}, 'embedding': {'scale': c.embed_scale}, 'layers': layers}
    d.update({k: v for k, v in (('eos_token_id', c.eos_token_id), ('pad_token_id', c.pad_token_id)) if v is not None})
    return d


def _puzonex_attention(m: Dict[str, Any], **kinds) -> 'AttentionSpec':
    return AttentionSpec(**{k: int(m[k]) for k in ('heads', 'kv_heads', 'dim', 'vdim')}, scale=float(m['scale']), window=int(m['mask']['size']), bias=True,
                         softcap=float(m['softcap']), **kinds)


def _puzonex_fields(cfg: Dict[str, Any]) -> Dict[str, Any]:
    """``config.json`` of a Puzonex checkpoint → keyword arguments of :class:`DecoderConfig`.  The number of rows of a distance table
    (``left.buckets``) is not in the original file: it is the shape of a tensor, and :func:`_puzonex_sizes` adds it."""
    specs = []
    for i, layer in enumerate(cfg['layers']):
        kind, m, mlp = layer['type'], layer['mixer'], layer.get('mlp')
        if kind == 'attention':
            mixer = _puzonex_attention(m, qk_norm=True, value_norm=True, log_bias=True, sinks=True)
        elif kind == 'mamba1':
            mixer = Mamba1Spec(**{k: int(m[k]) for k in ('inner', 'state', 'dt_rank', 'conv')})
        elif kind == 'parallel':
            left, right = m['left'], m['right']
            if 'buckets' not in left:
                raise ValueError(f"layer {i}: the size of its distance table is known from the checkpoint's tensors only; read the configuration with from_pretrained, "
                                 "or give left.buckets")
            mixer = SideBySideSpec(_puzonex_attention(left, qk_norm='whole', values_are_keys=True, temperature=True, buckets=int(left['buckets']), bias_max=float(left['bias_max']),
                                                      out_gate=True, out_bias=True),
                                   MatrixMemorySpec(**{k: int(right[k]) for k in ('heads', 'dim', 'vdim')}, gate_cap=float(right['gate_cap'])))
        else:
            raise NotImplementedError(f"layer {i}: mixer type {kind!r} is not implemented (attention, mamba1 and parallel are)")
        if mlp is not None and mlp['kind'] != 'dense':
            raise NotImplementedError(f"layer {i}: feed-forward kind {mlp['kind']!r} is not implemented (dense is)")
        specs.append(PostNormSpec(mixer, None if mlp is None else FeedForwardSpec(ff=int(mlp['ff']), act='gelu_tanh')))
    return dict(model_type='puzonex', vocab_size=int(cfg['vocab']), hidden_size=int(cfg['width']), rms_norm_eps=float(cfg['norm']['eps']), sinusoidal_base=10000.0,
                tie_word_embeddings=False, qk_norm=False, layer_specs=specs, eos_token_id=cfg.get('eos_token_id'), pad_token_id=cfg.get('pad_token_id'),
                torch_dtype=str(cfg.get('torch_dtype', 'bfloat16')))


def _puzonex_mapping(c: 'DecoderConfig') -> Dict[str, Any]:
    """The inverse of :func:`_puzonex_fields`."""
    def attention(a: 'AttentionSpec') -> Dict[str, Any]:
        return {**{k: getattr(a, k) for k in ('heads', 'kv_heads', 'dim', 'vdim', 'scale', 'softcap')}, 'mask': {'size': a.window}}

    layers = []
    for sp in c.layer_specs:
        m = sp.mixer
        if m.kind == 'attention':
            mixer = attention(m)
        elif m.kind == 'mamba1':
            mixer = {k: getattr(m, k) for k in ('inner', 'state', 'dt_rank', 'conv')}
        else:
            mixer = {'left': {**attention(m.left), 'bias_max': m.left.bias_max, 'buckets': m.left.buckets},
                     'right': {k: getattr(m.right, k) for k in ('heads', 'dim', 'vdim', 'gate_cap')}}
        layers.append({'type': m.kind, 'mixer': mixer, 'mlp': None if sp.mlp is None else {'kind': 'dense', 'ff': sp.mlp.ff}})
    d = {'architecture': 'Puzonex', 'vocab': c.vocab_size, 'width': c.hidden_size, 'norm': {'eps': c.rms_norm_eps}, 'layers': layers}
    d.update({k: v for k, v in (('eos_token_id', c.eos_token_id), ('pad_token_id', c.pad_token_id)) if v is not None})
    return d


def _puzonex_sizes(cfg: Dict[str, Any], shape: Callable[[str], Sequence[int]]) -> None:
    """What the file leaves to the checkpoint's tensors: ``shape`` gives a tensor's by its name."""
    for i, layer in enumerate(cfg['layers']):
        if layer['type'] == 'parallel':
            layer['mixer']['left']['buckets'] = int(shape(f'l{i}.mix.left.rel')[0])


# checkpoints whose config.json names its ``architecture`` and lists every layer: (reader → DecoderConfig fields, writer)
NATIVE_ARCHITECTURES = {'Pomelix': (_pomelix_fields, _pomelix_mapping), 'Moronex': (_moronex_fields, _moronex_mapping), 'Nilepel': (_nilepel_fields, _nilepel_mapping),
                        'Puzonex': (_puzonex_fields, _puzonex_mapping)}
# architectures whose files leave sizes to the tensors' shapes
_SIZES_FROM_TENSORS = {'Puzonex': _puzonex_sizes}


def _up8(n: int) -> int:
    return -(-n // 8) * 8


@dataclass
class LayerSpec:
    """Sizes and constants of one layer of a stack whose layers are listed one by one (``DecoderConfig.layer_specs``): an
    attention mixer with ``heads`` query and ``kv_heads`` key / value heads, query / key width ``dim`` and value width
    ``vdim``; ``conv`` taps of causal depth-wise convolution on q, k and v (1 = the newest row only, 0 = none);
    query temperature ``1 + temp_coef · ln(⌊(p + 1) / temp_every⌋ + 1)`` (``temp_every`` 0 = none); softmax ``scale``;
    ``v_mix``: values mixed with those of the first layer that has it; ``ff``: width of the gated feed-forward block
    (0 = the layer has none)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int = 0
    temp_coef: float = 0.0
    temp_every: int = 0
    v_mix: bool = False
    ff: int = 0

    is_moe = False

    @property
    def qkv_sizes(self) -> Tuple[int, int, int]:
        return self.heads * self.dim, self.kv_heads * self.dim, self.kv_heads * self.vdim

    # what a layer keeps per token, per sequence, and what it weighs (the same members exist on :class:`SandwichSpec`)
    def kv_rows(self) -> Tuple[int, int, int]:
        return self.kv_heads, _up8(self.dim), _up8(self.vdim)

    def conv_rows(self) -> Optional[Tuple[int, int]]:
        return (self.conv - 1, sum(self.qkv_sizes)) if self.conv > 1 else None

    def state_shape(self) -> Optional[Tuple[int, ...]]:
        return None

    def state_width(self) -> int:
        return 0

    def matmul_weights(self, width: int, active: bool = False) -> int:
        return width * sum(self.qkv_sizes) + width * self.heads * self.vdim + 3 * width * self.ff

    def small_weights(self, width: int) -> int:
        return self.conv * sum(self.qkv_sizes) + width * (3 if self.ff else 2) + int(self.v_mix)

    def attention_width(self) -> int:
        """Multiply-adds per key and query of the score and value products."""
        return (self.dim + self.vdim) * self.heads

    @property
    def ff_width(self) -> int:
        return self.ff


@dataclass
class RotarySpec:
    """Rotation of the leading ``dims`` dimensions of a head by position: pair ``i`` turns by ``base^(−2i/dims)`` per position.  A pair is
    ``(2i, 2i + 1)`` (``interleaved``) or ``(i, i + dims/2)``.  ``scaling`` (``factor``, ``low``, ``high``, ``original``): wavelengths above
    ``original / low`` are slowed down by ``factor``, those below ``original / high`` kept, the ones between blended."""
    dims: int
    base: float
    interleaved: bool = False
    scaling: Optional[Dict[str, float]] = None

    def __post_init__(self):
        if self.dims < 2 or self.dims % 2:
            raise ValueError(f'rotation over {self.dims} dimensions: a positive even number is needed')

    @property
    def pairs(self) -> int:
        return self.dims // 2

    def frequencies(self) -> List[float]:
        """Angle per position of every pair."""
        out = []
        for i in range(self.pairs):
            f = self.base**(-2.0 * i / self.dims)
            if self.scaling:
                factor, low, high, original = (float(self.scaling[k]) for k in ('factor', 'low', 'high', 'original'))
                turns = original * f / (2 * math.pi)               # over the original context
                if turns < low:
                    f = f / factor
                elif turns <= high:
                    s = (turns - low) / (high - low)
                    f = (1 - s) * f / factor + s * f
            out.append(f)
        return out


class MixerSpec:
    """What every kind of mixer answers for: what it keeps per token (``kv_rows``) and per sequence (``conv_rows``, ``state_shape``), what it
    borrows and how it rotates."""
    kv_from = rotary = None

    def kv_rows(self) -> Tuple[int, int, int]:
        return 0, 0, 0

    def conv_rows(self) -> Optional[Tuple[int, int]]:
        return None

    def state_shape(self) -> Optional[Tuple[int, ...]]:
        return None

    def state_width(self) -> int:
        """Elements of the state that a token writes and reads."""
        return math.prod(self.state_shape() or (0, ))

    def attention_width(self) -> int:
        """Multiply-adds per key and query of the score and value products."""
        return 0

    def kernel_parts(self) -> List[str]:
        """Kernels that not every stack needs (``ops/build.py``)."""
        return []


@dataclass
class AttentionSpec(MixerSpec):
    """Grouped-query attention.  Positions enter through a rotation of queries and keys (``rotary``) or through a number per head that is
    added to a score: ``log_bias`` (``−r1 ln(1 + r2 · distance)``) or a learned table of ``buckets`` rows over distances (exact up to half of them,
    then logarithmic up to ``bias_max``).  What a position sees: everything before it, its last ``window`` positions, or its own block
    of ``chunk`` positions counted from the first token.  Projections: ``bias`` on q, k and v; ``values_are_keys`` (the projected keys,
    before their norm); ``out_bias``.  Norms: ``qk_norm`` per head (True) or over all heads together (``'whole'``); ``value_norm`` (values
    over their root mean square).  Scores: times ``temperature`` (a number per head), through ``softcap · tanh(s / softcap)``, then the number for the
    distance; ``sinks`` (a logit per head in the denominator).  Output: ``head_gate`` (a sigmoid per head) or ``out_gate`` (one per element).
    ``kv_from``: index of the earlier layer whose keys and values this layer reads instead of its own."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[RotarySpec] = None
    window: int = 0
    chunk: int = 0
    bias: bool = False
    qk_norm: Union[bool, str] = False
    sinks: bool = False
    head_gate: bool = False
    kv_from: Optional[int] = None
    values_are_keys: bool = False
    value_norm: bool = False
    softcap: float = 0.0
    temperature: bool = False
    log_bias: bool = False
    buckets: int = 0
    bias_max: float = 0.0
    out_gate: bool = False
    out_bias: bool = False
    kind = 'attention'

    def __post_init__(self):
        if isinstance(self.rotary, dict):
            self.rotary = RotarySpec(**self.rotary)
        if self.heads % self.kv_heads:
            raise ValueError(f'{self.heads} query heads do not divide over {self.kv_heads} key / value heads')
        if self.rotary is not None and self.rotary.dims > self.dim:
            raise ValueError(f'rotation over {self.rotary.dims} of {self.dim} dimensions')
        if self.values_are_keys and self.vdim != self.dim:
            raise ValueError(f'values that are the keys: {self.vdim} wide, keys are {self.dim} wide')
        if self.rotary is not None and (self.values_are_keys or self.value_norm or self.qk_norm == 'whole'):
            raise ValueError('values_are_keys, value_norm and norms over all heads go with attention that does not rotate')
        if self.rotary is None and self.kv_from is not None:
            raise ValueError('attention that does not rotate has keys and values of its own')
        if self.buckets and (self.log_bias or self.buckets < 2 or not self.bias_max > self.buckets // 2):
            raise ValueError(f'a distance table of {self.buckets} rows up to {self.bias_max}: at least two rows, and a last distance beyond the exact half')

    @property
    def qkv_sizes(self) -> Tuple[int, int, int]:
        """Rows of the q, k and v projections (a layer that borrows keys and values has none of its own)."""
        own = 0 if self.kv_from is not None else self.kv_heads
        return self.heads * self.dim, own * self.dim, 0 if self.values_are_keys else own * self.vdim

    def in_parts(self) -> List[Tuple[str, int]]:
        """Projections of the layer input."""
        parts = [(n, w) for n, w in zip(('q_proj', 'k_proj', 'v_proj'), self.qkv_sizes) if w]
        return parts + ([('head_gate', self.heads)] if self.head_gate else []) + ([('out_gate', self.heads * self.vdim)] if self.out_gate else [])

    def distance_buckets(self) -> List[int]:
        """Row of the distance table for the distances 0 … ``bias_max``; all farther ones share the last."""
        half, far, out = self.buckets // 2, self.bias_max, []
        for n in range(int(math.ceil(far)) + 1):
            # the small term keeps a distance that lies on a boundary in the bucket that begins there
            out.append(n if n < half else min(self.buckets - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (self.buckets - half) + 1e-9)))
        return out

    def kernel_parts(self) -> List[str]:
        return ['rotary' if self.rotary is not None else 'heads']

    def kept(self) -> Tuple[Any, ...]:
        """What a borrowing layer must agree on with the layer it borrows from."""
        return self.kind, self.kv_heads, self.dim, self.vdim, self.rotary

    def lent_columns(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    def kv_rows(self) -> Tuple[int, int, int]:
        return (self.kv_heads, _up8(self.dim), _up8(self.vdim)) if self.kv_from is None else (0, 0, 0)

    def matmul_weights(self, width: int) -> int:
        return width * sum(n for _, n in self.in_parts()) + self.heads * self.vdim * width

    def small_weights(self) -> int:
        own = self.kv_from is None
        norms = self.dim * (self.heads + self.kv_heads) if self.qk_norm == 'whole' else self.dim * (2 if own else 1) if self.qk_norm else 0
        per_head = (1 if self.sinks else 0) + (1 if self.temperature else 0) + (2 if self.log_bias else 0) + self.buckets
        return (sum(self.qkv_sizes) if self.bias else 0) + norms + per_head * self.heads

    def attention_width(self) -> int:
        return (self.dim + self.vdim) * self.heads


@dataclass
class LatentSpec(MixerSpec):
    """Latent attention: keys (``dim`` per head) and values (``vdim``) expanded from one normed rank-``kv_rank`` latent per token, which
    is all the cache keeps, together with ``rot_dim`` rotated key dimensions that all heads share (0: no positions).  Queries through a
    normed rank-``q_rank`` bottleneck (0: a plain projection; a head's query is ``[dim | rot_dim]``).  ``window``: the last positions that a
    position sees (0: all).  ``sinks`` (a logit per head in the softmax), ``head_gate`` (a sigmoid per head on the output).  ``kv_from``:
    index of the earlier layer whose latents this layer reads instead of its own."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    kv_from: Optional[int] = None
    rot_dim: int = 0
    rotary: Optional[RotarySpec] = None
    window: int = 0
    sinks: bool = True
    head_gate: bool = True
    kind = 'latent_attention'
    chunk = 0

    def __post_init__(self):
        if isinstance(self.rotary, dict):
            self.rotary = RotarySpec(**self.rotary)
        if (self.rotary.dims if self.rotary else 0) != self.rot_dim:
            raise ValueError(f'the rotation covers {self.rotary.dims if self.rotary else 0} dimensions of a rotated part of {self.rot_dim}')
        if self.rot_dim and self.q_rank:
            raise ValueError('rotated queries come from a plain projection (q_rank 0)')

    @property
    def qk_width(self) -> int:
        return self.dim + self.rot_dim

    def in_parts(self) -> List[Tuple[str, int]]:
        """Projections of the layer input."""
        q = [('dq_proj', self.q_rank)] if self.q_rank else [('q_proj', self.heads * self.qk_width)]
        return q + ([('dkv_proj', self.kv_rank + self.rot_dim)] if self.kv_from is None else []) + ([('head_gate', self.heads)] if self.head_gate else [])

    def kept(self) -> Tuple[Any, ...]:
        """What a borrowing layer must agree on with the layer it borrows from."""
        return self.kind, self.kv_rank, self.rot_dim, self.rotary

    def lent_columns(self) -> int:
        return self.kv_rank + self.rot_dim

    def kv_rows(self) -> Tuple[int, int, int]:
        return (1, _up8(self.kv_rank + self.rot_dim), 0) if self.kv_from is None else (0, 0, 0)

    def matmul_weights(self, width: int) -> int:
        return width * sum(n for _, n in self.in_parts()) + self.heads * (self.dim * self.q_rank + (self.dim + self.vdim) * self.kv_rank + self.vdim * width)

    def small_weights(self) -> int:
        return self.q_rank + (self.kv_rank if self.kv_from is None else 0) + (self.heads if self.sinks else 0)

    def kernel_parts(self) -> List[str]:
        return ['latent'] + (['rotary'] if self.rotary is not None or not self.q_rank else [])

    def attention_width(self) -> int:
        return (self.qk_width + self.vdim) * self.heads


@dataclass
class HGRN2Spec(MixerSpec):
    """Linear attention whose forget gate (per head and channel, bounded from below) also decides what is written; ``heads``
    states of ``dim × vdim``."""
    heads: int
    dim: int
    vdim: int
    kind = 'hgrn2'

    def state_shape(self) -> Tuple[int, ...]:
        return self.heads, self.dim, self.vdim

    def kernel_parts(self) -> List[str]:
        return ['recurrent']

    def in_parts(self) -> List[Tuple[str, int]]:
        return [('q_proj', self.heads * self.dim), ('f_proj', self.heads * self.dim), ('v_proj', self.heads * self.vdim)]

    def matmul_weights(self, width: int) -> int:
        return width * self.heads * (2 * self.dim + 2 * self.vdim)

    def small_weights(self) -> int:
        return 2 * self.heads * self.dim + self.vdim


@dataclass
class Mamba1Spec(MixerSpec):
    """Selective scan: ``inner`` channels with ``state`` fp32 numbers each, whose decay and input depend on the token through a step size
    (of rank ``dt_rank``) behind a causal convolution of ``conv`` taps."""
    inner: int
    state: int
    dt_rank: int
    conv: int
    kind = 'mamba1'
    heads = 1

    def __post_init__(self):
        if self.conv < 1:
            raise ValueError(f'a convolution of {self.conv} taps')

    @property
    def dim(self) -> int:
        return self.inner

    def conv_rows(self) -> Optional[Tuple[int, int]]:
        return (self.conv - 1, self.inner) if self.conv > 1 else None

    def state_shape(self) -> Tuple[int, ...]:
        return self.inner, self.state

    def in_parts(self) -> List[Tuple[str, int]]:
        return [('in_proj', 2 * self.inner)]

    def matmul_weights(self, width: int) -> int:
        return 3 * width * self.inner + self.inner * (2 * self.dt_rank + 2 * self.state)

    def small_weights(self) -> int:
        return self.inner * (self.conv + 1 + 1 + self.state + 1)

    def kernel_parts(self) -> List[str]:
        return ['selective']


@dataclass
class MatrixMemorySpec(MixerSpec):
    """mLSTM: ``heads`` matrix memories of ``dim × vdim`` with a normaliser of ``dim`` and a running maximum, exponential input gates and
    sigmoid forget gates in the logarithm, both capped at ``gate_cap``."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float
    kind = 'mlstm'

    def state_shape(self) -> Tuple[int, ...]:
        """Per head the matrix by rows, the normaliser (filled up to whole vectors) and a vector that begins with the maximum."""
        return self.heads, -(-self.dim * self.vdim // 4) * 4 + -(-self.dim // 4) * 4 + 4

    def state_width(self) -> int:
        return self.heads * self.dim * (self.vdim + 1)

    def in_parts(self) -> List[Tuple[str, int]]:
        d, e = self.heads * self.dim, self.heads * self.vdim
        return [('q_proj', d), ('k_proj', d), ('v_proj', e), ('out_gate', e), ('i_gate', self.heads), ('f_gate', self.heads)]

    def matmul_weights(self, width: int) -> int:
        return width * (sum(n for _, n in self.in_parts()) + self.heads * self.vdim)

    def small_weights(self) -> int:
        return self.heads * (self.vdim + 2)

    def kernel_parts(self) -> List[str]:
        return ['memory']


@dataclass
class SideBySideSpec(MixerSpec):
    """Attention and a matrix memory on the same input; the result is half the sum of both, each RMS-normed over the model's width."""
    left: AttentionSpec
    right: MatrixMemorySpec
    kind = 'parallel'

    def __post_init__(self):
        if isinstance(self.left, dict):
            self.left = AttentionSpec(**self.left)
        if isinstance(self.right, dict):
            self.right = MatrixMemorySpec(**self.right)
        if self.left.kv_from is not None:
            raise ValueError('attention beside another mixer has keys and values of its own')

    heads = property(lambda self: self.left.heads)
    kv_heads = property(lambda self: self.left.kv_heads)
    dim = property(lambda self: self.left.dim)
    rotary = property(lambda self: self.left.rotary)

    def kv_rows(self) -> Tuple[int, int, int]:
        return self.left.kv_rows()

    def state_shape(self) -> Tuple[int, ...]:
        return self.right.state_shape()

    def state_width(self) -> int:
        return self.right.state_width()

    def in_parts(self) -> List[Tuple[str, int]]:
        return [(f'{side}_{n}', w) for side in ('left', 'right') for n, w in getattr(self, side).in_parts()]

    def matmul_weights(self, width: int) -> int:
        return self.left.matmul_weights(width) + self.right.matmul_weights(width)

    def small_weights(self) -> int:
        return self.left.small_weights() + self.right.small_weights()

    def attention_width(self) -> int:
        return self.left.attention_width()

    def kernel_parts(self) -> List[str]:
        return self.left.kernel_parts() + self.right.kernel_parts()


@dataclass
class FeedForwardSpec:
    """Gated feed-forward block of width ``ff``, or, with ``experts``, that many experts of which a token uses ``top``.

    Dense: ``act(gate) · up`` with ``act`` ``'silu'`` or ``'gelu_tanh'``, or with a ``limit`` ``g σ(1.702 g) (u + 1)`` on ``g ≤ limit``, ``|u| ≤ limit``.
    Experts: two matrices around the square of relu, or ``gated`` ones (three matrices, ``silu(gate) · up``).  ``scoring`` as in
    ``DecoderConfig.router_scoring``: ``'topk_softmax'`` (biased logits, a softmax over the chosen) or ``'softmax_grouped'`` (softmax over all;
    only experts of the ``keep`` best of ``groups`` groups of neighbours, each as good as its best expert; weights times ``scale``).
    ``shared``: width of an expert beside them that runs for every token, scaled by a sigmoid per token (0: none)."""
    ff: int
    experts: int = 0
    top: int = 0
    limit: float = 0.0
    gated: bool = False
    scoring: str = 'topk_softmax'
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared: int = 0
    act: str = 'silu'

    def __post_init__(self):
        if self.act not in ('silu', 'gelu_tanh') or (self.act != 'silu' and (self.limit or self.experts)):
            raise ValueError(f'activation {self.act!r}: silu, or gelu_tanh in a dense block without a limit')
        if not self.experts:
            return
        if self.experts % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError(f'{self.experts} experts in {self.groups} groups of which {self.keep} are kept')
        if not 1 <= self.top <= self.experts // self.groups * self.keep:
            raise ValueError(f'top {self.top} of {self.experts // self.groups * self.keep} experts that can be chosen')

    def matmul_weights(self, width: int, active: bool = False) -> int:
        if not self.experts:
            return 3 * width * self.ff
        per = (3 if self.gated else 2) * width * self.ff
        return width * self.experts + (self.top if active else self.experts) * per + (3 * width * self.shared + width if self.shared else 0)

    def small_weights(self) -> int:
        return self.experts if self.scoring == 'topk_softmax' else 0


_MIXER_SPECS = ((SideBySideSpec, 'left'), (LatentSpec, 'kv_rank'), (AttentionSpec, 'kv_heads'), (Mamba1Spec, 'inner'), (MatrixMemorySpec, 'gate_cap'), (HGRN2Spec, 'heads'))


@dataclass
class SandwichSpec:
    """One layer with a norm in front of and behind each sub-layer and a sigmoid gate (read from the sub-layer's input) on its
    result: a mixer and a feed-forward block (None: the layer has none)."""
    mixer: MixerSpec
    mlp: Optional[FeedForwardSpec] = None

    def __post_init__(self):
        if isinstance(self.mixer, dict):
            self.mixer = next(c for c, key in _MIXER_SPECS if key in self.mixer)(**self.mixer)
        if isinstance(self.mlp, dict):
            self.mlp = FeedForwardSpec(**self.mlp)

    heads = property(lambda self: self.mixer.heads)
    kv_heads = property(lambda self: getattr(self.mixer, 'kv_heads', self.mixer.heads))
    dim = property(lambda self: self.mixer.dim)
    v_mix = False

    @property
    def is_moe(self) -> bool:
        return self.mlp is not None and self.mlp.experts > 0

    @property
    def ff_width(self) -> int:
        return self.mlp.ff if self.mlp is not None else 0

    def kv_rows(self) -> Tuple[int, int, int]:
        return self.mixer.kv_rows()

    def conv_rows(self) -> Optional[Tuple[int, int]]:
        return self.mixer.conv_rows()

    def state_shape(self) -> Optional[Tuple[int, ...]]:
        return self.mixer.state_shape()

    def state_width(self) -> int:
        return self.mixer.state_width()

    def around(self, width: int) -> Tuple[int, int]:
        """Weights of what stands around one sub-layer: in products, and others."""
        return width * width, 3 * width

    def matmul_weights(self, width: int, active: bool = False) -> int:
        n = self.around(width)[0] + self.mixer.matmul_weights(width)
        return n + (self.around(width)[0] + self.mlp.matmul_weights(width, active) if self.mlp is not None else 0)

    def small_weights(self, width: int) -> int:
        n = self.around(width)[1] + self.inside(width) + self.mixer.small_weights()
        return n + (self.around(width)[1] + self.mlp.small_weights() if self.mlp is not None else 0)

    def attention_width(self) -> int:
        return self.mixer.attention_width()

    def inside(self, width: int) -> int:
        """Weights inside the mixer that are as wide as the model: norms of two results, the bias of an output projection."""
        m = self.mixer
        return (2 * width if m.kind == 'parallel' else 0) + (width if getattr(getattr(m, 'left', m), 'out_bias', False) else 0)


@dataclass
class PreNormSpec(SandwichSpec):
    """One layer with a norm in front of each sub-layer, whose result joins the stream as it is."""
    post: bool = False           # no norm behind the sub-layers (tells the kinds apart when read from a mapping)

    def around(self, width: int) -> Tuple[int, int]:
        return 0, width


@dataclass
class PostNormSpec(SandwichSpec):
    """One layer whose sub-layers read the stream as it is; a norm on each sub-layer's result before it joins."""
    pre: bool = False            # no norm in front of the sub-layers (tells the kinds apart when read from a mapping)

    def around(self, width: int) -> Tuple[int, int]:
        return 0, width


def _layer_spec(sp: Any) -> Any:
    if not isinstance(sp, dict):
        return sp
    if 'mixer' not in sp:
        return LayerSpec(**sp)
    return (PreNormSpec if 'post' in sp else PostNormSpec if 'pre' in sp else SandwichSpec)(**sp)


@dataclass
class DecoderConfig:
    vocab_size: int = 151936
    hidden_size: int = 4096
    intermediate_size: int = 12288
    num_hidden_layers: int = 36
    num_attention_heads: int = 32
    num_key_value_heads: int = 8
    head_dim: int = 128
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    rope_scaling: Optional[Dict[str, Any]] = None  # HF mapping: {'rope_type': 'llama3' | 'yarn' | 'linear', 'factor': …}
    tie_word_embeddings: bool = False
    qk_norm: bool = True
    attention_bias: bool = False
    rms_norm_offset: float = 0.0  # 1.0 for gemma-style "1 + w"
    # Qwen3.5 full-attention layers: rotary embedding on the leading ``head_dim * partial_rotary_factor`` dims only, and a
    # per-head sigmoid gate (a second half of the q projection) on the attention output; their q/k norms are "1 + w" too
    partial_rotary_factor: float = 1.0
    attn_output_gate: bool = False
    # GLM-4 family: the checkpoint's rotary pairs are (2i, 2i+1); the bridge permutes the q / k projection rows into the
    # (i, i + R/2) convention computed here (scores are unchanged by a common permutation of q and k dims), gate and up are
    # one fused tensor in the checkpoint, and ``glm4`` norms each sub-layer's output before the residual add
    rope_interleaved: bool = False
    sandwich_norm: bool = False
    # Gemma: gate activation of the feed-forward block ('silu' | 'gelu_pytorch_tanh') and the factor √hidden on the
    # token embeddings (rounded to the compute dtype, as the Hugging Face model forms it)
    hidden_act: str = 'silu'
    embed_scale: float = 1.0
    # attention window of checkpoints trained with one (Mistral-7B-v0.1, Phi-3-mini): rows longer than the window are
    # refused — every key inside the window is what the kernels here compute
    sliding_window: Optional[int] = None
    # Gemma-2 / Gemma-3: scores through ``cap · tanh(s / cap)``, output logits likewise; softmax scale ``query_pre_attn_scalar^-½``
    # instead of ``head_dim^-½``; sliding-window layers (``layer_types`` entries ``'sliding_attention'``) of Gemma-3 use a rotary
    # base of their own, without the long-context scaling of the global layers
    # GPT-OSS: a learned per-head sink logit in the attention softmax, biases on the output projection, the router and the expert
    # tensors, routing = softmax over the top-k router logits, experts with the clamped ``(up + 1) · gate · σ(1.702 · gate)`` unit
    # Granite: what each sub-layer adds to the residual stream is multiplied by ``residual_multiplier``, output logits are divided by
    # ``logits_scaling``, the softmax scale is ``attention_multiplier`` (kept in ``query_pre_attn_scalar`` as its inverse square)
    residual_multiplier: float = 1.0
    logits_scaling: float = 1.0
    # OLMo-2 / OLMo-3: no norm in front of a sub-layer, only the one on its output (``sandwich_norm`` without ``pre_norm``), and
    # q / k norms over the whole projection instead of per head
    pre_norm: bool = True
    qk_norm_full: bool = False
    # SmolLM3: per layer, 1 = rotary embedding as usual, 0 = no position information in that layer's attention
    no_rope_layers: Optional[List[int]] = None
    attn_sinks: bool = False
    o_proj_bias: bool = False
    router_linear_bias: bool = False
    expert_bias: bool = False
    expert_act: str = 'swiglu'
    attn_logit_softcapping: Optional[float] = None
    final_logit_softcapping: Optional[float] = None
    query_pre_attn_scalar: Optional[float] = None
    rope_local_theta: Optional[float] = None
    # MoE (num_experts == 0 → dense)
    num_experts: int = 0
    num_experts_per_tok: int = 8
    moe_intermediate_size: int = 768
    norm_topk_prob: bool = True
    router_aux_loss_coef: float = 0.0
    shared_expert_intermediate_size: int = 0
    # DeepSeek-V3 style routing: sigmoid scores, a per-expert selection bias that is not trained by the loss, experts in
    # ``n_group`` groups of which the ``topk_group`` best (by their two best biased scores) stay eligible, weights scaled by
    # ``routed_scaling_factor``; the first ``first_k_dense_replace`` layers keep a dense feed-forward block; the shared
    # expert has no gate of its own
    router_scoring: str = 'softmax'
    router_bias: bool = False
    n_group: int = 1
    topk_group: int = 1
    routed_scaling_factor: float = 1.0
    first_k_dense_replace: int = 0
    shared_expert_gate: bool = True
    # multi-head latent attention (DeepSeek-V2/V3): queries through a rank-``q_lora_rank`` bottleneck (None = a plain
    # projection), keys / values expanded from one rank-``kv_lora_rank`` latent per token (0 = ordinary attention); a head's
    # query / key is ``qk_nope_head_dim`` position-free dims plus ``qk_rope_head_dim`` rotary dims whose key part is shared
    # by all heads; values are ``v_head_dim`` wide
    q_lora_rank: Optional[int] = None
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 128
    qk_rope_head_dim: int = 64
    v_head_dim: int = 128
    mla_rope_interleave: bool = True
    initializer_range: float = 0.02
    model_type: str = 'qwen3'
    torch_dtype: str = 'bfloat16'
    max_position_embeddings: int = 40960
    pad_token_id: Optional[int] = None
    eos_token_id: Optional[int] = None
    # hybrid stacks: per-layer 'full_attention' | 'linear_attention' (Gated DeltaNet); None = all full attention
    layer_types: Optional[List[str]] = None
    linear_num_key_heads: int = 16
    linear_num_value_heads: int = 32
    linear_key_head_dim: int = 128
    linear_value_head_dim: int = 128
    linear_conv_kernel_dim: int = 4
    # vision-language (Qwen2-VL family): the vision tower's config.json section, placeholder token ids, and the split of
    # the rotary half-dimension over (time, height, width) positions
    vision: Optional[Dict[str, Any]] = None
    image_token_id: Optional[int] = None
    video_token_id: Optional[int] = None
    vision_start_token_id: Optional[int] = None
    vision_end_token_id: Optional[int] = None
    mrope_section: Optional[List[int]] = None
    mrope_interleaved: bool = False  # Qwen3-VL lays the three position components out t h w t h w … instead of in blocks
    # stacks whose layers are listed one by one, with a 32-bit residual stream: layers that run mixer and feed-forward side by side
    # on one norm, each result with a learned per-channel scale (``LayerSpec``; Pomelix), layers with norms around each sub-layer and a
    # gate on its result (``SandwichSpec``; Moronex), layers with a norm in front of each sub-layer (``PreNormSpec``; Nilepel), or layers with a
    # norm on each sub-layer's result only (``PostNormSpec``; Puzonex)
    layer_specs: Optional[List[Union[LayerSpec, SandwichSpec, PreNormSpec, PostNormSpec, Dict[str, Any]]]] = None
    # such stacks: sines and cosines of the position on top of the token embeddings, pair ``i`` at ``base^(−2i/hidden)`` per position (0: none)
    sinusoidal_base: float = 0.0

    def __post_init__(self):
        if self.layer_specs is not None:
            self.layer_specs = [_layer_spec(sp) for sp in self.layer_specs]
            first = self.layer_specs[0]
            self.num_hidden_layers = len(self.layer_specs)
            self.num_attention_heads, self.num_key_value_heads, self.head_dim = first.heads, first.kv_heads, first.dim
            self.intermediate_size = max(sp.ff_width for sp in self.layer_specs)
            for i, sp in enumerate(self.layer_specs):
                if sp.heads % sp.kv_heads:
                    raise ValueError(f'layer {i}: {sp.heads} query heads do not divide over {sp.kv_heads} key / value heads')
            mixed = [sp for sp in self.layer_specs if sp.v_mix]
            if any((sp.kv_heads, sp.vdim) != (mixed[0].kv_heads, mixed[0].vdim) for sp in mixed):
                raise ValueError('layers that mix values must agree on the number and width of the value heads')
            for i, sp in enumerate(self.layer_specs):
                j = getattr(getattr(sp, 'mixer', None), 'kv_from', None)
                if j is None:
                    continue
                src = self.layer_specs[j].mixer if 0 <= j < i else None
                if src is None or src.kind not in ('attention', 'latent_attention') or src.kv_from is not None or src.kept() != sp.mixer.kept():
                    raise ValueError(f'layer {i}: kv_from {j} is not an earlier layer with keys and values of its own and the same sizes and rotation {sp.mixer.kept()}')
        if self.vision is not None:
            from .vision import VisionConfig
            self.vision = VisionConfig.from_hf(self.vision).to_hf()  # only the fields the tower uses, in the family's spelling

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    @property
    def is_mla(self) -> bool:
        return self.kv_lora_rank > 0

    @property
    def first_mixing_layer(self) -> Optional[int]:
        """Index of the layer whose values the later value-mixing layers take in (None: no layer mixes)."""
        return next((i for i, sp in enumerate(self.layer_specs or []) if sp.v_mix), None)

    def kv_layout(self) -> List[Tuple[int, int, int]]:
        """Per layer ``(key / value heads, key row width, value row width)`` of the paged cache.  Layers with widths of their
        own keep rows of whole 16-byte vectors (widths rounded up to a multiple of 8, the rest zero); a latent is one key row
        that also serves as the value; layers that keep nothing per token have 0 heads."""
        if self.layer_specs is None:
            return [(self.num_key_value_heads, self.head_dim, self.head_dim)] * self.num_hidden_layers
        return [sp.kv_rows() for sp in self.layer_specs]

    def conv_layout(self) -> List[Optional[Tuple[int, int]]]:
        """Per layer ``(rows, channels)`` of the convolution history a sequence keeps between steps (None: no history)."""
        return [sp.conv_rows() for sp in self.layer_specs or []]

    def state_layout(self) -> List[Optional[Tuple[int, ...]]]:
        """Per layer shape of the (fp32) recurrent state a sequence carries from token to token (None: no state)."""
        return [sp.state_shape() for sp in self.layer_specs or []]

    def held_columns(self) -> List[Tuple[int, int]]:
        """``(layer, columns)`` of what later layers take from earlier ones besides the stream: the values of the first mixing
        layer, the latents of layers that others borrow."""
        if self.first_mixing_layer is not None:
            first = self.layer_specs[self.first_mixing_layer]
            return [(self.first_mixing_layer, first.kv_heads * first.vdim)]
        lent = sorted({sp.mixer.kv_from for sp in self.layer_specs or [] if getattr(getattr(sp, 'mixer', None), 'kv_from', None) is not None})
        return [(j, self.layer_specs[j].mixer.lent_columns()) for j in lent]

    def kernel_parts(self) -> List[str]:
        """Mechanisms of a stack with listed layers whose kernels not every such stack needs (``ops/build.py``)."""
        parts = set()
        for sp in self.layer_specs or []:
            m = getattr(sp, 'mixer', None)
            if m is None:
                parts.add('convolution')
            else:
                parts.update(m.kernel_parts())
                parts.update(['experts'] if sp.is_moe else [])
        return sorted(parts)

    def rotations(self) -> List[RotarySpec]:
        """The distinct rotations of a stack with listed layers, in the order in which layers first use them."""
        out: List[RotarySpec] = []
        for sp in self.layer_specs or []:
            rot = getattr(getattr(sp, 'mixer', None), 'rotary', None)
            if rot is not None and rot not in out:
                out.append(rot)
        return out

    def rotary_columns(self, layer_idx: int) -> Optional[Tuple[int, int]]:
        """``(first, number)`` of a layer's pairs in the table of all :meth:`rotations` (None: the layer does not rotate)."""
        at, mine = 0, getattr(self.layer_specs[layer_idx].mixer, 'rotary', None)
        for rot in self.rotations():
            if rot == mine:
                return at, rot.pairs
            at += rot.pairs
        return None

    def layer_is_moe(self, layer_idx: int) -> bool:
        return self.num_experts > 0 and layer_idx >= self.first_k_dense_replace

    def layer_window(self, layer_idx: int) -> Optional[int]:
        """Attention window of a layer: the model's ``sliding_window`` on every layer, or only on those that ``layer_types``
        marks ``'sliding_attention'``."""
        if not self.sliding_window:
            return None
        if self.layer_types and 'sliding_attention' in self.layer_types:
            return self.sliding_window if self.layer_types[layer_idx] == 'sliding_attention' else None
        return self.sliding_window

    @property
    def attn_scale(self) -> float:
        """Softmax scale of the attention scores: ``1/√d`` of the query / key width; DeepSeek's YaRN variant multiplies
        it by the square of ``0.1·mscale_all_dim·ln(factor) + 1``."""
        if not self.is_mla:
            return float(self.query_pre_attn_scalar or self.head_dim)**-0.5
        sc = (self.qk_nope_head_dim + self.qk_rope_head_dim)**-0.5
        rs = self.rope_scaling or {}
        if rs.get('mscale_all_dim') and float(rs.get('factor', 1.0)) > 1.0 and self.model_type != 'deepseek_v2':
            m = 0.1 * float(rs['mscale_all_dim']) * math.log(float(rs['factor'])) + 1.0
            sc = sc * m * m
        return sc

    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    def _attn_weights(self) -> int:
        h, nh = self.hidden_size, self.num_attention_heads
        if self.is_mla:
            qk = self.qk_nope_head_dim + self.qk_rope_head_dim
            q = h * self.q_lora_rank + self.q_lora_rank * nh * qk if self.q_lora_rank else h * nh * qk
            return q + h * (self.kv_lora_rank + self.qk_rope_head_dim) + self.kv_lora_rank * nh * (self.qk_nope_head_dim + self.v_head_dim) + nh * self.v_head_dim * h
        return h * (self.q_size + 2 * self.kv_size) + self.q_size * h + (self.q_size * h if self.attn_output_gate else 0)

    def _listed_matmul_weights(self, active: bool = False) -> int:
        return sum(sp.matmul_weights(self.hidden_size, active) for sp in self.layer_specs)

    def num_params(self) -> int:
        h, L = self.hidden_size, self.num_hidden_layers
        if self.layer_specs is not None:
            small = sum(sp.small_weights(h) for sp in self.layer_specs)
            return self._listed_matmul_weights() + small + self.vocab_size * h * (1 if self.tie_word_embeddings else 2) + h
        attn = self._attn_weights() + (2 * self.head_dim if self.qk_norm else 0)
        moe = self.num_experts * 3 * h * self.moe_intermediate_size + h * self.num_experts + 3 * h * self.shared_expert_intermediate_size
        dense = 3 * h * self.intermediate_size
        n_moe = sum(self.layer_is_moe(i) for i in range(L))
        emb = self.vocab_size * h * (1 if self.tie_word_embeddings else 2)
        return L * (attn + 2 * h) + n_moe * moe + (L - n_moe) * dense + emb + h

    @property
    def rotary_dim(self) -> int:
        """Leading dims of a head that carry the rotary embedding (even; the whole head unless ``partial_rotary_factor`` < 1)."""
        if self.is_mla:
            return self.qk_rope_head_dim
        return self.head_dim if self.partial_rotary_factor >= 1.0 else int(self.head_dim * self.partial_rotary_factor) // 2 * 2

    def flops_per_token(self, avg_context: float = 0.0) -> float:
        """Forward+backward matmul FLOPs per token (6·N_active + attention)."""
        h, L = self.hidden_size, self.num_hidden_layers
        if self.layer_specs is not None:
            attn = sum(sp.attention_width() for sp in self.layer_specs) * avg_context
            state = 2 * sum(sp.state_width() for sp in self.layer_specs)       # a write and a read of every state element
            return 6.0 * (self._listed_matmul_weights(active=True) + self.vocab_size * h + state) + 6.0 * attn
        attn_w = self._attn_weights()
        moe_w = self.num_experts_per_tok * 3 * h * self.moe_intermediate_size + h * self.num_experts + 3 * h * self.shared_expert_intermediate_size
        n_moe = sum(self.layer_is_moe(i) for i in range(L))
        dense = L * attn_w + n_moe * moe_w + (L - n_moe) * 3 * h * self.intermediate_size + self.vocab_size * h
        qk_v = (self.qk_nope_head_dim + self.qk_rope_head_dim + self.v_head_dim) * self.num_attention_heads if self.is_mla else 2 * self.q_size
        attn = L * qk_v * avg_context  # QKᵀ and PV, causal average context
        return 6.0 * dense + 6.0 * attn

    # ---------------------------------------------------------------- HF I/O
    @classmethod
    def from_hf(cls, cfg: Dict[str, Any]) -> 'DecoderConfig':
        cfg = dict(cfg)
        if cfg.get('architecture') in NATIVE_ARCHITECTURES:
            return cls(**NATIVE_ARCHITECTURES[cfg['architecture']][0](cfg))
        top = cfg
        if 'text_config' in cfg:
            cfg = dict(cfg['text_config'])
        mt = cfg.get('model_type', 'qwen3')
        if mt not in SUPPORTED_MODEL_TYPES and not os.environ.get('TWINKLE_ALLOW_UNKNOWN_ARCH'):
            # an unknown type may differ in ways a shared field list does not show (scaled embeddings or residuals, other
            # norms, partial rotary …): better refused than silently computed wrongly
            raise NotImplementedError(f'model_type {mt!r} is not among the decoder families implemented here {sorted(SUPPORTED_MODEL_TYPES)}; '
                                      'set TWINKLE_ALLOW_UNKNOWN_ARCH=1 to load it as a Llama-style decoder anyway')
        vision = top.get('vision_config')
        if vision is not None:
            vision = dict(vision)
            if vision.get('model_type', top.get('model_type', 'qwen2_vl')) not in ('qwen2_vl', 'qwen2_5_vl', 'qwen3_vl', 'qwen3_vl_moe', 'qwen3_5', 'qwen3_5_moe'):
                raise NotImplementedError(f"vision tower of type {vision.get('model_type')!r} is not supported (qwen2_vl, qwen2_5_vl, qwen3_vl and qwen3_5 are)")
        rs_any = cfg.get('rope_scaling') or cfg.get('rope_parameters') or top.get('rope_scaling') or {}
        q35 = mt.startswith('qwen3_5') or mt == 'qwen3_next'      # the hybrid family: gated attention, partial rotary, "1 + w" norms
        heads = cfg.get('num_attention_heads', 32)
        mla = mt in ('deepseek_v2', 'deepseek_v3', 'kimi_k2')
        v2 = mt == 'deepseek_v2'      # softmax scores, groups ranked by their best expert, no selection bias, weights not renormalised
        dsv3 = mla or mt == 'glm4_moe'        # GLM-4.5 routes like DeepSeek-V3 over ordinary grouped-query attention
        window = cfg.get('sliding_window')
        if mt.startswith('qwen') and not cfg.get('use_sliding_window'):
            window = None                    # the Qwen configs carry a window size that is switched off by default
        gemma23 = mt in ('gemma2', 'gemma3_text', 'gemma3')
        oss = mt == 'gpt_oss'
        granite = mt == 'granite'
        olmo = mt in ('olmo2', 'olmo3')
        rope_local = cfg.get('rope_local_base_freq')
        rp = cfg.get('rope_parameters')
        if isinstance(rp, dict) and isinstance(rp.get('full_attention'), dict):      # per-layer-type rotary settings (Gemma-3)
            rope_local = (rp.get('sliding_attention') or {}).get('rope_theta', rope_local)
            cfg['rope_parameters'] = dict(rp['full_attention'])
        act = cfg.get('hidden_activation') or cfg.get('hidden_act') or 'silu'
        if mt == 'gemma':
            act = 'gelu_pytorch_tanh'        # what the Hugging Face model runs whatever the (legacy) field says
        if act not in ('silu', 'gelu_pytorch_tanh'):
            raise NotImplementedError(f'feed-forward activation {act!r} is not supported (silu and gelu_pytorch_tanh are)')
        out = cls(
            vocab_size=cfg.get('vocab_size', 151936), hidden_size=cfg.get('hidden_size', 4096),
            intermediate_size=cfg.get('intermediate_size', 12288), num_hidden_layers=cfg.get('num_hidden_layers', 36),
            num_attention_heads=heads, num_key_value_heads=cfg.get('num_key_value_heads', heads),
            head_dim=(cfg.get('head_dim') or cfg.get('hidden_size', 4096) // heads) if not mla
            else int(cfg.get('qk_nope_head_dim', 128)) + int(cfg.get('qk_rope_head_dim', 64)), rms_norm_eps=cfg.get('rms_norm_eps', 1e-6),
            rope_theta=float(cfg.get('rope_theta', (cfg.get('rope_parameters') or {}).get('rope_theta', 1e6))),
            rope_scaling=_rope_scaling_of(cfg), tie_word_embeddings=bool(cfg.get('tie_word_embeddings', False)),
            pre_norm=not olmo, qk_norm_full=olmo,
            qk_norm=olmo or mt.startswith('qwen3') or mt.startswith('gemma3') or (mt == 'glm4_moe' and bool(cfg.get('use_qk_norm'))),
            attention_bias=bool(cfg.get('attention_bias', cfg.get('qkv_bias', cfg.get('bias', False)) if mt.startswith('internlm') else mt.startswith('qwen2'))),
            router_scoring=('softmax_grouped' if v2 else 'sigmoid') if dsv3 else ('topk_softmax' if oss else 'softmax'), router_bias=dsv3 and not v2,
            n_group=int(cfg.get('n_group') or 1) if (dsv3 and not (v2 and cfg.get('topk_method', 'greedy') == 'greedy')) else 1,
            topk_group=int(cfg.get('topk_group') or 1) if dsv3 else 1, routed_scaling_factor=float(cfg.get('routed_scaling_factor', 1.0)) if dsv3 else 1.0,
            first_k_dense_replace=int(cfg.get('first_k_dense_replace', 0)) if dsv3 else 0, shared_expert_gate=not dsv3,
            q_lora_rank=cfg.get('q_lora_rank') if mla else None, kv_lora_rank=int(cfg.get('kv_lora_rank', 0)) if mla else 0,
            qk_nope_head_dim=int(cfg.get('qk_nope_head_dim', 128)), qk_rope_head_dim=int(cfg.get('qk_rope_head_dim', 64)),
            v_head_dim=int(cfg.get('v_head_dim', 128)), mla_rope_interleave=bool(cfg.get('rope_interleave', True)),
            hidden_act=act, embed_scale=float(cfg.get('embed_scale', cfg.get('hidden_size', 4096)**0.5 if mt.startswith('gemma') else (cfg.get('embedding_multiplier', 1.0) if granite else 1.0))),
            attn_sinks=oss, o_proj_bias=oss and bool(cfg.get('attention_bias', True)), router_linear_bias=oss, expert_bias=oss,
            expert_act='clamped_glu' if oss else 'swiglu',
            attn_logit_softcapping=cfg.get('attn_logit_softcapping') if gemma23 else None,
            final_logit_softcapping=cfg.get('final_logit_softcapping') if gemma23 else None,
            query_pre_attn_scalar=cfg.get('query_pre_attn_scalar') if gemma23 else (float(cfg['attention_multiplier'])**-2 if (granite and cfg.get('attention_multiplier')) else None),
            residual_multiplier=float(cfg.get('residual_multiplier', 1.0)) if granite else 1.0,
            logits_scaling=float(cfg.get('logits_scaling', 1.0)) if granite else 1.0,
            rope_local_theta=float(rope_local) if (rope_local and mt.startswith('gemma3')) else None,
            sliding_window=int(window) if window else None,
            num_experts=cfg.get('num_experts', cfg.get('num_local_experts', cfg.get('n_routed_experts', 0))) or 0,
            num_experts_per_tok=cfg.get('num_experts_per_tok', 8),
            moe_intermediate_size=cfg.get('moe_intermediate_size', cfg.get('intermediate_size', 768) if mt in ('mixtral', 'gpt_oss') else 768),
            norm_topk_prob=(True if cfg.get('norm_topk_prob') is None else bool(cfg['norm_topk_prob'])) and not v2, router_aux_loss_coef=float(cfg.get('router_aux_loss_coef', 0.0)),
            shared_expert_intermediate_size=int(cfg.get('shared_expert_intermediate_size', 0) or 0) if not dsv3
            else int(cfg.get('moe_intermediate_size', 0)) * int(cfg.get('n_shared_experts') or 0),
            rms_norm_offset=float(cfg.get('rms_norm_offset', 1.0 if (mt.startswith('gemma') or q35) else 0.0)),
            partial_rotary_factor=float(cfg.get('partial_rotary_factor', (cfg.get('rope_parameters') or {}).get('partial_rotary_factor', 1.0)) or 1.0),
            attn_output_gate=bool(cfg.get('attn_output_gate', q35)),
            rope_interleaved=bool(cfg.get('rope_interleaved', mt in ('glm', 'glm4', 'ernie4_5'))),
            no_rope_layers=[int(v) for v in cfg['no_rope_layers']] if (mt == 'smollm3' and cfg.get('no_rope_layers')) else None, sandwich_norm=bool(cfg.get('sandwich_norm', mt == 'glm4' or gemma23 or olmo)),
            layer_types=list(cfg['layer_types']) if cfg.get('layer_types') and ('linear_attention' in cfg['layer_types'] or ('sliding_attention' in cfg['layer_types'] and window)) else None,
            linear_num_key_heads=cfg.get('linear_num_key_heads', 16), linear_num_value_heads=cfg.get('linear_num_value_heads', 32),
            linear_key_head_dim=cfg.get('linear_key_head_dim', 128), linear_value_head_dim=cfg.get('linear_value_head_dim', 128),
            linear_conv_kernel_dim=cfg.get('linear_conv_kernel_dim', 4),
            vision=vision, image_token_id=top.get('image_token_id'), video_token_id=top.get('video_token_id'),
            vision_start_token_id=top.get('vision_start_token_id'), vision_end_token_id=top.get('vision_end_token_id'),
            mrope_section=list(rs_any['mrope_section']) if isinstance(rs_any, dict) and rs_any.get('mrope_section') and (vision is not None or not q35) else None,
            mrope_interleaved=bool(isinstance(rs_any, dict) and rs_any.get('mrope_interleaved')),
            initializer_range=cfg.get('initializer_range', 0.02), model_type=mt,
            torch_dtype=str(cfg.get('torch_dtype', cfg.get('dtype', 'bfloat16'))),
            max_position_embeddings=cfg.get('max_position_embeddings', 40960), pad_token_id=cfg.get('pad_token_id'),
            eos_token_id=cfg.get('eos_token_id') if not isinstance(cfg.get('eos_token_id'), list) else cfg['eos_token_id'][0])
        return out

    @classmethod
    def from_pretrained(cls, path: str) -> 'DecoderConfig':
        with open(os.path.join(path, 'config.json')) as f:
            cfg = json.load(f)
        sizes = _SIZES_FROM_TENSORS.get(cfg.get('architecture'))
        if sizes is not None:
            from ..utils.safetensors_io import SafetensorLazyLoader
            loader = SafetensorLazyLoader(path)
            sizes(cfg, lambda name: loader.get_slice(name).get_shape())
            loader.close()
        return cls.from_hf(cfg)

    def to_hf(self) -> Dict[str, Any]:
        if self.layer_specs is not None:
            return NATIVE_ARCHITECTURES[self.model_type.capitalize()][1](self)
        arch = 'Qwen3MoeForCausalLM' if self.is_moe else ('Qwen3ForCausalLM' if self.qk_norm else 'LlamaForCausalLM')
        arch = {'mixtral': 'MixtralForCausalLM', 'qwen2_moe': 'Qwen2MoeForCausalLM', 'qwen2': 'Qwen2ForCausalLM', 'mistral': 'MistralForCausalLM',
                'seed_oss': 'SeedOssForCausalLM'}.get(self.model_type, arch)
        d = {
            'architectures': [arch], 'model_type': self.model_type if self.model_type in ('mixtral', 'qwen2_moe') else ('qwen3_moe' if self.is_moe else self.model_type),
            'vocab_size': self.vocab_size, 'hidden_size': self.hidden_size, 'intermediate_size': self.intermediate_size,
            'num_hidden_layers': self.num_hidden_layers, 'num_attention_heads': self.num_attention_heads,
            'num_key_value_heads': self.num_key_value_heads, 'head_dim': self.head_dim, 'rms_norm_eps': self.rms_norm_eps,
            'rope_theta': self.rope_theta, 'tie_word_embeddings': self.tie_word_embeddings, 'attention_bias': self.attention_bias,
            'hidden_act': self.hidden_act, 'initializer_range': self.initializer_range, 'torch_dtype': self.torch_dtype,
            'max_position_embeddings': self.max_position_embeddings,
        }
        if self.is_moe:
            d.update(num_experts=self.num_experts, num_experts_per_tok=self.num_experts_per_tok,
                     moe_intermediate_size=self.moe_intermediate_size, norm_topk_prob=self.norm_topk_prob,
                     router_aux_loss_coef=self.router_aux_loss_coef, decoder_sparse_step=1, mlp_only_layers=[])
            if self.shared_expert_intermediate_size:
                d['shared_expert_intermediate_size'] = self.shared_expert_intermediate_size
            if self.model_type == 'mixtral':
                d.update(num_local_experts=self.num_experts, intermediate_size=self.moe_intermediate_size, sliding_window=None)
        if self.rms_norm_offset:
            d['rms_norm_offset'] = self.rms_norm_offset
        if self.sliding_window:
            d['sliding_window'] = self.sliding_window
        if self.is_mla:
            d.update(architectures=['DeepseekV2ForCausalLM' if self.model_type == 'deepseek_v2' else 'DeepseekV3ForCausalLM'], model_type=self.model_type,
                     topk_method='group_limited_greedy' if self.n_group > 1 else 'greedy', q_lora_rank=self.q_lora_rank, kv_lora_rank=self.kv_lora_rank,
                     qk_nope_head_dim=self.qk_nope_head_dim, qk_rope_head_dim=self.qk_rope_head_dim, v_head_dim=self.v_head_dim,
                     rope_interleave=self.mla_rope_interleave, head_dim=self.qk_rope_head_dim, n_routed_experts=self.num_experts,
                     n_shared_experts=(self.shared_expert_intermediate_size // self.moe_intermediate_size) if self.num_experts else 0,
                     n_group=self.n_group, topk_group=self.topk_group, routed_scaling_factor=self.routed_scaling_factor,
                     first_k_dense_replace=self.first_k_dense_replace, norm_topk_prob=self.norm_topk_prob,
                     num_experts_per_tok=self.num_experts_per_tok, moe_intermediate_size=self.moe_intermediate_size)
            for k in ('num_experts', 'shared_expert_intermediate_size', 'decoder_sparse_step', 'mlp_only_layers'):
                d.pop(k, None)
        elif self.model_type == 'ernie4_5':
            d.update(architectures=['Ernie4_5ForCausalLM'], use_bias=self.attention_bias)
        elif self.model_type == 'smollm3':
            d.update(architectures=['SmolLM3ForCausalLM'], no_rope_layers=list(self.no_rope_layers or [1] * self.num_hidden_layers), use_sliding_window=False,
                     pad_token_id=self.pad_token_id if self.pad_token_id is not None else 0)
        elif self.model_type in ('olmo2', 'olmo3'):
            d.update(architectures=['Olmo3ForCausalLM' if self.model_type == 'olmo3' else 'Olmo2ForCausalLM'], model_type=self.model_type)
            if self.model_type == 'olmo3':
                d.update(sliding_window=self.sliding_window, layer_types=list(self.layer_types or ['full_attention'] * self.num_hidden_layers))
        elif self.model_type == 'granite':
            d.update(architectures=['GraniteForCausalLM'], embedding_multiplier=self.embed_scale, residual_multiplier=self.residual_multiplier,
                     logits_scaling=self.logits_scaling, attention_multiplier=self.attn_scale, mlp_bias=False)
        elif self.model_type == 'gpt_oss':
            d.update(architectures=['GptOssForCausalLM'], model_type='gpt_oss', num_local_experts=self.num_experts, intermediate_size=self.moe_intermediate_size,
                     sliding_window=self.sliding_window, layer_types=list(self.layer_types or ['full_attention'] * self.num_hidden_layers),
                     attention_bias=self.attention_bias, swiglu_limit=7.0, num_experts_per_tok=self.num_experts_per_tok,
                     router_aux_loss_coef=self.router_aux_loss_coef)
            for k in ('num_experts', 'moe_intermediate_size', 'norm_topk_prob', 'decoder_sparse_step', 'mlp_only_layers', 'shared_expert_intermediate_size'):
                d.pop(k, None)
        elif self.model_type == 'glm4_moe':
            d.update(architectures=['Glm4MoeForCausalLM'], model_type='glm4_moe', use_qk_norm=self.qk_norm, n_routed_experts=self.num_experts,
                     n_shared_experts=self.shared_expert_intermediate_size // self.moe_intermediate_size, n_group=self.n_group,
                     topk_group=self.topk_group, routed_scaling_factor=self.routed_scaling_factor, first_k_dense_replace=self.first_k_dense_replace,
                     partial_rotary_factor=self.partial_rotary_factor,
                     rope_parameters={'rope_type': 'default', 'rope_theta': self.rope_theta, 'partial_rotary_factor': self.partial_rotary_factor})
            for k in ('num_experts', 'shared_expert_intermediate_size', 'decoder_sparse_step', 'mlp_only_layers'):
                d.pop(k, None)
        elif self.model_type == 'phi3':
            d.update(architectures=['Phi3ForCausalLM'], partial_rotary_factor=self.partial_rotary_factor,
                     pad_token_id=self.pad_token_id, sliding_window=self.sliding_window,
                     original_max_position_embeddings=(self.rope_scaling or {}).get('original_max_position_embeddings', self.max_position_embeddings))
        elif self.model_type == 'gemma':
            d.update(architectures=['GemmaForCausalLM'], hidden_activation=self.hidden_act)
            d.pop('rms_norm_offset', None)
        elif self.model_type in ('gemma2', 'gemma3_text', 'gemma3'):
            g3 = self.model_type != 'gemma2'
            d.update(architectures=['Gemma3ForCausalLM' if g3 else 'Gemma2ForCausalLM'], model_type='gemma3_text' if g3 else 'gemma2',
                     hidden_activation=self.hidden_act, query_pre_attn_scalar=self.query_pre_attn_scalar, sliding_window=self.sliding_window,
                     attn_logit_softcapping=self.attn_logit_softcapping, final_logit_softcapping=self.final_logit_softcapping,
                     layer_types=list(self.layer_types or ['full_attention'] * self.num_hidden_layers))
            if g3:
                glob = dict(self.rope_scaling or {'rope_type': 'default'}, rope_theta=self.rope_theta)
                d['rope_parameters'] = {'full_attention': glob, 'sliding_attention': {'rope_type': 'default', 'rope_theta': self.rope_local_theta or self.rope_theta}}
                d.pop('rope_scaling', None)
                d.pop('rope_theta', None)
            d.pop('rms_norm_offset', None)
        elif self.model_type == 'internlm2':
            d.update(architectures=['InternLM2ForCausalLM'], bias=self.attention_bias)
        elif self.model_type == 'internlm3':
            d.update(architectures=['InternLM3ForCausalLM'], qkv_bias=self.attention_bias, bias=False)
        if self.rope_scaling:
            d['rope_scaling'] = dict(self.rope_scaling)
        if self.vision and not self.model_type.startswith('qwen3_5'):
            fam = self.vision.get('model_type', 'qwen2_vl')
            if fam == 'qwen3_vl' and self.is_moe:
                fam = 'qwen3_vl_moe'
            rope = {'type': 'mrope', 'mrope_section': list(self.mrope_section or [])}
            if fam.startswith('qwen3_vl'):
                rope = {'rope_type': 'default', 'mrope_section': list(self.mrope_section or []), 'mrope_interleaved': self.mrope_interleaved}
            text = dict(d, model_type=fam + '_text', rope_scaling=rope)
            text.pop('architectures', None)
            arch = {'qwen2_vl': 'Qwen2VLForConditionalGeneration', 'qwen2_5_vl': 'Qwen2_5_VLForConditionalGeneration',
                    'qwen3_vl': 'Qwen3VLForConditionalGeneration', 'qwen3_vl_moe': 'Qwen3VLMoeForConditionalGeneration'}[fam]
            vis = dict(self.vision, model_type=fam) if fam == 'qwen3_vl_moe' else dict(self.vision)
            return {'architectures': [arch], 'model_type': fam, 'text_config': text,
                    'vision_config': vis, 'image_token_id': self.image_token_id, 'video_token_id': self.video_token_id,
                    'vision_start_token_id': self.vision_start_token_id, 'vision_end_token_id': self.vision_end_token_id,
                    'tie_word_embeddings': self.tie_word_embeddings, 'torch_dtype': self.torch_dtype}
        if self.layer_types and 'linear_attention' not in self.layer_types:
            d['layer_types'] = list(self.layer_types)
        elif self.layer_types:
            d.update(layer_types=list(self.layer_types), linear_num_key_heads=self.linear_num_key_heads,
                     linear_num_value_heads=self.linear_num_value_heads, linear_key_head_dim=self.linear_key_head_dim,
                     linear_value_head_dim=self.linear_value_head_dim, linear_conv_kernel_dim=self.linear_conv_kernel_dim)
        if self.model_type in ('glm', 'glm4'):
            d.update(architectures=['Glm4ForCausalLM' if self.model_type == 'glm4' else 'GlmForCausalLM'], model_type=self.model_type,
                     partial_rotary_factor=self.partial_rotary_factor, pad_token_id=self.pad_token_id if self.pad_token_id is not None else 0,
                     rope_parameters={'rope_type': 'default', 'rope_theta': self.rope_theta, 'partial_rotary_factor': self.partial_rotary_factor})
        elif self.model_type == 'qwen3_next':
            d.update(architectures=['Qwen3NextForCausalLM'], model_type='qwen3_next', partial_rotary_factor=self.partial_rotary_factor,
                     rope_parameters={'rope_type': 'default', 'rope_theta': self.rope_theta, 'partial_rotary_factor': self.partial_rotary_factor},
                     layer_types=list(self.layer_types or ['full_attention'] * self.num_hidden_layers))
            d.pop('rms_norm_offset', None)
        elif self.model_type.startswith('qwen3_5'):
            # written as the text model of the family (what ``Qwen3_5ForCausalLM`` loads)
            d.update(architectures=['Qwen3_5MoeForCausalLM' if self.is_moe else 'Qwen3_5ForCausalLM'],
                     model_type='qwen3_5_moe_text' if self.is_moe else 'qwen3_5_text', partial_rotary_factor=self.partial_rotary_factor,
                     rope_parameters={'rope_type': 'default', 'rope_theta': self.rope_theta, 'partial_rotary_factor': self.partial_rotary_factor},
                     layer_types=list(self.layer_types or ['full_attention'] * self.num_hidden_layers))
            d.pop('rms_norm_offset', None)
            if self.vision:      # the full model: the Qwen3-VL tower without its deep-stack taps in front of the hybrid decoder
                fam = 'qwen3_5_moe' if self.is_moe else 'qwen3_5'
                d['rope_parameters'].update(mrope_section=list(self.mrope_section or []), mrope_interleaved=self.mrope_interleaved)
                text = {k: v for k, v in d.items() if k != 'architectures'}
                return {'architectures': ['Qwen3_5MoeForConditionalGeneration' if self.is_moe else 'Qwen3_5ForConditionalGeneration'], 'model_type': fam,
                        'text_config': text, 'vision_config': dict(self.vision, model_type=fam), 'image_token_id': self.image_token_id,
                        'video_token_id': self.video_token_id, 'vision_start_token_id': self.vision_start_token_id,
                        'vision_end_token_id': self.vision_end_token_id, 'tie_word_embeddings': self.tie_word_embeddings, 'torch_dtype': self.torch_dtype}
        elif self.partial_rotary_factor != 1.0 or self.attn_output_gate:
            d.update(partial_rotary_factor=self.partial_rotary_factor, attn_output_gate=self.attn_output_gate)
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, 'config.json'), 'w') as f:
            json.dump(self.to_hf(), f, indent=2)


def _nilepel_bench_mixer(i: int) -> Dict[str, Any]:
    """Mixer of layer ``i`` of the Nilepel benchmark preset."""
    heads = dict(heads=32, dim=128, vdim=128)
    if i % 4 == 1:
        return dict(heads, q_rank=0, kv_rank=512, scale=192**-0.5, rot_dim=64, rotary=dict(dims=64, base=1e4, interleaved=True), window=4096, sinks=False, head_gate=False)
    grouped = dict(heads, kv_heads=4, scale=128**-0.5, sinks=True)
    if i % 4 == 2:
        return dict(grouped, rotary=dict(dims=128, base=5e5, interleaved=True), chunk=4096)
    return dict(grouped, rotary=dict(dims=128, base=1e6, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192)), window=1024, bias=True, qk_norm=True, head_gate=True,
                kv_from=i - 3 if i % 4 == 3 else None)


def _puzonex_bench_mixer(i: int) -> Dict[str, Any]:
    """Mixer of layer ``i`` of the Puzonex benchmark preset."""
    if i % 4 >= 2:
        return dict(inner=8192, state=16, dt_rank=256, conv=4)
    heads = dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=128**-0.5, bias=True)
    if i % 4 == 1:
        return dict(heads, qk_norm=True, value_norm=True, log_bias=True, sinks=True, softcap=30.0, window=4096)
    return dict(left=dict(heads, qk_norm='whole', values_are_keys=True, temperature=True, buckets=32, bias_max=1024, softcap=50.0, window=1024, out_gate=True, out_bias=True),
                right=dict(heads=16, dim=128, vdim=256, gate_cap=15.0))


PRESETS: Dict[str, Dict[str, Any]] = {
    # the smallest end-to-end configuration (LoRA SFT on CPU)
    'tiny-dense': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=2, num_attention_heads=4,
                       num_key_value_heads=2, head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=True,
                       torch_dtype='float32'),
    'tiny-hybrid': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=4, num_attention_heads=4,
                        num_key_value_heads=2, head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=True, torch_dtype='float32',
                        layer_types=['linear_attention', 'full_attention', 'linear_attention', 'full_attention'], linear_num_key_heads=2,
                        linear_num_value_heads=4, linear_key_head_dim=32, linear_value_head_dim=32),
    # the Qwen3.5 text stack in small: three Gated DeltaNet layers per full-attention layer, output gate, rotary on a quarter
    # of the head, "1 + w" norms
    'tiny-qwen3.5': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=4, num_attention_heads=4,
                         num_key_value_heads=2, head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=True, torch_dtype='float32',
                         model_type='qwen3_5_text', rms_norm_offset=1.0, partial_rotary_factor=0.25, attn_output_gate=True,
                         layer_types=['linear_attention', 'linear_attention', 'linear_attention', 'full_attention'], linear_num_key_heads=2,
                         linear_num_value_heads=4, linear_key_head_dim=32, linear_value_head_dim=32),
    # DeepSeek-V3 in small: latent attention with a query bottleneck, one dense layer then mixture-of-experts layers with sigmoid
    # routing over expert groups, selection bias and an ungated shared expert
    'tiny-deepseek': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=3, num_attention_heads=4, num_key_value_heads=4,
                          head_dim=48, rope_theta=1e4, tie_word_embeddings=False, qk_norm=False, torch_dtype='float32', model_type='deepseek_v3',
                          q_lora_rank=64, kv_lora_rank=32, qk_nope_head_dim=32, qk_rope_head_dim=16, v_head_dim=32, num_experts=8,
                          num_experts_per_tok=2, moe_intermediate_size=128, shared_expert_intermediate_size=128, shared_expert_gate=False,
                          router_scoring='sigmoid', router_bias=True, n_group=4, topk_group=2, routed_scaling_factor=2.5, first_k_dense_replace=1),
    # GPT-OSS in small: sink logits, alternating sliding-window layers, biased projections / router / experts, top-k-then-softmax routing
    'tiny-gpt-oss': dict(vocab_size=1024, hidden_size=256, num_hidden_layers=4, num_attention_heads=4, num_key_value_heads=2, head_dim=64,
                         rope_theta=1.5e5, tie_word_embeddings=False, qk_norm=False, torch_dtype='float32', model_type='gpt_oss', attention_bias=True,
                         o_proj_bias=True, attn_sinks=True, router_linear_bias=True, expert_bias=True, expert_act='clamped_glu',
                         router_scoring='topk_softmax', num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128, sliding_window=16,
                         layer_types=['sliding_attention', 'full_attention', 'sliding_attention', 'full_attention']),
    'tiny-moe': dict(vocab_size=1024, hidden_size=256, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2,
                     head_dim=64, rope_theta=1e4, tie_word_embeddings=True, num_experts=8, num_experts_per_tok=2,
                     moe_intermediate_size=128, router_aux_loss_coef=1e-3, torch_dtype='float32'),
    'tiny-vl': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2,
                    head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=False, attention_bias=True, torch_dtype='float32',
                    model_type='qwen2_vl_text', mrope_section=[8, 12, 12], image_token_id=265, video_token_id=267, vision_start_token_id=264,
                    vision_end_token_id=266,  # ids of these tokens in the byte-level test tokenizer
                    vision=dict(depth=2, embed_dim=64, hidden_size=256, num_heads=4, mlp_ratio=2, patch_size=14,
                                                          spatial_merge_size=2, temporal_patch_size=2, in_channels=3)),
    'tiny-vl3': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=3, num_attention_heads=4, num_key_value_heads=2,
                     head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=True, torch_dtype='float32', model_type='qwen3_vl_text',
                     mrope_section=[8, 12, 12], mrope_interleaved=True, image_token_id=265, video_token_id=267, vision_start_token_id=264,
                     vision_end_token_id=266,
                     vision=dict(depth=3, hidden_size=64, out_hidden_size=256, intermediate_size=96, num_heads=4, patch_size=16, spatial_merge_size=2,
                                 temporal_patch_size=2, in_channels=3, num_position_embeddings=64, deepstack_visual_indexes=[0, 2])),
    # Qwen3.5 vision-language in small: the Qwen3-VL tower (no deep-stack taps) in front of the hybrid decoder
    'tiny-qwen3.5-vl': dict(vocab_size=1024, hidden_size=256, intermediate_size=688, num_hidden_layers=4, num_attention_heads=4, num_key_value_heads=2,
                            head_dim=64, rope_theta=1e4, tie_word_embeddings=True, qk_norm=True, torch_dtype='float32', model_type='qwen3_5',
                            rms_norm_offset=1.0, partial_rotary_factor=0.25, attn_output_gate=True,
                            layer_types=['linear_attention', 'linear_attention', 'linear_attention', 'full_attention'], linear_num_key_heads=2,
                            linear_num_value_heads=4, linear_key_head_dim=32, linear_value_head_dim=32, mrope_section=[2, 3, 3], mrope_interleaved=True,
                            image_token_id=265, video_token_id=267, vision_start_token_id=264, vision_end_token_id=266,
                            vision=dict(depth=2, hidden_size=64, out_hidden_size=256, intermediate_size=96, num_heads=4, patch_size=16, spatial_merge_size=2,
                                        temporal_patch_size=2, in_channels=3, num_position_embeddings=64)),
    'tiny-moe-shared': dict(vocab_size=1024, hidden_size=256, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2,
                            head_dim=64, rope_theta=1e4, tie_word_embeddings=True, num_experts=8, num_experts_per_tok=2,
                            moe_intermediate_size=128, shared_expert_intermediate_size=192, torch_dtype='float32'),
    # Pomelix in small: layers of unequal widths and head counts, one without a feed-forward block, one without convolution
    'tiny-pomelix': dict(vocab_size=1024, hidden_size=192, tie_word_embeddings=True, qk_norm=False, torch_dtype='float32', model_type='pomelix',
                         rms_norm_eps=1e-5, residual_multiplier=0.5,
                         layer_specs=[dict(heads=6, kv_heads=2, dim=24, vdim=40, scale=0.3, conv=3, temp_coef=0.2, temp_every=16, v_mix=False, ff=256),
                                      dict(heads=4, kv_heads=2, dim=32, vdim=32, scale=0.2, conv=4, temp_coef=0.2, temp_every=16, v_mix=True, ff=0),
                                      dict(heads=8, kv_heads=2, dim=16, vdim=32, scale=0.25, conv=0, v_mix=True, ff=160)]),
    # Pomelix layers at the sizes of the Qwen3 presets (benchmarks)
    'pomelix-0.6b': dict(vocab_size=151936, hidden_size=1024, tie_word_embeddings=True, qk_norm=False, model_type='pomelix', rms_norm_eps=1e-5,
                         residual_multiplier=0.5, layer_specs=[dict(heads=16, kv_heads=8, dim=128, vdim=128, scale=128**-0.5, conv=4, temp_coef=0.1,
                                                                    temp_every=4096, v_mix=True, ff=3072)] * 28),
    'pomelix-8b': dict(vocab_size=151936, hidden_size=4096, tie_word_embeddings=True, qk_norm=False, model_type='pomelix', rms_norm_eps=1e-5,
                       residual_multiplier=0.5, layer_specs=[dict(heads=32, kv_heads=8, dim=128, vdim=128, scale=128**-0.5, conv=4, temp_coef=0.1,
                                                                  temp_every=4096, v_mix=True, ff=12288)] * 36),
    # Moronex in small: recurrent and latent-attention layers of unequal sizes, a borrowed latent, dense / expert / no feed-forward
    'tiny-moronex': dict(vocab_size=1024, hidden_size=192, tie_word_embeddings=False, qk_norm=False, torch_dtype='float32', model_type='moronex',
                         rms_norm_eps=1e-5, rms_norm_offset=1.0,
                         layer_specs=[dict(mixer=dict(heads=3, dim=24, vdim=48), mlp=dict(ff=320)),
                                      dict(mixer=dict(heads=6, dim=40, vdim=24, q_rank=72, kv_rank=56, scale=0.2), mlp=dict(ff=64, experts=6, top=2)),
                                      dict(mixer=dict(heads=2, dim=48, vdim=40)),
                                      dict(mixer=dict(heads=4, dim=24, vdim=32, q_rank=48, kv_rank=56, scale=0.25, kv_from=1), mlp=dict(ff=80, experts=5, top=3))]),
    # Moronex layers at the width, experts and depth of Qwen3-30B-A3B (benchmarks): three recurrent layers per latent-attention layer,
    # every second of those borrowing the latents of the one before
    'moronex-30b-a3b': dict(vocab_size=151936, hidden_size=2048, tie_word_embeddings=False, qk_norm=False, model_type='moronex', rms_norm_eps=1e-6,
                            rms_norm_offset=1.0,
                            layer_specs=[dict(mixer=dict(heads=16, dim=128, vdim=128) if i % 4 != 3 else
                                              dict(heads=32, dim=128, vdim=128, q_rank=1024, kv_rank=512, scale=128**-0.5, kv_from=i - 4 if i % 8 == 7 else None),
                                              mlp=dict(ff=6144) if i == 0 else dict(ff=1152, experts=128, top=8)) for i in range(48)]),
    # Nilepel in small: a window with experts beside a shared one, a chunk, rotated latents, borrowed keys and values
    'tiny-nilepel': dict(vocab_size=1024, hidden_size=192, tie_word_embeddings=False, qk_norm=False, torch_dtype='float32', model_type='nilepel', rms_norm_eps=1e-5, embed_scale=4.0,
                         layer_specs=[dict(mixer=dict(heads=6, kv_heads=2, dim=24, vdim=40, scale=0.2, rotary=dict(dims=16, base=1e4), window=48, bias=True, qk_norm=True,
                                                      sinks=True, head_gate=True),
                                           mlp=dict(ff=64, experts=6, top=2, gated=True, scoring='softmax_grouped', groups=3, keep=2, scale=1.5, shared=48), post=False),
                                      dict(mixer=dict(heads=4, kv_heads=4, dim=32, vdim=32, scale=0.2, rotary=dict(dims=32, base=1e3, interleaved=True), chunk=40, sinks=True),
                                           mlp=dict(ff=256, limit=2.0), post=False),
                                      dict(mixer=dict(heads=5, dim=24, vdim=24, q_rank=0, kv_rank=56, scale=0.2, rot_dim=16, rotary=dict(dims=16, base=1e4, interleaved=True), window=64,
                                                      sinks=False, head_gate=False), mlp=None, post=False),
                                      dict(mixer=dict(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.2, rotary=dict(dims=16, base=1e4), window=32, bias=True, qk_norm=True,
                                                      sinks=True, head_gate=True, kv_from=0), mlp=dict(ff=128, limit=1.0), post=False)]),
    # Nilepel layers at the width, experts and depth of Qwen3-30B-A3B (benchmarks): of four layers a window of 1024, rotated latents in a
    # window of 4096, a chunk of 4096, and a window on the first one's keys and values
    'nilepel-30b-a3b': dict(vocab_size=151936, hidden_size=2048, tie_word_embeddings=False, qk_norm=False, model_type='nilepel', rms_norm_eps=1e-6, embed_scale=2048**0.5,
                            layer_specs=[dict(mixer=_nilepel_bench_mixer(i), mlp=dict(ff=6144, limit=7.0) if i == 0 else
                                              dict(ff=768, experts=128, top=8, gated=True, scoring='softmax_grouped', groups=8, keep=4, scale=1.0, shared=768), post=False)
                                         for i in range(48)]),
    # Puzonex in small: attention beside a matrix memory, a scan, attention with sinks, a layer without a feed-forward block
    'tiny-puzonex': dict(vocab_size=1024, hidden_size=192, tie_word_embeddings=False, qk_norm=False, torch_dtype='float32', model_type='puzonex', rms_norm_eps=1e-5, sinusoidal_base=1e4,
                         layer_specs=[dict(mixer=dict(left=dict(heads=6, kv_heads=2, dim=24, vdim=24, scale=0.2, window=40, bias=True, qk_norm='whole', values_are_keys=True,
                                                                temperature=True, softcap=20.0, buckets=16, bias_max=32, out_gate=True, out_bias=True),
                                                      right=dict(heads=3, dim=24, vdim=40, gate_cap=8.0)), mlp=dict(ff=256, act='gelu_tanh'), pre=False),
                                      dict(mixer=dict(inner=224, state=12, dt_rank=24, conv=3), mlp=dict(ff=160, act='gelu_tanh'), pre=False),
                                      dict(mixer=dict(heads=4, kv_heads=4, dim=32, vdim=40, scale=0.2, window=24, bias=True, qk_norm=True, value_norm=True, log_bias=True, sinks=True,
                                                      softcap=15.0), mlp=None, pre=False)]),
    # Puzonex layers at the width of Qwen3-8B and about its parameters (benchmarks): of four layers attention beside a matrix memory in a window of 1024,
    # attention in a window of 4096, and two scans
    'puzonex-8b': dict(vocab_size=151936, hidden_size=4096, tie_word_embeddings=False, qk_norm=False, model_type='puzonex', rms_norm_eps=1e-5, sinusoidal_base=1e4,
                       layer_specs=[dict(mixer=_puzonex_bench_mixer(i), mlp=dict(ff=12288, act='gelu_tanh'), pre=False) for i in range(28)]),
    'qwen3-0.6b': dict(hidden_size=1024, intermediate_size=3072, num_hidden_layers=28, num_attention_heads=16,
                       num_key_value_heads=8, head_dim=128, tie_word_embeddings=True),
    'qwen3-8b': dict(hidden_size=4096, intermediate_size=12288, num_hidden_layers=36, num_attention_heads=32,
                     num_key_value_heads=8, head_dim=128),
    'qwen3-32b': dict(hidden_size=5120, intermediate_size=25600, num_hidden_layers=64, num_attention_heads=64,
                      num_key_value_heads=8, head_dim=128),
    'qwen3-30b-a3b': dict(hidden_size=2048, intermediate_size=6144, num_hidden_layers=48, num_attention_heads=32,
                          num_key_value_heads=4, head_dim=128, num_experts=128, num_experts_per_tok=8,
                          moe_intermediate_size=768, router_aux_loss_coef=1e-3),
}


def preset(name: str, **overrides) -> DecoderConfig:
    kw = dict(PRESETS[name.lower()])
    n = overrides.get('num_hidden_layers')
    if kw.get('layer_specs') and n:      # listed layers: the list repeated or cut to the wanted depth
        kw['layer_specs'] = (list(kw['layer_specs']) * -(-n // len(kw['layer_specs'])))[:n]
    kw.update(overrides)
    return DecoderConfig(**kw)
