"""What decoder models put together from mixers.py have in common: layers whose configuration lists them
one by one, a 32-bit residual stream, weights by name, and a cache run (a pool of keys and values, of
latents, or of recurrent states) for every time a layer is run per token."""
from __future__ import annotations

from typing import Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from .cache import PagedKVCache, RecurrentStateCache
from .loader import copy_weights
from .parallel_state import get_tensor_model_parallel_world_size


class DecoderLayer(nn.Module):
    """norm1, a mixer and, where there is a feed-forward, norm2 and the feed-forward."""

    def __init__(self, mixer: nn.Module, mlp: Optional[nn.Module], width: int, norm_init: float, device):
        super().__init__()
        norm = lambda: nn.Parameter(torch.full((width,), norm_init, dtype=torch.float32, device=device),
                                    requires_grad=False)
        self.mixer, self.norm1 = mixer, norm()
        self.mlp, self.norm2 = mlp, norm() if mlp is not None else None


class LayeredDecoder(nn.Module):
    """A subclass sets `layers` (DecoderLayers), calls `plan_cache` and adds its own tensors in
    `top_weights`."""
    supports_portions = True            # a prompt may be continued from the cache and state

    def __init__(self, cfg, device, seed: int, dtype: torch.dtype):
        super().__init__()
        if get_tensor_model_parallel_world_size() != 1:
            raise ValueError("this model runs on one rank")
        # 16-bit GEMMs accumulate in 32 bits throughout, 32-bit ones use no reduced-precision mode
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        torch.backends.cuda.matmul.allow_fp16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        self._gen = torch.Generator(device=device).manual_seed(seed)

    def _random(self, *shape, std: float, dtype: Optional[torch.dtype] = None) -> nn.Parameter:
        t = torch.empty(shape, dtype=dtype or self.dtype, device=self.device)
        return nn.Parameter(t.normal_(0, std, generator=self._gen), requires_grad=False)

    # -- cache -------------------------------------------------------------------------
    def plan_cache(self, order: Sequence[int]) -> List[int]:
        """`order`: layer numbers in the order they run.  Returns each run's number among the runs of its
        kind; a mixer with `shares` reads the (only) run of that layer and has none of its own."""
        runs, at = [], {}
        self._kv_shapes: List[Tuple[int, int, int]] = []
        self._state_shapes: List[Tuple[int, int, int]] = []
        self._normalised: List[bool] = []
        windows: List[Optional[int]] = []
        for i in order:
            mixer = self.layers[i].mixer
            if mixer.kind == "kv":
                windows.append(mixer.window)
                if mixer.shares is not None:
                    runs.append(at[mixer.shares])
                    continue
                self._kv_shapes.append(mixer.cache_shape)
                runs.append(len(self._kv_shapes) - 1)
            else:
                self._state_shapes.append(mixer.cache_shape)
                self._normalised.append(mixer.normalised)
                runs.append(len(self._state_shapes) - 1)
            at[i] = runs[-1]
        # how far any layer looks back; None: to the first token
        self.window = None if None in windows else max(windows, default=0)
        self.kv_heads = max([h for h, _, _ in self._kv_shapes], default=1)
        return runs

    def make_cache(self, num_blocks: int, block_size: int, max_seqs: int) -> PagedKVCache:
        state = None
        if self._state_shapes:
            state = RecurrentStateCache(self._state_shapes, max_seqs, self.device, self._normalised)
        return PagedKVCache(len(self._kv_shapes), num_blocks, self.kv_heads, block_size, self.dtype, self.device,
                            layer_shapes=self._kv_shapes, window=self.window, state=state)

    # -- weights -----------------------------------------------------------------------
    def top_weights(self) -> Dict[str, torch.Tensor]:
        """Checkpoint names of the tensors outside the layers."""
        raise NotImplementedError

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        want = {k: [v] for k, v in self.top_weights().items()}
        for i, layer in enumerate(self.layers):
            want[f"l{i}.norm1"] = [layer.norm1]
            want.update({f"l{i}.mix.{k}": [v] for k, v in layer.mixer.weight_views().items()})
            if layer.mlp is not None:
                want[f"l{i}.norm2"] = [layer.norm2]
                want.update({f"l{i}.mlp.{k}": [v] for k, v in layer.mlp.weight_views().items()})
        copy_weights(want, tensors)
        self.finalize()

    def finalize(self) -> None:
        for layer in self.layers:
            layer.mixer.prepare()

    # -- sampling ------------------------------------------------------------------------
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def greedy_tokens(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits(hidden).argmax(dim=-1)
