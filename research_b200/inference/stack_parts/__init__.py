"""Building blocks of layer-stack models on the engine: one class per kind of mixer and feed-forward.

A part is made once per runner and kind. It knows the limits of its kernels, allocates and loads the padded weights of
every layer of its kind (``make`` / ``load``), the cache or state of every run of such a layer (``new_cache``) and the shared
activations (``allocate``), plans a step for all its layers at once (``plan``) and runs one layer (``forward``).
"""

from ...models.stack import (ClampedGluSpec, DeltaRuleSpec, ExpertsSpec, GluSpec, GroupedAttentionSpec, KeyValueAttentionSpec, LatentAttentionSpec,
                             LightningSpec, MatrixMemorySpec, NormedPairSpec, ParallelSpec, PolyNormSpec, TimeMixSpec)
from .feedforward import DensePart, ExpertsPart, PolyNormPart
from .grouped import GroupedPart
from .keyvalue import KeyValuePart
from .latent import LatentPart
from .parallel import NormedPairPart, ParallelPart
from .recurrent import DeltaPart, RecurrentPart, TimeMixPart

MIXER_PARTS = {LatentAttentionSpec: LatentPart, KeyValueAttentionSpec: KeyValuePart, LightningSpec: RecurrentPart, MatrixMemorySpec: RecurrentPart,
               GroupedAttentionSpec: GroupedPart, TimeMixSpec: TimeMixPart, ParallelSpec: ParallelPart, NormedPairSpec: NormedPairPart,
               DeltaRuleSpec: DeltaPart}
FEED_FORWARD_PARTS = {ClampedGluSpec: DensePart, GluSpec: DensePart, PolyNormSpec: PolyNormPart, ExpertsSpec: ExpertsPart}
