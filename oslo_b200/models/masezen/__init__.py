from .modeling_masezen import (  # noqa: F401
    MasezenConfig, MasezenModel, MasezenForCausalLM, MasezenForSequenceClassification, MasezenLayerPolicy, MasezenBlock,
    MasezenPreTrainedModel)
