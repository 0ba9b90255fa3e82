// Model families of the decode driver.  A directory with a config.json is a layered model (model_spec.cu picks the
// architecture); one without is a tree in the INT4 container format.  Built once more with BW_CONFIG_MODELS_ONLY for
// programs that serve config.json models alone and do not link the INT4 kernels.
#include <stdio.h>

#include "decode_model.h"

namespace bw {

std::unique_ptr<DecodeModel> make_decode_model(const std::string& dir) {
    FILE* f = fopen((dir + "/config.json").c_str(), "rb");
    if (f) {
        fclose(f);
        return make_layered_model();
    }
#ifdef BW_CONFIG_MODELS_ONLY
    return nullptr;
#else
    return make_int4_model();
#endif
}

}  // namespace bw
